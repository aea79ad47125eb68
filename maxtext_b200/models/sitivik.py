"""Sitivik: a decoder whose layers run softmax attention and a linear recurrence side by side, with differential attention in between.

Every layer names its own mixer, sizes and feed-forward (`layer_specs`):

  parallel     sliding-window attention beside retention; each result is RMS-normalised, the halves are added
  parallel_2   chunked attention beside the gated delta rule with a decay per key channel, weighted by two constants
  attention    differential attention over every earlier token, without rotation, with a query temperature

The residual stream is fp32 and pre-normed; a learned factor per lane scales every branch, and after the feed-forward a second, narrow
embedding of the token joins the stream (`layers.parallel.TokenSide`). The head is the embedding table. The attention kinds are
`layers.blocks.Attention` with per-layer sizes, the recurrences `layers.retention` and `layers.channel_delta`, the pairs
`layers.parallel.ParallelMixer`. This file holds what is particular to the design: how its config.json becomes configuration keys,
its layer plans, and how its tensors map to parameters.
"""
from __future__ import annotations

import torch

MIXERS = ("parallel", "parallel_2", "attention")


# ------------------------------------------------------------------------------------------ configuration
def keys_from_json(spec: dict, shapes: dict) -> dict:
  layers = []
  for i, lay in enumerate(spec["layers"]):
    kind, mixer = lay["type"], dict(lay["mixer"])
    if kind not in MIXERS:
      raise ValueError(f"layer {i}: unknown mixer type {kind!r} (known: {list(MIXERS)})")
    mlp = lay.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
      raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    if kind == "parallel_2":                                       # ranks that only the tensors give
      mixer["right"] = dict(mixer["right"], decay_rank=int(shapes[f"l{i}.mix.right.a1"][0]), gate_rank=int(shapes[f"l{i}.mix.right.g1"][0]))
    layers.append({"type": kind, "mixer": mixer, "mlp": dict(mlp) if mlp is not None else None})
  return {"decoder_block": "sitivik", "layer_specs": layers, "base_emb_dim": int(spec["width"]), "vocab_size": int(spec["vocab"]),
          "base_num_decoder_layers": len(layers), "normalization_layer_epsilon": float(spec["norm"]["eps"]),
          "embedding_multiplier": float(spec["embedding"]["scale"]), "token_side_dim": int(spec["token_side"]["dim"]),
          "mlp_activations": ["silu", "linear"], "logits_via_embedding": True, "normalize_embedding_logits": False}


def validate(t: dict) -> None:
  """Cross-field checks of the layer list (run with the other validators when a configuration is built)."""
  def need(ok, why):
    if not ok:
      raise ValueError(why)

  def heads(at, m, widest):
    need(m["heads"] % m["kv_heads"] == 0, f"{at}: heads must be a multiple of kv_heads")
    need(max(m["dim"], m["vdim"]) <= widest and min(m["dim"], m["vdim"]) >= 1, f"{at}: head widths between 1 and {widest} are supported")

  def rotation(at, m):
    need(m["rot"]["dims"] % 2 == 0 and 0 <= m["rot"]["dims"] <= m["dim"], f"{at}: rot.dims must be even and at most dim")

  need(len(t["layer_specs"]) == int(t["base_num_decoder_layers"]),
       f"layer_specs names {len(t['layer_specs'])} layers, base_num_decoder_layers is {t['base_num_decoder_layers']}")
  need(int(t["token_side_dim"]) >= 1, "token_side_dim must be positive")
  for i, lay in enumerate(t["layer_specs"]):
    m, kind, at = lay["mixer"], lay["type"], f"layer_specs[{i}]"
    need(kind in MIXERS, f"{at}: unknown mixer type {kind!r}")
    if kind == "attention":
      heads(at, m, 256)
      need(float(m["q_temp"]["every"]) > 0, f"{at}: q_temp.every must be positive")
      continue
    left, right = m["left"], m["right"]
    heads(at + ".left", left, 512)
    rotation(at + ".left", left)
    need(int(left["mask"]["size"]) >= 1, f"{at}.left: the mask must hold at least one token")
    need(max(right["dim"], right["vdim"]) <= 256, f"{at}.right: key and value widths up to 256 are supported")
    if kind == "parallel":
      rotation(at + ".right", right)
      need(len(right["decay"]) == right["heads"], f"{at}.right: one decay per head")
      need(all(0.0 < float(d) <= 1.0 for d in right["decay"]), f"{at}.right: decays lie in (0, 1]")
    else:
      heads(at + ".right", right, 256)
      need(1 <= right["conv"] <= 17, f"{at}.right: the convolution needs between one tap and 17")


def _mixer_plan(kind: str, m: dict) -> dict:
  """The part of a block's plan that its mixer decides."""
  from .transformer import BlockPlan
  if kind == "attention":
    return dict(attention="gqa", mixer=m, attn_bias=True, attn_out_bias=False, gated_attn=True, gate="head")
  if kind == "parallel":
    left = BlockPlan(attention="gqa", mixer=m["left"], mask="window", interleaved=True, qk_norm=True, global_qk_norm=True, attn_bias=True,
                     attn_out_bias=True, gated_attn=True)
    return dict(attention="parallel", mixer=m, pair=(left, BlockPlan(attention="retention", mixer=m["right"])), join=(0.5, 0.5, True))
  left = BlockPlan(attention="gqa", mixer=m["left"], mask="chunk", interleaved=True, qk_norm=True, attn_bias=True, attn_out_bias=False, gated_attn=True,
                   sink_value=0.0)
  return dict(attention="parallel", mixer=m, pair=(left, BlockPlan(attention="channel_delta", mixer=m["right"])),
              join=(float(m["left_scale"]), float(m["right_scale"]), False))


def layer_plans(c) -> list:
  from .transformer import BlockPlan, LayerPlan
  plans, stacks = [], {}
  for lay in c.layer_specs:
    kind, mlp = lay["type"], lay["mlp"]
    # layers of one type and one set of sizes are stacked together in the checkpoint tree
    sig = repr((kind, sorted(lay["mixer"].items(), key=str), mlp))
    if sig not in stacks:
      n = sum(1 for s in stacks.values() if s == f"{kind}_layers" or s.startswith(f"{kind}_layers_"))
      stacks[sig] = f"{kind}_layers" + (f"_{n}" if n else "")
    plans.append(LayerPlan(stacks[sig], [BlockPlan(
        attn_name="mixer", pre_attn_norm="pre_mixer_norm", pre_mlp_norm="pre_mlp_norm" if mlp is not None else None,
        mlp="dense" if mlp is not None else "none", mlp_hidden=int(mlp["ff"]) if mlp is not None else None, residual_fp32=True, layer_scale=True,
        token_side=int(c.token_side_dim), **_mixer_plan(kind, lay["mixer"]))]))
  return plans


# ------------------------------------------------------------------------------------------ weights
def _attention(get, m):
  for ours, theirs in (("query", "q"), ("key", "k"), ("value", "v")):
    yield ours + "/kernel", get(theirs)
    yield ours + "/bias", get(theirs + ".b")
  yield "gate/kernel", get("g")
  yield "out/kernel", get("o")


def _normed_attention(get, m):
  yield from _attention(get, m)
  yield "query_norm/scale", get("q.norm")
  yield "key_norm/scale", get("k.norm")


def _window(get, m):
  yield from _normed_attention(get, m)
  yield "out/bias", get("o.b")


def _differential(get, m):
  yield from _attention(get, m)
  for n in ("q1", "k1", "q2", "k2"):
    yield "lambda/" + n, get("l" + n)


def _retention(get, m):
  yield "in_proj/kernel", torch.cat([get("q"), get("k"), get("v"), get("g")], 0)
  yield "out_proj/kernel", get("o")


def _channel_delta(get, m):
  from ..layers.channel_delta import ChannelDeltaSizes
  s = ChannelDeltaSizes(int(m["kv_heads"]), int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), int(m["decay_rank"]), int(m["gate_rank"]))

  def rows(t, n):
    return torch.nn.functional.pad(t, (0, 0, 0, n - t.shape[0]))
  yield "in_proj/kernel", torch.cat([get("q"), get("k"), get("v")] + [rows(get(n), w) for n, w in zip(("b", "a1", "g1"), s.columns[1:])], 0)
  yield "conv1d/kernel", torch.cat([get("q.conv"), get("k.conv"), get("v.conv")], 0).t().contiguous()[:, None, :]
  yield "decay_proj/kernel", torch.nn.functional.pad(get("a2"), (0, s.columns[2] - s.decay_rank))
  yield "decay_proj/bias", get("dt_bias")
  yield "A_log", get("A_log")
  yield "gate_proj/kernel", torch.nn.functional.pad(get("g2"), (0, s.columns[3] - s.gate_rank))
  yield "norm/scale", get("norm")
  yield "out_proj/kernel", get("o")


def _mixer(kind, get, m):
  if kind == "attention":
    yield from _differential(get, m)
    return
  left, right = (_window, _retention) if kind == "parallel" else (_normed_attention, _channel_delta)
  for side, pack in (("left", left), ("right", right)):
    for leaf, value in pack(lambda n, side=side: get(f"{side}.{n}"), m[side]):
      yield f"{side}/{leaf}", value
    if kind == "parallel":
      yield f"{side}_norm/scale", get(f"{side}.out")


def tensors_for(store, c, get):
  """(parameter name, internal-layout value) for every parameter; `get(name)` reads one tensor of the folder in fp32."""
  yield "token_embedder/embedding", get("embed")
  yield "decoder/decoder_norm/scale", get("final.norm")
  dim, table = int(c.token_side_dim), get("side.embed")
  if table.shape[1] != dim * len(c.layer_specs):
    raise ValueError(f"side.embed: {table.shape[1]} columns, expected {dim} for each of {len(c.layer_specs)} layers")
  seen = {}
  for i, (lay, plan) in enumerate(zip(c.layer_specs, layer_plans(c))):
    n = seen.get(plan.stack, 0)
    seen[plan.stack] = n + 1
    pre = f"{plan.stack}_{n}/"
    yield pre + "pre_mixer_norm/scale", get(f"l{i}.norm1")
    yield pre + "layer_scale/mixer", get(f"l{i}.ls1")
    for leaf, value in _mixer(lay["type"], lambda n_, i=i: get(f"l{i}.mix.{n_}"), lay["mixer"]):
      yield pre + "mixer/" + leaf, value
    if lay["mlp"] is not None:
      yield pre + "pre_mlp_norm/scale", get(f"l{i}.norm2")
      yield pre + "layer_scale/mlp", get(f"l{i}.ls2")
      for ours, theirs in (("wi_0", "gate"), ("wi_1", "up"), ("wo", "down")):
        yield f"{pre}mlp/{ours}/kernel", get(f"l{i}.mlp.{theirs}")
    yield pre + "token_side/embedding", table[:, i * dim:(i + 1) * dim].contiguous()
    yield pre + "token_side/gate/kernel", get(f"l{i}.side.gate")
    yield pre + "token_side/proj/kernel", get(f"l{i}.side.proj")
    yield pre + "token_side/norm/scale", get(f"l{i}.side.norm")
