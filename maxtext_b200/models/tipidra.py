"""Tipidra: a decoder whose layers mix capped softmax attention with a sink and selective scans, over several residual streams.

Every layer names its own mixer, sizes and feed-forward (`layer_specs`). The residual stream is `streams` fp32 copies of the model
width; around every sublayer a static hyper-connection (`layers.mhc.StaticHyperConnection`) forms the sublayer's input from the copies,
mixes the copies among themselves and adds the output to each of them with its own weight. Norms are layer norms with a bias.

The attention layers are `layers.blocks.Attention` with per-layer sizes (rotation of the first lanes, then a scale-free RMS norm of q
and k, capped scores, a sink, a separate output gate), the recurrent layers `layers.ssm.SelectiveScan`, the routed feed-forwards
`layers.moe.RoutedMoE` in its scaled-input form. This file holds what is particular to the design: how its config.json becomes
configuration keys, its layer plans, and how its tensors map to parameters.
"""
from __future__ import annotations

import torch

MIXERS = {"attention": "gqa", "mamba1": "ssm"}
MLPS = ("dense", "moe")


# ------------------------------------------------------------------------------------------ configuration
def keys_from_json(spec: dict, shapes: dict) -> dict:
  layers = []
  for i, lay in enumerate(spec["layers"]):
    kind = lay["type"]
    if kind not in MIXERS:
      raise ValueError(f"layer {i}: unknown mixer type {kind!r} (known: {sorted(MIXERS)})")
    mlp = lay.get("mlp")
    if mlp is not None and mlp.get("kind") not in MLPS:
      raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r} (known: {list(MLPS)})")
    layers.append({"type": kind, "mixer": dict(lay["mixer"]), "mlp": dict(mlp) if mlp is not None else None})
  return {"decoder_block": "tipidra", "layer_specs": layers, "base_emb_dim": int(spec["width"]), "vocab_size": int(spec["vocab"]),
          "base_num_decoder_layers": len(layers), "normalization_layer_epsilon": float(spec["norm"]["eps"]),
          "embedding_multiplier": float(spec["embedding"]["scale"]), "mhc_expansion_rate": int(spec["streams"]),
          "final_logits_soft_cap": float(spec["logit_softcap"]), "mlp_activations": ["gelu", "linear"], "logits_via_embedding": False}


def validate(t: dict) -> None:
  """Cross-field checks of the layer list (run with the other validators when a configuration is built)."""
  def need(ok, why):
    if not ok:
      raise ValueError(why)
  need(len(t["layer_specs"]) == int(t["base_num_decoder_layers"]),
       f"layer_specs names {len(t['layer_specs'])} layers, base_num_decoder_layers is {t['base_num_decoder_layers']}")
  need(1 <= int(t["mhc_expansion_rate"]) <= 16, "mhc_expansion_rate: between 1 and 16 residual streams are supported")
  for i, lay in enumerate(t["layer_specs"]):
    m, kind, mlp = lay["mixer"], lay["type"], lay["mlp"]
    need(kind in MIXERS, f"layer_specs[{i}]: unknown mixer type {kind!r}")
    if kind == "attention":
      need(m["heads"] % m["kv_heads"] == 0, f"layer_specs[{i}]: heads must be a multiple of kv_heads")
      need(m["rot"]["dims"] % 2 == 0 and 0 <= m["rot"]["dims"] <= m["dim"], f"layer_specs[{i}]: rot.dims must be even and at most dim")
      need(m["softcap"] > 0, f"layer_specs[{i}]: softcap must be positive")
      need(max(m["dim"], m["vdim"]) <= 512, f"layer_specs[{i}]: head widths above 512 are not supported")
    else:
      need(1 <= m["conv"] <= 17, f"layer_specs[{i}]: the convolution needs between one tap and 17")
      need(1 <= m["state"] <= 256 and m["dt_rank"] >= 1, f"layer_specs[{i}]: state (up to 256) and dt_rank must be positive")
    if mlp is not None and mlp["kind"] == "moe":
      r = mlp["router"]
      need(1 <= r["top"] <= r["experts"], f"layer_specs[{i}]: router.top must lie between 1 and router.experts")
      need(r["experts"] <= 512 and r["top"] <= 32, f"layer_specs[{i}]: at most 512 experts and 32 of them per token are supported")
      need(mlp["expert"]["limit"] > 0, f"layer_specs[{i}]: expert.limit must be positive")


def layer_plans(c) -> list:
  from .transformer import BlockPlan, LayerPlan
  plans, stacks = [], {}
  for lay in c.layer_specs:
    kind, mlp = lay["type"], lay["mlp"]
    # layers of one type and one set of sizes are stacked together in the checkpoint tree
    sig = repr((kind, sorted(lay["mixer"].items(), key=str), mlp))
    if sig not in stacks:
      n = sum(1 for s in stacks.values() if s.startswith(f"{kind}_layers"))
      stacks[sig] = f"{kind}_layers" + (f"_{n}" if n else "")
    routed = mlp is not None and mlp["kind"] == "moe"
    plans.append(LayerPlan(stacks[sig], [BlockPlan(
        attention=MIXERS[kind], mixer=lay["mixer"], attn_name="mixer", pre_attn_norm="pre_mixer_norm",
        pre_mlp_norm="pre_mlp_norm" if mlp is not None else None, norm_kind="layernorm", hyper="static",
        mlp="none" if mlp is None else "moe" if routed else "dense", mlp_hidden=int(mlp["ff"]) if mlp is not None and not routed else None,
        moe=mlp if routed else None, moe_style="scaled_input" if routed else "", l2_qk_norm=kind == "attention", sinks=kind == "attention",
        gated_attn=kind == "attention")]))
  return plans


# ------------------------------------------------------------------------------------------ weights
def _attention(get, m):
  for ours, theirs in (("query", "q"), ("key", "k"), ("value", "v"), ("gate", "g"), ("out", "o")):
    yield ours + "/kernel", get(theirs)
  yield "sinks", get("sink")


def _scan(get, m):
  from ..layers.ssm import ScanSizes
  s = ScanSizes(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
  x = get("x")
  if tuple(x.shape) != (s.rank + 2 * s.state, s.inner):
    raise ValueError(f"mix.x: tensor of shape {tuple(x.shape)}, expected {(s.rank + 2 * s.state, s.inner)}")
  rows = torch.zeros(s.proj_rows, s.inner)
  rows[:s.rank] = x[:s.rank]
  rows[s.rank_padded:s.rank_padded + 2 * s.state] = x[s.rank:]
  yield "in_proj/kernel", get("in")
  yield "conv1d/kernel", get("conv").t().contiguous()[:, None, :]
  yield "conv1d/bias", get("conv.b")
  yield "x_proj/kernel", rows
  yield "dt_proj/kernel", torch.nn.functional.pad(get("dt"), (0, s.rank_padded - s.rank))
  yield "dt_proj/bias", get("dt.b")
  yield "A_log", get("A_log")
  yield "D", get("D")
  yield "out_proj/kernel", get("o")


_PACK = {"attention": _attention, "mamba1": _scan}


def _feed_forward(get, mlp):
  if mlp["kind"] == "dense":
    for ours, theirs in (("wi_0", "gate"), ("wi_1", "up"), ("wo", "down")):
      yield ours + "/kernel", get(theirs)
    return
  yield "gate/kernel", get("router")
  for ours, theirs in (("wi_0", "gate"), ("wi_1", "up"), ("wo", "down")):
    yield ours, torch.stack([get(f"e{e}.{theirs}") for e in range(int(mlp["router"]["experts"]))])


def tensors_for(store, c, get):
  """(parameter name, internal-layout value) for every parameter; `get(name)` reads one tensor of the folder in fp32."""
  yield "token_embedder/embedding", get("embed")
  yield "decoder/decoder_norm/scale", get("final.norm")
  yield "decoder/decoder_norm/bias", get("final.norm.b")
  yield "decoder/logits_dense/kernel", get("head")
  seen = {}
  for i, (lay, plan) in enumerate(zip(c.layer_specs, layer_plans(c))):
    n = seen.get(plan.stack, 0)
    seen[plan.stack] = n + 1
    pre, mlp = f"{plan.stack}_{n}/", lay["mlp"]
    for q, (norm, conn) in ((1, ("pre_mixer_norm", "mixer_streams")), (2, ("pre_mlp_norm", "mlp_streams"))):
      if q == 2 and mlp is None:
        continue
      yield pre + norm + "/scale", get(f"l{i}.norm{q}")
      yield pre + norm + "/bias", get(f"l{i}.norm{q}.b")
      for leaf in ("in", "mix", "out"):
        yield f"{pre}{conn}/{leaf}", get(f"l{i}.hc{q}.{leaf}")
    for leaf, value in _PACK[lay["type"]](lambda n_, i=i: get(f"l{i}.mix.{n_}"), lay["mixer"]):
      yield pre + "mixer/" + leaf, value
    if mlp is not None:
      for leaf, value in _feed_forward(lambda n_, i=i: get(f"l{i}.mlp.{n_}"), mlp):
        yield pre + "mlp/" + leaf, value
