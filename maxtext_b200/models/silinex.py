"""Silinex: a decoder whose layers mix gated delta networks, gated linear attention and sliding-window latent attention.

Every layer names its own mixer, sizes and feed-forward (`layer_specs`). The residual stream is kept in fp32; each sublayer is
normalised before it reads the stream and again before its output, times a constant, joins it:

  x <- x + m * norm1b(mixer(norm1(x)));   x <- x + m * norm2b(mlp(norm2(x)))

with zero-centred RMS scales, an ungated exact-GELU feed-forward and a separate output head. The gated delta layers are
`layers.gdn.GatedDeltaNet` and the latent-attention layers `layers.blocks.MLA` (a window and an explicit score scale added) with
per-layer sizes; gated linear attention is `layers.gla`. This file holds what is particular to the design: how its config.json
becomes configuration keys, its layer plans, and how its tensors map to parameters.
"""
from __future__ import annotations

import torch

MIXERS = {"delta": "gdn", "gla": "gla", "latent_attention": "mla"}


# ------------------------------------------------------------------------------------------ configuration
def keys_from_json(spec: dict, shapes: dict) -> dict:
  layers = []
  for i, lay in enumerate(spec["layers"]):
    kind, mixer = lay["type"], dict(lay["mixer"])
    if kind not in MIXERS:
      raise ValueError(f"layer {i}: unknown mixer type {kind!r} (known: {sorted(MIXERS)})")
    mlp = lay.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
      raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    if kind == "gla":
      mixer["decay_rank"] = int(shapes[f"l{i}.mix.a1"][0])       # the rank of the decay projection is given by its tensor only
    layers.append({"type": kind, "mixer": mixer, "mlp": dict(mlp) if mlp is not None else None})
  return {"decoder_block": "silinex", "layer_specs": layers, "base_emb_dim": int(spec["width"]), "vocab_size": int(spec["vocab"]),
          "base_num_decoder_layers": len(layers), "normalization_layer_epsilon": float(spec["norm"]["eps"]),
          "residual_multiplier": float(spec["residual_mult"]), "mlp_activations": ["gelu_exact"], "logits_via_embedding": False}


def validate(t: dict) -> None:
  """Cross-field checks of the layer list (run with the other validators when a configuration is built)."""
  def need(ok, why):
    if not ok:
      raise ValueError(why)
  need(len(t["layer_specs"]) == int(t["base_num_decoder_layers"]),
       f"layer_specs names {len(t['layer_specs'])} layers, base_num_decoder_layers is {t['base_num_decoder_layers']}")
  for i, lay in enumerate(t["layer_specs"]):
    m, kind = lay["mixer"], lay["type"]
    need(kind in MIXERS, f"layer_specs[{i}]: unknown mixer type {kind!r}")
    if kind == "delta":
      need(m["heads"] % m["kv_heads"] == 0, f"layer_specs[{i}]: heads must be a multiple of kv_heads")
      need(m["conv"] >= 1, f"layer_specs[{i}]: the convolution needs at least one tap")
    if kind == "latent_attention":
      need(m["rot"]["dims"] == m["rot_dim"], f"layer_specs[{i}]: rot.dims must equal rot_dim")
      need(m["rot_dim"] % 2 == 0, f"layer_specs[{i}]: rot_dim must be even")
      need(int(m["mask"]["size"]) >= 1, f"layer_specs[{i}]: the window must hold at least one token")


def layer_plans(c) -> list:
  from .transformer import BlockPlan, LayerPlan
  plans, stacks = [], {}
  for lay in c.layer_specs:
    kind = lay["type"]
    # layers of one type and one set of sizes are stacked together in the checkpoint tree
    sig = repr((kind, sorted(lay["mixer"].items(), key=str), lay["mlp"]))
    if sig not in stacks:
      n = sum(1 for s in stacks.values() if s.startswith(f"{kind}_layers"))
      stacks[sig] = f"{kind}_layers" + (f"_{n}" if n else "")
    dense = lay["mlp"] is not None
    plans.append(LayerPlan(stacks[sig], [BlockPlan(
        attention=MIXERS[kind], mixer=lay["mixer"], attn_name="mixer", pre_attn_norm="pre_mixer_norm", post_attn_norm="post_mixer_norm",
        pre_mlp_norm="pre_mlp_norm" if dense else None, post_mlp_norm="post_mlp_norm" if dense else None, norm_offset=1.0,
        mlp="dense" if dense else "none", mlp_hidden=int(lay["mlp"]["ff"]) if dense else None,
        residual_fp32=True, residual_mult=float(c.residual_multiplier))]))
  return plans


# ------------------------------------------------------------------------------------------ weights
def _delta(get, m):
  """Rows of the packed projections, per key head: [q | k | v of its value heads | gate of its value heads] and [b | a]."""
  hk, hv, dk, dv = int(m["kv_heads"]), int(m["heads"]), int(m["dim"]), int(m["vdim"])
  r = hv // hk
  q, k = get("q").view(hk, dk, -1), get("k").view(hk, dk, -1)
  v, z = get("v").view(hk, r * dv, -1), get("g").view(hk, r * dv, -1)
  b, a = get("b").view(hk, r, -1), get("a").view(hk, r, -1)
  taps = torch.cat([get("q.conv"), get("k.conv"), get("v.conv")], 0)                # [channels, taps]
  yield "in_proj_qkvz/kernel", torch.cat([q, k, v, z], 1).flatten(0, 1)
  yield "in_proj_ba/kernel", torch.cat([b, a], 1).flatten(0, 1)
  yield "conv1d/kernel", taps.t().contiguous()[:, None, :]
  yield "A_log", get("A_log")
  yield "dt_bias", get("dt_bias")
  yield "norm/rms_norm/scale", get("norm")
  yield "out_proj/kernel", get("o")


def _gla(get, m):
  from ..layers.gla import padded_rank
  a1, a2 = get("a1"), get("a2")
  pad = padded_rank(a1.shape[0]) - a1.shape[0]
  rows = [get("q"), get("k"), get("v"), get("g"), torch.nn.functional.pad(a1, (0, 0, 0, pad))]
  yield "in_proj/kernel", torch.cat(rows, 0)
  yield "decay_proj/kernel", torch.nn.functional.pad(a2, (0, pad))
  yield "decay_proj/bias", get("a2.b")
  yield "norm/scale", get("norm")
  yield "out_proj/kernel", get("o")


def _latent(get, m):
  h, nope, vd = int(m["heads"]), int(m["dim"]), int(m["vdim"])
  uk, uv = get("uk").view(h, nope, -1), get("uv").view(h, vd, -1)
  yield "wq_a/kernel", get("dq")
  yield "q_norm/scale", get("dq.norm")
  yield "wq_b/kernel", get("uq")
  yield "wkv_a/kernel", get("dkv")
  yield "kv_norm/scale", get("dkv.norm")
  yield "wkv_b/kernel", torch.cat([uk, uv], 1).flatten(0, 1)
  yield "out/kernel", get("o")


_PACK = {"delta": _delta, "gla": _gla, "latent_attention": _latent}


def tensors_for(store, c, get):
  """(parameter name, internal-layout value) for every parameter; `get(name)` reads one tensor of the folder in fp32."""
  yield "token_embedder/embedding", get("embed")
  yield "decoder/decoder_norm/scale", get("final.norm")
  yield "decoder/logits_dense/kernel", get("head")
  seen = {}
  for i, (lay, plan) in enumerate(zip(c.layer_specs, layer_plans(c))):
    n = seen.get(plan.stack, 0)
    seen[plan.stack] = n + 1
    pre = f"{plan.stack}_{n}/"
    for ours, theirs in (("pre_mixer_norm", "norm1"), ("post_mixer_norm", "norm1b"), ("pre_mlp_norm", "norm2"), ("post_mlp_norm", "norm2b")):
      if lay["mlp"] is None and "mlp" in ours:
        continue
      yield pre + ours + "/scale", get(f"l{i}.{theirs}")
    for leaf, value in _PACK[lay["type"]](lambda n_, i=i: get(f"l{i}.mix.{n_}"), lay["mixer"]):
      yield pre + "mixer/" + leaf, value
    if lay["mlp"] is not None:
      yield pre + "mlp/wi/kernel", get(f"l{i}.mlp.up")
      yield pre + "mlp/wo/kernel", get(f"l{i}.mlp.down")
