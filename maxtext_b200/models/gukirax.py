"""Gukirax: a decoder whose heads mix their scores, with gated sandwich-normed branches and a stretch of layers that runs in a loop.

Every layer names its own sizes and feed-forward (`layer_specs`):

  attention   the values are the keys as projected; q and k are rotated and RMS-normalised per head; a matrix mixes the heads' scores in
              front of the softmax, whose denominator holds a learned sink per head
  dense       feed-forward with xIELU
  moe         experts with a squared relu, weighted by soft-max probabilities that are not renormalised, beside a shared expert

The residual stream is fp32. Each sublayer's result is gated lane by lane by a projection of what the sublayer reads, layer-normalised and added;
the embeddings are normalised as well, and the head is the embedding table. `layer_loop` runs a stretch of layers several times; every pass
begins with a projection of the stream beside the embedding output, and has caches of its own. The attention is `layers.blocks.Attention`,
the experts are `layers.moe.RoutedAndSharedMoE`, the stream is `models.transformer.DecoderBlock._call_gated_stream`. This file holds what is
particular to the design: how its config.json becomes configuration keys, its layer plans, and how its tensors map to parameters.
"""
from __future__ import annotations

import torch

MLPS = ("dense", "moe")


# ------------------------------------------------------------------------------------------ configuration
def keys_from_json(spec: dict, shapes: dict) -> dict:
  layers = []
  for i, lay in enumerate(spec["layers"]):
    if lay["type"] != "attention":
      raise ValueError(f"layer {i}: unknown mixer type {lay['type']!r} (known: attention)")
    mlp = lay.get("mlp")
    if mlp is not None and mlp.get("kind") not in MLPS:
      raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r} (known: {list(MLPS)})")
    layers.append({"type": "attention", "mixer": dict(lay["mixer"]), "mlp": dict(mlp) if mlp is not None else None})
  loop = spec.get("loop")
  return {"decoder_block": "gukirax", "layer_specs": layers, "layer_loop": dict(loop) if loop else {}, "base_emb_dim": int(spec["width"]),
          "vocab_size": int(spec["vocab"]), "base_num_decoder_layers": len(layers), "normalization_layer_epsilon": float(spec["norm"]["eps"]),
          "final_logits_scale": float(spec["logit_scale"]), "final_logits_soft_cap": float(spec["logit_softcap"]), "mlp_activations": ["xielu"],
          "logits_via_embedding": True, "normalize_embedding_logits": False}


def validate(t: dict) -> None:
  """Cross-field checks of the layer list (run with the other validators when a configuration is built)."""
  def need(ok, why):
    if not ok:
      raise ValueError(why)
  n = len(t["layer_specs"])
  need(n == int(t["base_num_decoder_layers"]), f"layer_specs names {n} layers, base_num_decoder_layers is {t['base_num_decoder_layers']}")
  need(int(t["base_emb_dim"]) <= 8192, "base_emb_dim: widths above 8192 are not supported")
  loop = t["layer_loop"]
  if loop:
    need(0 <= loop["start"] < loop["stop"] <= n and loop["times"] >= 1, f"layer_loop: a non-empty stretch of the {n} layers, run at least once")
    need(max(int(t.get("ici_pipeline_parallelism") or 1), int(t.get("dcn_pipeline_parallelism") or 1)) == 1, "layer_loop: not split over pipeline stages")
  for i, lay in enumerate(t["layer_specs"]):
    m, mlp, at = lay["mixer"], lay["mlp"], f"layer_specs[{i}]"
    need(lay["type"] == "attention", f"{at}: unknown mixer type {lay['type']!r}")
    need(m["heads"] % m["kv_heads"] == 0, f"{at}: heads must be a multiple of kv_heads")
    need(m["dim"] == m["vdim"], f"{at}: the values are the keys, so dim and vdim must agree")
    need(m["rot"]["dims"] % 2 == 0 and 0 <= m["rot"]["dims"] <= m["dim"], f"{at}: rot.dims must be even and at most dim")
    need(m["dim"] <= 512, f"{at}: head widths above 512 are not supported")
    if mlp is not None and mlp["kind"] == "moe":
      r = mlp["router"]
      need(1 <= r["top"] <= r["experts"], f"{at}: router.top must lie between 1 and router.experts")
      need(r["experts"] <= 512 and r["top"] <= 32, f"{at}: at most 512 experts and 32 of them per token are supported")


def layer_plans(c) -> list:
  from .transformer import BlockPlan, LayerPlan
  plans, stacks = [], {}
  for i, lay in enumerate(c.layer_specs):
    mlp, opens = lay["mlp"], bool(c.layer_loop) and i == int(c.layer_loop["start"])
    # layers of one kind and one set of sizes are stacked together in the checkpoint tree
    sig = repr((opens, sorted(lay["mixer"].items(), key=str), mlp))
    if sig not in stacks:
      stacks[sig] = "attention_layers" + (f"_{len(stacks)}" if stacks else "")
    routed = mlp is not None and mlp["kind"] == "moe"
    plans.append(LayerPlan(stacks[sig], [BlockPlan(
        attention="gqa", mixer=lay["mixer"], attn_name="mixer", pre_attn_norm="pre_mixer_norm", post_attn_norm="post_mixer_norm",
        pre_mlp_norm="pre_mlp_norm" if mlp is not None else None, post_mlp_norm="post_mlp_norm" if mlp is not None else None,
        norm_kind="layernorm_scale", residual_fp32=True, residual_gate=True, share_kv=True, l2_qk_norm=True, sinks=True, talk=True,
        mlp="none" if mlp is None else "moe_shared" if routed else "dense", mlp_hidden=int(mlp["ff"]) if mlp is not None and not routed else None,
        moe=mlp if routed else None, moe_style="prob_weighted" if routed else "")], pass_input=opens))
  return plans


# ------------------------------------------------------------------------------------------ weights
def _attention(get):
  for ours, theirs in (("query", "q"), ("key", "k"), ("out", "o"), ("talk", "talk")):
    yield ours + "/kernel", get(theirs)
  yield "sinks", get("sink")


def _feed_forward(get, mlp):
  if mlp["kind"] == "dense":
    yield "wi/kernel", get("up")
    yield "wo/kernel", get("down")
    yield "act", get("act")
    return
  yield "routed_experts/gate/kernel", get("router")
  for ours, theirs in (("wi_0", "up"), ("wo", "down")):
    yield "routed_experts/" + ours, torch.stack([get(f"e{e}.{theirs}") for e in range(int(mlp["router"]["experts"]))])
  if mlp.get("shared") is not None:
    yield "shared_expert/wi/kernel", get("shared.up")
    yield "shared_expert/wo/kernel", get("shared.down")


def tensors_for(store, c, get):
  """(parameter name, internal-layout value) for every parameter; `get(name)` reads one tensor of the folder in fp32."""
  yield "token_embedder/embedding", get("embed")
  yield "decoder/embedding_norm/scale", get("embed.norm")
  yield "decoder/decoder_norm/scale", get("final.norm")
  seen = {}
  for i, (lay, plan) in enumerate(zip(c.layer_specs, layer_plans(c))):
    n = seen.get(plan.stack, 0)
    seen[plan.stack] = n + 1
    pre, mlp = f"{plan.stack}_{n}/", lay["mlp"]
    if plan.pass_input:
      yield pre + "pass_input/kernel", get("loop.in")
    for q, sub in ((1, "mixer"), (2, "mlp")):
      if q == 2 and mlp is None:
        continue
      yield f"{pre}pre_{sub}_norm/scale", get(f"l{i}.norm{q}")
      yield f"{pre}post_{sub}_norm/scale", get(f"l{i}.norm{q}b")
      yield f"{pre}residual_gate/{sub}/kernel", get(f"l{i}.rg{q}")
      yield f"{pre}residual_gate/{sub}/bias", get(f"l{i}.rg{q}.b")
    for leaf, value in _attention(lambda n_, i=i: get(f"l{i}.mix.{n_}")):
      yield pre + "mixer/" + leaf, value
    if mlp is not None:
      for leaf, value in _feed_forward(lambda n_, i=i: get(f"l{i}.mlp.{n_}"), mlp):
        yield pre + "mlp/" + leaf, value
