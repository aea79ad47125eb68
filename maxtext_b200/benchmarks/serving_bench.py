"""Serving throughput of the mixed-mixer models beside plain models of equal size, and the device time of every serving kernel.

`python bench.py --serving [--serving-models a,b] [--serving-lengths 512,2048] [--serving-slots 1,32]` prints one JSON line per model:

  prefill: tokens/s of one prompt per length (CUDA events around `MaxEngine.prefill`, median of the iterations)
  decode:  tokens/s of a full decode state per slot count, every slot holding `context` tokens, CUDA-graph replay
  kernels: device microseconds per launch by kernel (PyTorch profiler, a separate untimed pass), one prompt and one decode step

and one last line `rooflines`: every serving kernel at the layer sizes of silinex-1b, tipidra-1b, sitivik-1b and gukirax-1b (8192 prompt tokens; 128 sequences with 2048 cached tokens),
its time by CUDA events with L2 flushed, its algorithmic bytes or products, and the fraction of the measured copy bandwidth or GEMM rate,
beside the like operation of the models that existed before (`like`).

Weights are random; the work does not depend on their values. The models:

  silinex-1b   the catalog entry: gated delta, sliding-window latent attention and gated linear attention layers in turn
  mla-1b       the same width, depth and feed-forward size with the DeepSeek block (latent attention in every layer, gated MLP of equal size)
  llama-1b     the same with grouped-query attention
  silinex-5b, mla-5b   the same two at width 4096, 32 heads, 24 layers
  tipidra-1b   the catalog entry: capped attention and selective-scan layers in turn, every other pair with routed experts, two residual streams
  moe-1b       the same width, depth and active weights with the Mixtral block (grouped-query attention, routed experts in every layer)
  tipidra-5b, moe-5b   the same two at width 4096, 32 heads, 24 layers
  sitivik-1b   the catalog entry: windowed attention beside retention, chunked attention beside the channel-wise gated delta rule, differential attention
  sitivik-5b   the same at width 4096, 32 heads, 24 layers
  gukirax-1b   the catalog entry: heads that mix their scores, gated branches, dense and routed feed-forwards, 12 layers of which four run twice
  gukirax-5b   the same at width 4096, 32 heads, 18 layers of which six run twice
"""
from __future__ import annotations

import json
import os
import statistics

import torch

def _silinex(width, heads, ff, layers, q_rank):
  """Gated delta, latent attention (window 2048) and gated linear attention layers in turn, sized by `heads` of 128 lanes."""
  mlp = {"kind": "dense", "ff": ff}
  kinds = [
      {"type": "delta", "mixer": {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}, "mlp": mlp},
      {"type": "latent_attention", "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": q_rank, "kv_rank": 512, "scale": 192 ** -0.5,
                                             "mask": {"size": 2048}, "rot": {"base": 500000.0, "dims": 64}}, "mlp": mlp},
      {"type": "gla", "mixer": {"heads": heads, "dim": 64, "vdim": 128, "tau": 16.0, "decay_rank": 32}, "mlp": mlp}]
  return dict(decoder_block="silinex", base_emb_dim=width, base_num_decoder_layers=layers, layer_specs=[kinds[i % 3] for i in range(layers)],
              mlp_activations=["gelu_exact"], residual_multiplier=0.6, vocab_size=65536, logits_via_embedding=False)


def _plain(width, heads, ff, layers, q_rank=0):
  """The same width, depth and feed-forward weights (gated, so two thirds of the hidden width) with one attention kind in every layer."""
  keys = dict(base_emb_dim=width, base_num_query_heads=heads, base_num_decoder_layers=layers, base_mlp_dim=-(-2 * ff // 3 // 64) * 64, vocab_size=65536,
              logits_via_embedding=False)
  if q_rank:
    return dict(keys, decoder_block="deepseek", attention_type="mla", base_num_kv_heads=heads, first_num_dense_layers=layers, q_lora_rank=q_rank,
                kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128)
  return dict(keys, decoder_block="llama2", base_num_kv_heads=heads // 2, head_dim=128)


def _tipidra(width, heads, ff, expert_ff, layers):
  """Capped attention and selective scans (twice the width, 16 states) in turn; dense, routed, routed, dense feed-forwards in turn."""
  a = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "rot": {"base": 500000.0, "dims": 64}, "scale": 128 ** -0.5, "softcap": 40.0}
  s = {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}
  dense, routed = {"kind": "dense", "ff": ff}, {"kind": "moe", "router": {"experts": 16, "top": 2}, "expert": {"ff": expert_ff, "limit": 7.0}}
  kinds = [{"type": "attention", "mixer": a, "mlp": dense}, {"type": "mamba1", "mixer": s, "mlp": routed},
           {"type": "attention", "mixer": a, "mlp": routed}, {"type": "mamba1", "mixer": s, "mlp": dense}]
  return dict(decoder_block="tipidra", base_emb_dim=width, base_num_decoder_layers=layers, layer_specs=[kinds[i % 4] for i in range(layers)],
              mlp_activations=["gelu", "linear"], embedding_multiplier=width ** 0.5, mhc_expansion_rate=2, final_logits_soft_cap=30.0, vocab_size=65536,
              logits_via_embedding=False)


def _moe(width, heads, expert_ff, layers):
  return dict(decoder_block="mixtral", base_emb_dim=width, base_num_query_heads=heads, base_num_kv_heads=heads // 4, head_dim=128, base_mlp_dim=expert_ff,
              base_moe_mlp_dim=expert_ff, num_experts=16, num_experts_per_tok=2, base_num_decoder_layers=layers, vocab_size=65536, logits_via_embedding=False)


def _sitivik(width, heads, ff, layers):
  """Pairs (window 2048 beside retention, chunks of 2048 beside the channel-wise delta rule) and differential attention in turn."""
  rot = {"base": 500000.0, "dims": 128}
  left = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 2048}, "rot": rot}
  stretched = {**left, "rot": {**rot, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
  ret = {"heads": heads, "dim": 64, "vdim": 128, "rot": {"base": 10000.0, "dims": 64}, "decay": [1.0 - 2.0 ** (-5.0 - 5.0 * i / (heads - 1)) for i in range(heads)]}
  delta = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 128, "gate_rank": 128}
  diff = {"heads": heads, "kv_heads": heads // 4, "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.4, "q_temp": {"coef": 0.1, "every": 8192}}
  kinds = [("parallel", {"left": stretched, "right": ret}), ("attention", diff), ("parallel", {"left": stretched, "right": ret}),
           ("parallel_2", {"left": left, "right": delta, "left_scale": 0.7, "right_scale": 0.7})]
  return dict(decoder_block="sitivik", base_emb_dim=width, base_num_decoder_layers=layers, token_side_dim=64, vocab_size=65536, logits_via_embedding=True,
              normalize_embedding_logits=False, mlp_activations=["silu", "linear"], embedding_multiplier=width ** 0.5,
              layer_specs=[{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)])


def _gukirax(width, heads, ff, expert_ff, layers, loop):
  """Heads that mix their scores in every layer; the first and the last feed-forward dense, the others routed beside a shared expert."""
  a = {"heads": heads, "kv_heads": 4, "dim": 128, "vdim": 128, "rot": {"base": 500000.0, "dims": 64}, "scale": 128 ** -0.5}
  routed = {"kind": "moe", "router": {"experts": 16, "top": 2}, "expert": {"ff": expert_ff}, "shared": {"ff": expert_ff}}
  mlps = [{"kind": "dense", "ff": ff} if i in (0, layers - 1) else routed for i in range(layers)]
  return dict(decoder_block="gukirax", base_emb_dim=width, base_num_decoder_layers=layers, layer_loop=dict(zip(("start", "stop", "times"), loop)),
              layer_specs=[{"type": "attention", "mixer": a, "mlp": m} for m in mlps], mlp_activations=["xielu"], final_logits_scale=1.0,
              final_logits_soft_cap=30.0, vocab_size=65536, logits_via_embedding=True, normalize_embedding_logits=False)


MODELS = {
    "silinex-1b": dict(model_name="silinex-1b"),
    "mla-1b": _plain(2048, 16, 8192, 18, 768),
    "llama-1b": _plain(2048, 16, 8192, 18),
    "silinex-5b": _silinex(4096, 32, 16384, 24, 1536),
    "mla-5b": _plain(4096, 32, 16384, 24, 1536),
    "tipidra-1b": dict(model_name="tipidra-1b"),
    "moe-1b": _moe(2048, 16, 2560, 16),
    "tipidra-5b": _tipidra(4096, 32, 12288, 4096, 24),
    "moe-5b": _moe(4096, 32, 5120, 24),
    "sitivik-1b": dict(model_name="sitivik-1b"),
    "sitivik-5b": _sitivik(4096, 32, 9216, 24),
    "gukirax-1b": dict(model_name="gukirax-1b"),
    "gukirax-5b": _gukirax(4096, 32, 12288, 4096, 18, (6, 12, 2)),
}


def make_engine(name: str, max_len: int, slots: int = 1):
  from ..config import pyconfig
  from ..inference.maxengine import MaxEngine
  cfg = pyconfig.initialize(["serving", os.path.join(pyconfig.CONFIG_ROOT, "base.yml")], num_devices=1, max_target_length=max_len,
                            max_prefill_predict_length=max_len - 64, per_device_batch_size=slots, dtype="bfloat16", weight_dtype="bfloat16", hardware="gpu",
                            enable_checkpointing=False, log_config=False, cuda_graphs=True, decode_sampling_strategy="greedy", **MODELS[name])
  eng = MaxEngine(cfg, device=torch.device("cuda", torch.cuda.current_device()))
  eng.load_params()
  return eng


def _events(fn, iters: int, warmup: int = 3, drain: bool = True) -> float:
  """Median device milliseconds of fn over `iters` calls, L2 flushed in between. `drain` waits for the flush before fn is issued, so that
  the host's part of a multi-launch fn counts; without it a single kernel is queued behind the flush and timed alone."""
  flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device="cuda")
  for _ in range(warmup):
    fn()
  out = []
  for _ in range(iters):
    flush.zero_()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if drain:
      torch.cuda.synchronize()
    a.record()
    fn()
    b.record()
    torch.cuda.synchronize()
    out.append(a.elapsed_time(b))
  return statistics.median(out)


def filled_state(eng, slots: int, context: int):
  state = eng.init_decode_state(slots)
  for per_layer in state.caches:
    for c in per_layer:
      for n in ("latent", "k_rope", "k", "v"):
        t = getattr(c, n, None)
        if isinstance(t, torch.Tensor):
          t.normal_()
  state.next_pos.fill_(context)
  state.active.fill_(True)
  state.tokens.random_(1, 1000)
  return state


def kernel_times(fn) -> dict:
  from torch.profiler import ProfilerActivity, profile
  fn()
  torch.cuda.synchronize()
  with profile(activities=[ProfilerActivity.CUDA]) as prof:
    fn()
    torch.cuda.synchronize()
  out = {}
  for e in prof.key_averages():
    us = getattr(e, "device_time_total", 0.0) or getattr(e, "self_device_time_total", 0.0)
    if us > 0:
      out[e.key[:90]] = {"launches": e.count, "us": round(us / e.count, 2), "total_us": round(us, 1)}
  return dict(sorted(out.items(), key=lambda kv: -kv[1]["total_us"]))


def run(names, lengths, slot_counts, context: int, iters: int = 10, kernels: bool = True):
  rows = []
  for name in names:
    row = {"model": name, "dtype": "bf16", "data": "random weights and tokens", "context": context, "prefill": {}, "decode": {}, "kernels": {}}
    eng = make_engine(name, max(lengths + [context]) + 64)
    row["parameters"] = eng.model.store.num_parameters()
    for n in lengths:
      toks = torch.randint(1, 1000, (n,))
      ms = _events(lambda: eng.prefill(toks, n), iters)
      row["prefill"][n] = {"ms": round(ms, 3), "tokens_per_s": round(n / ms * 1e3)}
    if kernels:
      toks = torch.randint(1, 1000, (max(lengths),))
      row["kernels"]["prefill"] = kernel_times(lambda: eng.prefill(toks, max(lengths)))
    for s in slot_counts:
      state = filled_state(eng, s, context)
      ms = _events(lambda: eng.generate(state), iters)
      row["decode"][s] = {"ms": round(ms, 3), "tokens_per_s": round(s / ms * 1e3)}
      if kernels and s == max(slot_counts):
        row["kernels"]["decode"] = kernel_times(lambda: eng.generate(state))
      eng._graphs.clear()
      del state
      torch.cuda.empty_cache()
    rows.append(row)
    del eng
    import gc
    gc.collect()
    torch.cuda.empty_cache()
  return rows


def rooflines(iters: int = 10) -> dict:
  """name -> {us, bytes | flops, fraction of roofline, like}."""
  from ..layers.gdn import gated_delta_chunked, gated_delta_recurrent
  from ..ops import backend
  E = backend.ext(required=True)
  root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
  peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
  if os.path.isfile(os.path.join(root, "MEASURED_PEAKS.json")):
    with open(os.path.join(root, "MEASURED_PEAKS.json"), encoding="utf-8") as fh:
      peaks = {**json.load(fh), "source": "measured"}
  bf, dev = torch.bfloat16, "cuda"
  rows = {}

  def t(*shape, dtype=bf):
    return torch.randn(*shape, dtype=dtype, device=dev) if dtype.is_floating_point else torch.zeros(*shape, dtype=dtype, device=dev)

  def add(name, fn, nbytes=0, flops=0, like="", it=iters):
    us = _events(fn, it, 2, drain=False) * 1e3
    ideal = max(nbytes / (peaks["hbm_gbs"] * 1e3), flops / (peaks["bf16_tflops"] * 1e6))
    rows[name] = {"us": round(us, 1), "bytes": int(nbytes), "flops": int(flops), "fraction": round(ideal / us, 3), "like": like}

  def longs(n, v=0):
    return torch.full((n,), v, dtype=torch.long, device=dev)
  N, D, F_ = 8192, 2048, 8192
  hk, hv, dk, dv = 8, 16, 128, 128
  # ---- prompts
  x32, b, w, y = t(N, D, dtype=torch.float32), t(N, D), t(D), t(N, D)
  add("residual_norm", lambda: E.residual_norm(x32, b, w, 0.5, w, y, 1e-6, 1e-6, 1.0), 12 * N * D, like="rmsnorm")
  add("rmsnorm", lambda: E.rmsnorm_fwd(b, w, 1e-6, 0.0, y, None), 4 * N * D)
  h, h2 = t(N, F_), t(N, F_)
  add("act gelu_exact", lambda: E.act_fwd(h.view(-1), h2.view(-1), 4), 4 * N * F_, like="gated_act")
  add("gated_act", lambda: E.gated_act_fwd(h, h2.view(-1)[: N * F_ // 2].view(N, F_ // 2), 0), 3 * N * F_)
  cd, per = 2 * hk * dk + hv * dv, 2 * hk * dk + 2 * hv * dv
  qkvz, ba, cw, mixed, o = t(N, per), t(N, 2 * hv), t(4, cd), t(N, cd), t(N, hv * dv)
  conv, rec, one, A, nw = t(1, 3, cd, dtype=torch.float32), t(1, hv, dk, dv, dtype=torch.float32), longs(1), t(hv), t(dv)
  add("delta_conv", lambda: E.delta_conv(qkvz, cw, hk, hv, dk, dv, N, conv, one, one, None, mixed), 4 * N * cd, like="rmsnorm")
  add("delta_chunks (both kernels)", lambda: E.delta_chunks(mixed, ba, A, A, hk, hv, dk, dv, N, rec, one, one, None, o), 2 * N * (cd + hv * dv + 2 * hv),
      like="gated delta composition")
  q, k, v = (t(1, N, hv, d) for d in (dk, dk, dv))
  g, be = -torch.rand(1, N, hv, device=dev), torch.rand(1, N, hv, device=dev)
  add("gated delta composition", lambda: gated_delta_chunked(q, k, v, g, be, 64), 2 * N * (cd + hv * dv + 2 * hv), it=3)
  add("gated_head_norm", lambda: E.gated_head_norm(o, qkvz, hv, dv, 2, 512, 768, nw, 1e-6, y.view(-1)[: N * hv * dv].view(N, hv * dv)), 6 * N * hv * dv,
      like="rmsnorm")
  H, gk, rank = 16, 64, 32
  gx, la, dw, db = t(N, 2 * H * (gk + dv) + rank), -torch.rand(N, H * gk, device=dev) * 0.05, t(H * gk, rank), t(H * gk)
  rec2 = t(1, H, gk, dv, dtype=torch.float32)
  add("gla_decay", lambda: E.gla_decay(gx, 2 * H * (gk + dv), dw, db, 16.0, la), 2 * N * rank + 4 * N * H * gk, like="rmsnorm")
  la.uniform_(-0.05, 0.0)
  add("gla_chunks (both kernels)", lambda: E.gla_chunks(gx, la, H, gk, dv, N, rec2, one, one, None, o), N * (2 * 2 * H * (gk + dv) + 4 * H * gk),
      like="gated delta composition")
  nope, dr, vd, R, Q = 128, 64, 128, 512, 768
  inv, pos = torch.rand(dr // 2, device=dev), torch.arange(N, device=dev)
  qa, kva, qw, kw, cq, lat, kr = t(N, Q), t(N, R + dr), t(Q), t(R), t(N, Q), t(N, R), t(N, dr)
  c_lat, c_kr = t(1, N, R), t(1, N, dr)
  add("mla_prep", lambda: E.mla_prep(qa, qw, kva, kw, 1e-6, pos, inv, True, cq, lat, kr, c_lat, c_kr, one, one, None), 2 * N * (2 * Q + 3 * (R + dr)),
      like="rmsnorm")
  qh, kv = t(N, H, nope + dr), t(N, H, nope + vd)
  qp, kp, vp = t(N, H, 192), t(N, H, 192), t(N, H, 128)
  add("mla_pack (both kernels)", lambda: E.mla_pack(qh, kv, kr, pos, inv, True, nope, vd, qp, kp, vp), 2 * N * H * (2 * 192 + 256 + 192 + 128), like="rmsnorm")
  from ..ops import functional as F
  with torch.no_grad():
    win = 2048
    pairs = N * win - win * win // 2
    add("flash forward, window 2048", lambda: F.attention_fwd(qp[None], kp[None], vp[None], None, None, 0.1, 0.0, win), 0, 2 * pairs * H * (192 + 128),
        like="flash forward, causal")
    add("flash forward, causal", lambda: F.attention_fwd(qp[None], kp[None], vp[None], None, None, 0.1, 0.0, 0), 0, N * N * H * (192 + 128))
  # several residual streams, selective scan, capped attention with a gate, experts with scaled inputs
  xs, mix, wr = t(N, 2, D, dtype=torch.float32), t(2, 2) * 0.1, t(2)
  add("stream_mix, 2 streams", lambda: E.stream_mix(xs, b, None, 1, mix, wr, wr, w, w, y, 1e-5), N * D * (2 * 2 * 4 + 4), like="rmsnorm")
  C, NS, rk = 4096, 16, 128
  px, sx, sy, cw4, cb, q2 = t(N, 2 * C), t(N, C), t(N, C), t(4, C), t(C), t(N, rk + 2 * NS)
  hist, srec, sdt = t(1, 3, C, dtype=torch.float32), t(1, 1, C, NS, dtype=torch.float32), t(N, C, dtype=torch.float32)
  A16, D16 = torch.rand(C, NS, device=dev).to(bf), t(C)
  add("ssm_conv", lambda: E.ssm_conv(px, cw4, cb, N, hist, one, one, None, sx), 4 * N * C, like="delta_conv")
  add("ssm_scan", lambda: E.ssm_scan(sx, px, q2, sdt, cb, A16, D16, rk, NS, N, srec, one, one, None, sy), N * C * 10 + 4 * N * NS,
      like="gla_chunks (both kernels)")
  HQ, HG, hd = 16, 4, 128
  pk, qo, ko = t(N, (2 * HQ + 2 * HG) * hd), t(N, HQ, hd), t(N, HG, hd)
  ck, cv, inv64 = t(1, N, HG, hd), t(1, N, HG, hd), torch.rand(32, device=dev)
  qs, ks, vs, gs = torch.split(pk, [HQ * hd, HG * hd, HG * hd, HQ * hd], -1)
  pos0 = torch.arange(N, device=dev)
  add("qkv_prep", lambda: E.qkv_prep(qs, ks, vs, hd, hd, pos0, inv64, 64, 1e-5, qo, ko, None, ck, cv, one, one, None), 2 * N * hd * (2 * HQ + 5 * HG),
      like="rmsnorm")
  from ..ops import functional as F
  with torch.no_grad():
    vv = vs.as_strided((1, N, HG, hd), (N * vs.stride(0), vs.stride(0), hd, 1), vs.storage_offset())
    sink = torch.zeros(HQ, device=dev)
    qn, kn = qo[None] * 0.1, ko[None]
    add("flash forward, capped, sink", lambda: F.attention_fwd(qn, kn, vv, None, None, 0.09, 40.0, 0, sinks=sink, cap_mode=F.CAP_SMALL), 0, N * N * HQ * 2 * hd,
        like="flash forward, causal, 128")
    add("flash forward, capped by an exponential", lambda: F.attention_fwd(qn, kn, vv, None, None, 0.09, 40.0, 0, sinks=sink, cap_mode=F.CAP_EXACT), 0,
        N * N * HQ * 2 * hd, like="flash forward, causal, 128")
    add("flash forward, causal, 128", lambda: F.attention_fwd(qn, kn, vv, None, None, 0.09, 0.0, 0), 0, N * N * HQ * 2 * hd)
  go_ = t(N, HQ * hd)
  add("head_gate", lambda: E.head_gate(qo, gs, hd, go_), 6 * N * HQ * hd, like="rmsnorm")
  from ..ops import moe_ops
  nE, top, Fe = 16, 2, 2048
  P = lambda *s: type("P", (), {"data": t(*s)})()  # noqa: E731
  lay = type("L", (), dict(style="scaled_input", k=top, E=nE, limit=7.0, gate=P(nE, D), wi_0=P(nE, Fe, D), wi_1=P(nE, Fe, D), wo=P(nE, D, Fe)))()
  xin = t(N, D)
  idx, wts, _, _ = E.router_topk(F.mm(xin, lay.gate.data, False, True, out_dtype=torch.float32), None, top, 1, True, True, 1.0)
  with torch.no_grad():
    add("experts, scaled inputs (whole layer)", lambda: moe_ops.serve_scored(xin, lay), 0, 6 * N * top * D * Fe, like="experts, silu (whole layer)")
    add("experts, silu (whole layer)", lambda: moe_ops.moe_ffn_padded(xin, wts, idx, lay.wi_0, lay.wi_1, lay.wo, nE, "silu"), 0, 6 * N * top * D * Fe)
  plan = moe_ops.GroupPlan(idx, nE)
  gu, he = t(plan.rows_max, 2 * Fe), t(plan.rows_max, Fe)
  add("expert_act", lambda: E.expert_act(gu, wts.view(-1), plan.row_pair, plan.offs, 7.0, he), 6 * N * top * Fe, like="gated_act")
  # two mixers side by side, retention, channel-wise delta rule, differential attention
  b2 = t(N, D)
  add("residual_join, two normed branches", lambda: E.residual_join(x32, b, w, w, 0.5, b2, None, w, 0.5, w, w, y, 1e-6), N * D * (8 + 3 * 2), like="residual_norm")
  add("residual_join, one branch", lambda: E.residual_join(x32, b, None, None, 1.0, None, None, None, 1.0, w, w, y, 1e-6), N * D * (8 + 2 * 2), like="residual_norm")
  sg, stab, stok, so = t(N, 64), t(65536, 64), torch.randint(0, 65536, (N,), device=dev), t(N, 64)
  add("token_gate", lambda: E.token_gate(sg, stab, stok, so), 6 * N * 64, like="gated_act, small")
  add("gated_act, small", lambda: E.gated_act_fwd(so, sg.view(-1)[: N * 32].view(N, 32), 0), 3 * N * 64)
  qb, kb_, vb_, qnw, knw, inv128, vo = t(HQ * hd), t(HG * hd), t(HG * hd), t(HQ * hd), t(HG * hd), torch.rand(64, device=dev), t(N, HG, hd)
  add("qkv_prep, bias, norm over all heads, pairs", lambda: E.qkv_prep(qs, ks, vs, hd, hd, pos0, inv128, 128, 1e-5, qo, ko, vo, ck, cv, one, one, None, qb, kb_, vb_, qnw,
                                                                       knw, True, 1, 0.0, 0.0), 2 * N * hd * (2 * HQ + 6 * HG), like="qkv_prep")
  add("qkv_prep, bias, norm per head, pairs", lambda: E.qkv_prep(qs, ks, vs, hd, hd, pos0, inv128, 128, 1e-5, qo, ko, vo, ck, cv, one, one, None, qb, kb_, vb_, qnw[:hd],
                                                                 knw[:hd], True, 1, 0.0, 0.0), 2 * N * hd * (2 * HQ + 6 * HG), like="qkv_prep")
  q2o = t(N, 2 * HQ, hd)
  add("qkv_prep, two maps, temperature", lambda: E.qkv_prep(qs, ks, vs, 64, hd, pos0, None, 0, -1.0, q2o, ko, vo, ck, cv, one, one, None, qb, kb_, vb_, None, None, False, 2,
                                                            0.1, 8192.0), 2 * N * hd * (3 * HQ + 6 * HG), like="qkv_prep")
  with torch.no_grad():
    add("flash forward, window 2048, 128", lambda: F.attention_fwd(qn, kn, vo[None], None, None, 0.09, 0.0, win), 0, 2 * pairs * HQ * 2 * hd,
        like="flash forward, window 2048")
    cpairs = N * 2048 // 2
    add("flash forward, chunks of 2048, sink", lambda: F.attention_fwd(qn, kn, vo[None], None, None, 0.09, 0.0, 0, chunk=2048, sinks=sink), 0,
        2 * cpairs * HQ * 2 * hd, like="flash forward, window 2048")
    q2n = q2o[None] * 0.1
    add("flash forward, two maps of 64", lambda: F.attention_fwd(q2n, kn, vo[None], None, None, 0.12, 0.0, 0), 0, N * N * 2 * HQ * (64 + hd),
        like="flash forward, causal, 128")
  o2, lam = t(N, 2 * HQ, hd), [t(64) * 0.1 for _ in range(4)]
  gh = t(N, 64)
  add("diff_combine", lambda: E.diff_combine(o2, lam, 0.4, 1e-6, gh, hd, go_, True), 2 * N * hd * 3 * HQ, like="head_gate")
  rx, rrec, ro = t(N, 2 * H * (gk + dv)), t(1, H, gk, dv, dtype=torch.float32), t(N, H * dv)
  ld, rinv = torch.log(torch.rand(H, device=dev) * 0.05 + 0.95), torch.rand(gk // 2, device=dev)
  add("retention_chunks (both kernels)", lambda: E.retention_chunks(rx, ld, rinv, gk, H, gk, dv, N, rrec, one, one, None, ro), 2 * N * 2 * H * (gk + dv),
      like="gla_chunks (both kernels)")
  ccd = H * 3 * 128
  cmix, cbeta, cda, cA, cdt = t(N, ccd), t(N, H), t(N, H * 128, dtype=torch.float32), t(H) * 0.1 - 1.0, t(H * 128)
  crec, cconv, craw, ccw = t(1, H, 128, 128, dtype=torch.float32), t(1, 3, ccd, dtype=torch.float32), t(N, ccd + 512), t(4, ccd)
  add("channel_delta_scan, chunks (both kernels)", lambda: E.channel_delta_scan(cmix, cbeta, cda, cA, cdt, H, H, 128, 128, N, crec, one, one, None, ro, True),
      N * H * (2 * 4 * 128 + 4 * 128 + 2), like="delta_chunks (both kernels)")
  add("ssm_conv, no bias", lambda: E.ssm_conv(craw[:, :ccd], ccw, None, N, cconv, one, one, None, cmix), 4 * N * ccd, like="delta_conv")
  add("gated_head_norm, sigmoid", lambda: E.gated_head_norm(ro, go_, H, 128, 1, 0, 128, nw, 1e-6, o, True), 6 * N * H * 128, like="gated_head_norm")
  # heads that mix their scores, gated sandwich-normed branches, xIELU, ungated experts
  talk, pk2 = t(HQ, HQ) * 0.2, t(N, (HQ + HG) * hd + D)
  tq, tk, tg = torch.split(pk2, [HQ * hd, HG * hd, D], -1)
  qf, ow = t(N, HQ, HG * hd), t(N, HQ * hd)
  add("qkv_prep, mixing folded into the queries", lambda: E.qkv_prep(tq, tk, tk, hd, hd, pos0, inv64, 64, 1e-5, qf, ko, None, ck, cv, one, one, None, talk=talk),
      2 * N * hd * (HQ + HQ * HG + 4 * HG), like="qkv_prep")
  vr = tk.as_strided((1, N, HG, hd), (N * tk.stride(0), tk.stride(0), hd, 1), tk.storage_offset())
  qf4 = qf[None] * 0.1
  sinkh = t(HQ)
  add("wide_flash (mixed scores, sink)", lambda: E.wide_flash(qf4, ko[None], vr, ow, None, None, None, None, sinkh, 0.09, 0, 0, 0), 0, N * N * HQ * (2 * hd + HQ),
      like="flash forward, causal, 128")
  rows["wide_flash (mixed scores, sink)"]["products_issued"] = int(N * N * HQ * (HG * hd + hd))
  bd = t(D)
  add("residual_gate", lambda: E.residual_gate(x32, b, None, 1, None, tg, bd, w, w, y, 1e-6, True, False), N * D * (8 + 3 * 2), like="residual_norm")
  er, edest = t(2 * N + 2048, D), torch.randperm(2 * N + 2048, device=dev)[:2 * N].int()
  add("residual_gate, rows of two experts and a shared one", lambda: E.residual_gate(x32, er, edest, 2, b, tg, bd, w, w, y, 1e-6, True, False),
      N * D * (8 + 5 * 2), like="residual_norm")
  hx, ha, par = t(N, 6144 + D), t(N, 6144), t(2)
  add("act xielu", lambda: E.act_rows(hx[:, :6144], ha, 6, par), 4 * N * 6144, like="gated_act")
  add("act relu2", lambda: E.act_rows(hx[:, :2048], ha.view(-1)[: N * 2048].view(N, 2048), 5, None), 4 * N * 2048, like="gated_act")
  glay = type("L", (), dict(style="prob_weighted", k=top, E=nE, limit=0.0, gate=lay.gate, wi_0=lay.wi_0, wi_1=None, wo=lay.wo))()
  with torch.no_grad():
    add("experts, squared relu (whole layer)", lambda: moe_ops.serve_scored(xin, glay), 0, 4 * N * top * D * Fe, like="experts, silu (whole layer)")
  add("expert_act, squared relu", lambda: E.expert_act(he, wts.view(-1), plan.row_pair, plan.offs, 0.0, gu.view(-1)[: he.numel()].view(he.shape)), 4 * N * top * Fe,
      like="expert_act")
  cat, wl, xl = t(N, 2 * D), t(D, 2 * D), t(N, D, dtype=torch.float32)
  add("gemm, input of a pass (fp32 result)", lambda: F.mm(cat, wl, False, True, out=xl), 0, 4 * N * D * D, like="gemm, 8192 rows")
  add("gemm, 8192 rows", lambda: F.mm(cat, wl, False, True, out=y), 0, 4 * N * D * D)
  # ---- decoding: 128 sequences, 2048 cached tokens
  B, L = 128, 2048
  ids, lens = torch.arange(B, device=dev), longs(B, L - 1)
  dconv, drec, dout = t(B, 3, cd, dtype=torch.float32), t(B, hv, dk, dv, dtype=torch.float32), t(B, hv * dv)
  st = 8 * B * hv * dk * dv + 2 * B * (per + hv * dv) + 8 * B * 3 * cd
  add("delta_decode", lambda: E.delta_decode(qkvz[:B], ba[:B], cw, A, A, nw, 1e-6, hk, hv, dk, dv, dconv, drec, ids, lens, dout), st,
      like="gated delta step composition")
  q1, k1, v1 = (t(B, 1, hv, d) for d in (dk, dk, dv))
  g1, b1 = -torch.rand(B, 1, hv, device=dev), torch.rand(B, 1, hv, device=dev)
  add("gated delta step composition", lambda: gated_delta_recurrent(q1, k1, v1, g1, b1, drec), 8 * B * hv * dk * dv)
  grec = t(B, H, gk, dv, dtype=torch.float32)
  add("gla_decode", lambda: E.gla_decode(gx[:B], dw, db, nw, 1e-6, 16.0, H, gk, dv, grec, ids, lens, dout), 8 * B * H * gk * dv, like="gated delta step composition")
  lc, kc, qd = t(B, L, R), t(B, L, dr), t(B, H, R + dr)
  sp = E.mla_decode_splits(B, H, L)
  part, ml = t(B, H, sp, R, dtype=torch.float32), torch.rand(B, H, sp, 2, device=dev) + 0.1
  add("mla_decode_attn", lambda: E.mla_decode_attn(qd, lc, kc, ids, lens, 0.1, 2048, sp, part, ml), 2 * B * L * (R + dr), like="cached_decode, 128 sequences")
  wb, qin, vout = t(H * (nope + vd), R), t(B, H, nope + dr), t(B, H, vd)
  add("mla_absorb", lambda: E.mla_absorb(qin, wb, pos[:B], inv, True, nope, vd, qd), 2 * (H * nope * R + B * H * (nope + 2 * dr + R)), like="gemm, M = 128")
  add("mla_value_up", lambda: E.mla_value_up(part, ml, wb, nope, vout), 2 * H * vd * R + 4 * B * H * R + 2 * B * H * vd, like="gemm, M = 128")
  ga, gw, go = t(B, 2048), t(2048, 2048), t(B, 2048)
  add("gemm, M = 128", lambda: F.mm(ga, gw, False, True, out=go), 2 * (2048 * 2048 + 2 * B * 2048))
  for Bd in (1, 128):
    xd = xin[:Bd].contiguous()
    with torch.no_grad():
      idx, wts, _, _ = E.router_topk(F.mm(xd, lay.gate.data, False, True, out_dtype=torch.float32), None, top, 1, True, True, 1.0)
      plan = moe_ops.GroupPlan(idx, nE)
    hit = int((plan.sizes > 0).sum())
    hd_, yd = t(Bd * top, Fe), t(Bd * top, D)
    add(f"expert_up, {Bd} tokens", lambda: E.expert_up(xd, lay.wi_0.data, lay.wi_1.data, wts.view(-1), idx.view(-1), plan.sizes, plan.offs, plan.row_pair, top, 7.0,
                                                       hd_), 2 * hit * 2 * Fe * D, like=f"experts, silu (whole layer), {Bd} tokens")
    add(f"expert_down, {Bd} tokens", lambda: E.expert_down(hd_, lay.wo.data, idx.view(-1), plan.sizes, plan.offs, plan.row_pair, yd), 2 * hit * Fe * D,
        like=f"experts, silu (whole layer), {Bd} tokens")
    with torch.no_grad():
      add(f"experts, scaled inputs (whole layer), {Bd} tokens", lambda: moe_ops.serve_scored(xd, lay), 2 * hit * 3 * Fe * D,
          like=f"experts, silu (whole layer), {Bd} tokens")
      add(f"experts, silu (whole layer), {Bd} tokens", lambda: moe_ops.moe_ffn_padded(xd, wts, idx, lay.wi_0, lay.wi_1, lay.wo, nE, "silu"), 2 * hit * 3 * Fe * D)
  brec, bhist = t(B, 1, C, NS, dtype=torch.float32), t(B, 3, C, dtype=torch.float32)
  add("ssm_conv, 128 tokens", lambda: E.ssm_conv(px[:B], cw4, cb, 1, bhist, ids, lens, None, sx[:B]), B * C * (4 + 8 * 3), like="rmsnorm, 128 tokens")
  add("ssm_scan, 128 tokens", lambda: E.ssm_scan(sx[:B], px[:B], q2[:B], sdt[:B], cb, A16, D16, rk, NS, 1, brec, ids, lens, None, sy[:B]),
      B * C * (8 * NS + 10) + 2 * C * NS, like="gla_decode")
  kc4, vc4, q16, g16 = t(B, L, HG, hd), t(B, L, HG, hd), t(B, HQ, hd), t(B, HQ * hd)
  sinkb = t(HQ)
  for Bd in (1, 32, 128):
    sp = E.cached_decode_splits(Bd, HQ, HG, L)
    pt, ml2, od = t(Bd, HQ, sp, hd, dtype=torch.float32), t(Bd, HQ, sp, 2, dtype=torch.float32), t(Bd, HQ * hd)
    add(f"cached_decode, {Bd} sequences", lambda: E.cached_decode(q16[:Bd], kc4[:Bd], vc4[:Bd], ids[:Bd], lens[:Bd], 0.09, 40.0, 0, sinkb, g16[:Bd], sp, pt, ml2, od),
        2 * 2 * Bd * L * HG * hd, like="mla_decode_attn")
  q32, ghd = t(B, 2 * HQ, hd), t(B, HQ)
  for Bd in (1, 128):
    sp = E.cached_decode_splits(Bd, 2 * HQ, HG, L)
    pt, ml2, od = t(Bd, 2 * HQ, sp, hd, dtype=torch.float32), t(Bd, 2 * HQ, sp, 2, dtype=torch.float32), t(Bd, HQ * hd)
    add(f"cached_decode, two maps, {Bd} sequences", lambda: E.cached_decode(q32[:Bd], kc4[:Bd], vc4[:Bd], ids[:Bd], lens[:Bd], 0.12, 0.0, 0, None, ghd[:Bd], sp, pt, ml2,
                                                                           od, per_head=True, lam=lam, diff=0.4, eps=1e-6), 2 * 2 * Bd * L * HG * hd,
        like=f"cached_decode, {Bd} sequences")
  qw, sinkw = t(B, HQ, HG * hd) * 0.1, t(HQ)
  for Bd in (1, 32, 128):
    sp = E.cached_decode_splits(Bd, HQ, 1, L)
    pt, ml2, od = t(Bd, HQ, sp, hd, dtype=torch.float32), t(Bd, HQ, sp, 2, dtype=torch.float32), t(Bd, HQ * hd)
    add(f"wide_decode, {Bd} sequences", lambda: E.wide_decode(qw[:Bd], kc4[:Bd], vc4[:Bd], ids[:Bd], lens[:Bd], 0.09, 0, 0, sinkw, sp, pt, ml2, od),
        2 * 2 * Bd * L * HG * hd, like=f"cached_decode, {Bd} sequences")
  add("qkv_prep, mixing folded, 128 tokens", lambda: E.qkv_prep(tq[:B], tk[:B], tk[:B], hd, hd, lens, inv64, 64, 1e-5, qw, None, None, kc4, vc4, ids, lens, None,
                                                                talk=talk), 2 * B * hd * (HQ + HQ * HG + 3 * HG), like="rmsnorm, 128 tokens")
  add("residual_gate, 128 tokens", lambda: E.residual_gate(x32[:B], b[:B], None, 1, None, tg[:B], bd, w, w, y[:B], 1e-6, True, False), B * D * 14,
      like="rmsnorm, 128 tokens")
  add("act xielu, 128 tokens", lambda: E.act_rows(hx[:B, :6144], ha[:B], 6, par), 4 * B * 6144, like="rmsnorm, 128 tokens")
  for Bd in (1, 128):
    xd = xin[:Bd].contiguous()
    with torch.no_grad():
      gidx = E.router_topk(F.mm(xd, lay.gate.data, False, True, out_dtype=torch.float32), None, top, 1, False, True, 1.0)[0]
      hit = int((moe_ops.GroupPlan(gidx, nE).sizes > 0).sum())
      add(f"experts, squared relu (whole layer), {Bd} tokens", lambda: moe_ops.serve_scored(xd, glay), 2 * hit * 2 * Fe * D,
          like=f"experts, silu (whole layer), {Bd} tokens")
  brr = t(B, H, gk, dv, dtype=torch.float32)
  add("retention_decode", lambda: E.retention_decode(rx[:B], ld, rinv, gk, 1e-6, H, gk, dv, brr, ids, lens, dout), 8 * B * H * gk * dv, like="gla_decode")
  bcr, bcc = t(B, H, 128, 128, dtype=torch.float32), t(B, 3, ccd, dtype=torch.float32)
  add("channel_delta_decode", lambda: E.channel_delta_decode(craw[:B, :ccd], cbeta[:B], ccw, cda[:B], cA, cdt, go_[:B], nw, 1e-6, H, H, 128, 128, bcc, bcr, ids, lens,
                                                             dout), 8 * B * H * 128 * 128 + 8 * B * 3 * ccd, like="delta_decode")
  add("residual_join, 128 tokens", lambda: E.residual_join(x32[:B], b[:B], w, w, 0.5, b2[:B], None, w, 0.5, w, w, y[:B], 1e-6), B * D * 14,
      like="rmsnorm, 128 tokens")
  add("stream_mix, 128 tokens", lambda: E.stream_mix(xs[:B], b[:B], None, 1, mix, wr, wr, w, w, y[:B], 1e-5), B * D * (2 * 2 * 4 + 4), like="rmsnorm, 128 tokens")
  add("rmsnorm, 128 tokens", lambda: E.rmsnorm_fwd(b[:B], w, 1e-6, 0.0, y[:B], None), 4 * B * D)
  return {"rooflines": rows, "hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "peaks": peaks["source"]}


def main(models: str = "", lengths: str = "512,2048,8192", slots: str = "1,32,128", context: int = 2048, iters: int = 10) -> int:
  names = [m for m in models.split(",") if m] or list(MODELS)
  for row in run(names, [int(x) for x in lengths.split(",")], [int(x) for x in slots.split(",")], context, iters):
    print(json.dumps(row))
  print(json.dumps(rooflines(iters)))
  return 0
