"""Serving throughput of a mixed-mixer model beside plain models of equal size, and the device time of every serving kernel.

`python bench.py --serving [--serving-models a,b] [--serving-lengths 512,2048] [--serving-slots 1,32]` prints one JSON line per model:

  prefill: tokens/s of one prompt per length (CUDA events around `MaxEngine.prefill`, median of the iterations)
  decode:  tokens/s of a full decode state per slot count, every slot holding `context` tokens, CUDA-graph replay
  kernels: device microseconds per launch by kernel (PyTorch profiler, a separate untimed pass), one prompt and one decode step

Weights are random; the work does not depend on their values. The models:

  silinex-1b   the catalog entry: gated delta, sliding-window latent attention and gated linear attention layers in turn
  mla-1b       the same width, depth and feed-forward size with the DeepSeek block (latent attention in every layer, gated MLP of equal size)
  llama-1b     the same with grouped-query attention
"""
from __future__ import annotations

import json
import os
import statistics

import torch

MODELS = {
    "silinex-1b": ["model_name=silinex-1b"],
    "mla-1b": ["decoder_block=deepseek", "attention_type=mla", "base_emb_dim=2048", "base_num_query_heads=16", "base_num_kv_heads=16", "first_num_dense_layers=18",
               "base_num_decoder_layers=18", "base_mlp_dim=5461", "q_lora_rank=768", "kv_lora_rank=512", "qk_nope_head_dim=128",
               "qk_rope_head_dim=64", "v_head_dim=128", "vocab_size=65536", "logits_via_embedding=false"],
    "llama-1b": ["decoder_block=llama2", "base_emb_dim=2048", "base_num_query_heads=16", "base_num_kv_heads=8", "head_dim=128",
                 "base_num_decoder_layers=18", "base_mlp_dim=5461", "vocab_size=65536", "logits_via_embedding=false"],
}


def make_engine(name: str, max_len: int, slots: int = 1):
  from ..config import pyconfig
  from ..inference.maxengine import MaxEngine
  over = [o if not o.startswith("base_mlp_dim=") else f"base_mlp_dim={-(-int(o.split('=')[1]) // 64) * 64}" for o in MODELS[name]]
  cfg = pyconfig.initialize(["serving", os.path.join(pyconfig.CONFIG_ROOT, "base.yml")] + over +
                            [f"max_target_length={max_len}", f"max_prefill_predict_length={max_len - 64}", f"per_device_batch_size={slots}", "dtype=bfloat16",
                             "weight_dtype=bfloat16", "hardware=gpu", "enable_checkpointing=false", "log_config=false", "cuda_graphs=true",
                             "decode_sampling_strategy=greedy"], num_devices=1)
  eng = MaxEngine(cfg, device=torch.device("cuda", torch.cuda.current_device()))
  eng.load_params()
  return eng


def _events(fn, iters: int, warmup: int = 3) -> float:
  """Median device milliseconds of fn over `iters` calls, L2 flushed in between."""
  flush = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device="cuda")
  for _ in range(warmup):
    fn()
  out = []
  for _ in range(iters):
    flush.zero_()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
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


def main(models: str = "", lengths: str = "512,2048,8192", slots: str = "1,32,128", context: int = 2048, iters: int = 10) -> int:
  names = [m for m in models.split(",") if m] or list(MODELS)
  for row in run(names, [int(x) for x in lengths.split(",")], [int(x) for x in slots.split(",")], context, iters):
    print(json.dumps(row))
  return 0
