"""`bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N`: replay a trace of token ids through the decode engine.

Steps arrive on standard input, one JSON object per line:

  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

`entries` are one batch: each request's next tokens and the places among them whose logits are wanted. `end` lists requests that are
finished after the step. The logits of a step go to DIR/<step>.f32 (fp32, little endian, [wanted, vocab], in the order of the
entries), then `done <step>` is printed. Nothing is sampled; every step is one `MaxEngine.extend` call on the engine's slots.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from ..ops import backend


class TraceRunner:
  """Maps request ids to slots of a decode state; the state grows when a batch needs more slots than it has and none is in use."""

  def __init__(self, engine):
    self.engine, self.state, self.slot_of, self.free = engine, None, {}, []

  def _reserve(self, n: int):
    have = 0 if self.state is None else int(self.state.tokens.shape[0])
    if len(self.free) >= n:
      return
    if self.slot_of:
      raise RuntimeError(f"{n} requests join a running batch of {have} slots")
    self.state = None                                      # give the old caches back before the larger ones are allocated
    self.state = self.engine.init_decode_state(n)
    self.free = list(range(n))

  @torch.no_grad()
  def step(self, entries: list, end: list):
    """Returns the wanted logits [n, V] on the host, or None when nothing is wanted."""
    out = None
    if entries:
      fresh = [e["id"] for e in entries if e["id"] not in self.slot_of]
      self._reserve(len(fresh))
      for rid in fresh:
        self.slot_of[rid] = self.free.pop(0)
      want = [list(e.get("want") or []) for e in entries]
      logits = self.engine.extend(self.state, [self.slot_of[e["id"]] for e in entries], [e["tokens"] for e in entries], want)
      out = logits.float().cpu() if any(want) else None
      if self.engine.device.type == "cuda" and backend.ext(required=True).kernel_status(True) != 0:
        raise RuntimeError("a kernel gave up a bounded wait: the results of this step are not valid")
    for rid in end:
      slot = self.slot_of.pop(rid)
      self.engine.free_slot(self.state, slot)
      self.free.append(slot)
    return out


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda"):
  from ..config import pyconfig
  from .maxengine import MaxEngine
  if device == "cuda" and not torch.cuda.is_available():
    raise RuntimeError("a CUDA device is needed")
  backend.serving_only()
  if dtype == "float32":
    torch.set_float32_matmul_precision("highest")          # no reduced-precision products
  cfg = pyconfig.initialize(["trace_run", os.path.join(pyconfig.CONFIG_ROOT, "base.yml"), f"model_dir={model_dir}"], num_devices=1, dtype=dtype,
                            weight_dtype=dtype, max_target_length=int(max_tokens) + 1, max_prefill_predict_length=int(max_tokens),
                            enable_checkpointing=False, log_config=False, hardware="gpu" if device == "cuda" else "cpu")
  engine = MaxEngine(cfg, device=torch.device(device, 0) if device == "cuda" else device)
  engine.load_params()
  return engine


def main(argv=None) -> int:
  ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n", 1)[0])
  ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
  ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
  ap.add_argument("--out", required=True, help="folder for the logits")
  ap.add_argument("--max-tokens", required=True, type=int, help="the most tokens that live requests hold at any time")
  ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: evaluate the definitions without kernels")
  args = ap.parse_args(argv)
  runner = TraceRunner(build_engine(args.model, args.dtype, args.max_tokens, args.device))
  for line in sys.stdin:
    if not line.strip():
      continue
    s = json.loads(line)
    out = runner.step(s.get("entries") or [], s.get("end") or [])
    if out is not None:
      with open(os.path.join(args.out, f"{s['step']}.f32"), "wb") as fh:
        fh.write(out.contiguous().numpy().astype("<f4", copy=False).tobytes())
    print(f"done {s['step']}", flush=True)
  return 0
