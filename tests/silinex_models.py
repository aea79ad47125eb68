"""Random Silinex models for the tests: specs of several sizes, seeded weights, and helpers that run them through the framework."""
import json
import os

import torch
from helpers import BASE_YML

import silinex_oracle as O


def delta(heads, kv_heads, dim, vdim, conv):
  return {"type": "delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def gla(heads, dim, vdim, tau, rank):
  return {"type": "gla", "mixer": dict(heads=heads, dim=dim, vdim=vdim, tau=tau), "_rank": rank}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, scale, base=10000.0):
  return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                                                    mask={"size": window}, rot={"base": base, "dims": rot_dim})}


def spec(layers, width, vocab=67, eps=1e-5, mult=0.8, ff=None):
  """layers: list of mixer descriptions; ff: list of feed-forward widths (None: the layer has none)."""
  ff = ff if ff is not None else [2 * width] * len(layers)
  out = []
  for lay, f in zip(layers, ff):
    out.append({**lay, "mlp": {"kind": "dense", "ff": f} if f is not None else None})
  return {"architecture": "Silinex", "layers": out, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


# every size differs from every other where the equations allow it; odd sizes take the unvectorised kernels
SPECS = {
    "delta": spec([delta(6, 3, 12, 20, 3)], 48, ff=[None]),
    "delta_one_tap": spec([delta(2, 2, 7, 9, 1)], 40, eps=0.03, mult=1.0),
    "delta_wide": spec([delta(4, 2, 64, 48, 4)], 72, ff=[56]),
    "delta_six_taps": spec([delta(3, 3, 16, 16, 6)], 64, mult=1.3),
    "gla": spec([gla(3, 10, 14, 4.0, 5)], 56, ff=[None]),
    "gla_fast_decay": spec([gla(2, 32, 64, 1.0, 8)], 64, eps=0.02),
    "gla_wide": spec([gla(5, 48, 32, 16.0, 24)], 80, mult=0.5),
    "latent": spec([latent(3, 10, 6, 14, 20, 36, 7, 0.31)], 44, ff=[None]),
    "latent_window_1": spec([latent(2, 8, 4, 8, 12, 16, 1, 0.2)], 32),
    "latent_tc": spec([latent(20, 16, 16, 24, 40, 64, 70, 0.17, 500.0)], 80, ff=[96]),
    "latent_tc_wide": spec([latent(6, 32, 16, 48, 64, 192, 33, 0.11)], 96),
    "mixed": spec([gla(3, 16, 24, 8.0, 12), latent(4, 12, 8, 16, 24, 32, 5, 0.27), delta(4, 2, 16, 24, 3), latent(2, 20, 4, 10, 30, 48, 11, 0.2, 300.0),
                   delta(2, 1, 24, 8, 2), gla(2, 8, 40, 2.0, 8)], 60, vocab=93, ff=[70, None, 40, 100, None, 64]),
    "mixed_even": spec([latent(4, 32, 32, 64, 48, 128, 12, 0.15), delta(4, 2, 32, 64, 4), gla(2, 64, 32, 8.0, 16), delta(2, 2, 64, 32, 4)], 128, vocab=120),
}


def weights(sp, seed=0, sharp=2.0):
  """fp32 weights (values exact in bf16). `sharp` scales the query projections, so that single keys stand out."""
  g = torch.Generator().manual_seed(seed)
  W = {}

  def mat(name, out, inp, gain=1.0):
    W[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

  def vec(name, n, mean=0.0, std=0.2):
    W[name] = mean + std * torch.randn(n, generator=g)
  d = sp["width"]
  mat("embed", sp["vocab"], d, d ** 0.5)
  for i, lay in enumerate(sp["layers"]):
    m, p = lay["mixer"], f"l{i}.mix."
    norms = ["norm1", "norm1b"] + (["norm2", "norm2b"] if lay["mlp"] is not None else [])
    for n in norms:
      vec(f"l{i}.{n}", d)
    H, dv = m["heads"], m["vdim"]
    if lay["type"] == "delta":
      kd = m["kv_heads"] * m["dim"]
      for n, rows in (("q", kd), ("k", kd), ("v", H * dv)):
        mat(p + n, rows, d)
        W[p + n + ".conv"] = torch.randn(rows, m["conv"], generator=g) * 0.6
      mat(p + "b", H, d, 1.5)
      mat(p + "a", H, d)
      vec(p + "A_log", H, -1.0, 1.0)
      vec(p + "dt_bias", H, -1.0, 1.0)
      vec(p + "norm", dv, 1.0)
      mat(p + "g", H * dv, d)
      mat(p + "o", d, H * dv)
    elif lay["type"] == "gla":
      for n, rows in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * dv), ("g", H * dv)):
        mat(p + n, rows, d)
      mat(p + "o", d, H * dv)
      vec(p + "norm", dv, 1.0)
      mat(p + "a1", lay["_rank"], d)
      mat(p + "a2", H * m["dim"], lay["_rank"], 2.0)
      vec(p + "a2.b", H * m["dim"], 1.0, 1.5)
    else:
      R, dr = m["kv_rank"], m["rot_dim"]
      mat(p + "dq", m["q_rank"], d)
      vec(p + "dq.norm", m["q_rank"], 1.0)
      mat(p + "uq", H * (m["dim"] + dr), m["q_rank"], sharp)
      mat(p + "dkv", R + dr, d)
      vec(p + "dkv.norm", R, 1.0)
      mat(p + "uk", H * m["dim"], R)
      mat(p + "uv", H * dv, R)
      mat(p + "o", d, H * dv)
    if lay["mlp"] is not None:
      mat(f"l{i}.mlp.up", lay["mlp"]["ff"], d)
      mat(f"l{i}.mlp.down", d, lay["mlp"]["ff"])
  vec("final.norm", d)
  mat("head", sp["vocab"], d)
  return {k: v.bfloat16().float() for k, v in W.items()}


def write_folder(path, sp, W):
  from safetensors.torch import save_file
  os.makedirs(path, exist_ok=True)
  clean = {**sp, "layers": [{k: v for k, v in lay.items() if not k.startswith("_")} for lay in sp["layers"]]}
  with open(os.path.join(path, "config.json"), "w") as fh:
    json.dump(clean, fh)
  save_file({k: v.bfloat16().contiguous() for k, v in W.items()}, os.path.join(path, "model.safetensors"))
  return str(path)


def config(path, dtype, device, max_len=160, **kw):
  from maxtext_b200.config import pyconfig
  return pyconfig.initialize(["t", BASE_YML, f"model_dir={path}"], num_devices=1, dtype=dtype, weight_dtype=dtype, max_target_length=max_len,
                             max_prefill_predict_length=max_len - 1, enable_checkpointing=False, log_config=False, per_device_batch_size=1,
                             hardware="gpu" if device == "cuda" else "cpu", decode_sampling_strategy="greedy", **kw)


def engine(path, dtype="float32", device="cpu", max_len=160, **kw):
  from maxtext_b200.inference.maxengine import MaxEngine
  e = MaxEngine(config(path, dtype, device, max_len, **kw), device=device)
  e.load_params()
  return e


def prompt(n, sp, seed=1):
  g = torch.Generator().manual_seed(seed)
  return torch.randint(0, sp["vocab"], (n,), generator=g).tolist()


def oracle_logits(sp, W, tokens):
  return O.forward({k: v.double() for k, v in W.items()}, sp, tokens)


def rel_rows(got, want):
  """Root mean square of the difference over that of the expected values, per row."""
  got, want = got.double().cpu(), want.double()
  return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()


def rel(got, want):
  return rel_rows(got, want).max().item()


def run_pieces(eng, tokens, sizes, state=None, slot=0):
  """Logits of all positions, the sequence fed in pieces of the given sizes (the last size repeats)."""
  state = state if state is not None else eng.init_decode_state(slot + 1)
  out, at, i = [], 0, 0
  while at < len(tokens):
    n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
    out.append(eng.extend(state, [slot], [tokens[at:at + n]], [list(range(n))]))
    at, i = at + n, i + 1
  return torch.cat(out)


def greedy_oracle(sp, W, tokens, n):
  toks = list(tokens)
  for _ in range(n):
    toks.append(int(oracle_logits(sp, W, toks)[-1].argmax()))
  return toks[len(tokens):]
