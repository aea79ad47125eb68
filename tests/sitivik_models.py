"""Random Sitivik models for the tests: specs of several sizes and seeded weights. How a folder is written and run is shared with the other
model-folder families (`silinex_models`)."""
import torch

import sitivik_oracle as O
from silinex_models import config, engine, prompt, rel, rel_rows, run_pieces, write_folder  # noqa: F401


def window(heads, kv_heads, dim, vdim, rot, size, scale, base=700.0, scaling=None):
  turn = {"base": base, "dims": rot}
  if scaling:
    turn["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
  return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask={"size": size}, rot=turn, scale=scale)


def retention(dim, vdim, rot, decay, base=90.0):
  return dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay), rot={"base": base, "dims": rot})


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
  return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, _ranks=(decay_rank, gate_rank))


def parallel(left, right):
  return {"type": "parallel", "mixer": {"left": left, "right": right}}


def parallel_2(left, right, left_scale=0.7, right_scale=1.2):
  return {"type": "parallel_2", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def differential(heads, kv_heads, dim, vdim, scale, diff=0.35, coef=0.4, every=11):
  return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff, q_temp={"coef": coef, "every": every})}


def spec(layers, width, vocab=71, eps=1e-5, embed=3.0, side=10):
  """layers: (mixer, feed-forward width or None) pairs."""
  return {"architecture": "Sitivik", "layers": [{**m, "mlp": {"kind": "dense", "ff": f} if f else None} for m, f in layers], "embedding": {"scale": embed},
          "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


SLOW = (0.97, 0.999)
# every size differs from every other where the equations allow it; odd sizes take the unvectorised kernels
SPECS = {
    "window": spec([(parallel(window(6, 3, 20, 12, 8, 7, 0.3), retention(14, 10, 6, (0.9, 0.99, 0.5))), None)], 48),
    "window_stretched": spec([(parallel(window(4, 1, 24, 40, 24, 33, 0.25, 5000.0, (3.0, 1.0, 5.0, 100.0)), retention(24, 40, 24, SLOW)), 36)], 44, eps=0.02, side=7),
    "window_one": spec([(parallel(window(3, 3, 16, 24, 2, 1, 0.2, 40.0), retention(12, 20, 0, (0.8,))), None)], 40),
    "window_odd": spec([(parallel(window(2, 1, 11, 7, 6, 5, 0.4), retention(9, 5, 4, (0.95, 0.3))), 21)], 33, side=3),
    "window_64": spec([(parallel(window(20, 1, 64, 64, 32, 20, 0.1), retention(64, 32, 64, SLOW + (0.7,))), 96)], 80, embed=1.0, side=8),
    "window_128": spec([(parallel(window(4, 2, 128, 128, 64, 40, 0.05), retention(128, 64, 32, SLOW)), 64)], 96, side=16),
    "window_beyond_flash": spec([(parallel(window(2, 1, 200, 136, 64, 9, 0.05), retention(200, 136, 64, (0.9, 1.0))), None)], 72),
    "chunk": spec([(parallel_2(window(6, 2, 18, 14, 12, 8, 0.3), delta(6, 3, 12, 20, 3, 5, 9)), None)], 48),
    "chunk_one": spec([(parallel_2(window(2, 1, 12, 8, 4, 1, 0.3), delta(2, 2, 8, 12, 1, 1, 2)), 20)], 40),
    "chunk_odd": spec([(parallel_2(window(5, 5, 13, 9, 10, 13, 0.4), delta(3, 1, 7, 9, 6, 3, 4), 1.3, 0.4), 21)], 33, eps=0.03, side=5),
    "chunk_64": spec([(parallel_2(window(4, 4, 64, 48, 16, 31, 0.15), delta(4, 2, 32, 64, 4, 8, 16)), 96)], 80, side=8),
    "chunk_wide": spec([(parallel_2(window(8, 2, 96, 112, 96, 50, 0.08), delta(4, 4, 128, 48, 4, 24, 24)), 64)], 96),
    "delta_unaligned": spec([(parallel_2(window(2, 2, 160, 120, 40, 17, 0.06), delta(2, 1, 40, 24, 2, 12, 10)), None)], 64),
    "differential": spec([(differential(6, 3, 20, 12, 0.3), None)], 48),
    "differential_one_kv_head": spec([(differential(5, 1, 14, 18, 0.4, 0.8, 0.1, 3), 36)], 44, eps=0.02),
    "differential_odd": spec([(differential(2, 2, 11, 7, 0.4, 0.1, 1.0, 1), 21)], 33, side=3),
    "differential_64": spec([(differential(8, 2, 32, 64, 0.2), 96)], 80, side=8),
    "differential_128": spec([(differential(4, 2, 64, 128, 0.12), 64)], 96, embed=1.0),
    "differential_192": spec([(differential(4, 4, 88, 40, 0.1), None)], 64),
    "differential_apart": spec([(differential(2, 1, 104, 72, 0.1), 40)], 56),
    "differential_widest": spec([(differential(2, 1, 136, 200, 0.08), None)], 72),
    "mixed": spec([(parallel(window(4, 2, 24, 16, 12, 6, 0.3), retention(16, 24, 8, (0.95, 0.6, 0.999))), 70), (differential(4, 2, 20, 28, 0.3), 50),
                   (parallel_2(window(6, 3, 16, 20, 8, 9, 0.35), delta(4, 2, 24, 16, 3, 6, 10)), None),
                   (parallel(window(4, 2, 24, 16, 12, 6, 0.3), retention(16, 24, 8, (0.95, 0.6, 0.999))), 70),
                   (parallel_2(window(2, 1, 40, 24, 40, 4, 0.2, 300.0), delta(2, 1, 16, 32, 2, 4, 4), 0.4, 1.5), 44)], 60, vocab=93, side=9),
    "mixed_even": spec([(parallel(window(8, 2, 64, 64, 32, 24, 0.12, 1000.0, (2.0, 1.0, 4.0, 60.0)), retention(32, 64, 32, SLOW + (0.9, 0.5))), 128),
                        (differential(8, 4, 64, 128, 0.1), 256), (parallel_2(window(4, 4, 128, 64, 128, 40, 0.08), delta(8, 4, 32, 32, 4, 16, 8)), 128),
                        (differential(4, 1, 32, 64, 0.15), None)], 128, vocab=120, side=16),
}


def weights(sp, seed=0):
  """fp32 weights (values exact in bf16)."""
  g = torch.Generator().manual_seed(seed)
  W = {}

  def mat(name, out, inp, gain=1.0):
    W[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

  def vec(name, n, mean=0.0, std=0.2):
    W[name] = mean + std * torch.randn(n, generator=g)

  def biased(p, m, maps=1):
    for n, rows in (("q", m["heads"] * maps * m["dim"]), ("k", m["kv_heads"] * maps * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
      mat(p + n, rows, d)
      vec(p + n + ".b", rows, 0.0, 0.5)
  d, L = sp["width"], len(sp["layers"])
  mat("embed", sp["vocab"], d, d ** 0.5)
  W["side.embed"] = torch.randn(sp["vocab"], L * sp["token_side"]["dim"], generator=g)
  for i, lay in enumerate(sp["layers"]):
    m, p, f = lay["mixer"], f"l{i}.mix.", lay["mlp"]
    vec(f"l{i}.norm1", d, 1.0)
    vec(f"l{i}.ls1", d, 0.8, 0.3)
    if lay["type"] == "attention":
      biased(p, m, 2)
      for n in ("lq1", "lk1", "lq2", "lk2"):
        vec(p + n, m["dim"], 0.0, 0.6 * m["dim"] ** -0.25)
      mat(p + "g", m["heads"], d)
      mat(p + "o", d, m["heads"] * m["vdim"])
    else:
      a, r = m["left"], m["right"]
      biased(p + "left.", a)
      whole = lay["type"] == "parallel"
      vec(p + "left.q.norm", a["heads"] * a["dim"] if whole else a["dim"], 1.0)
      vec(p + "left.k.norm", a["kv_heads"] * a["dim"] if whole else a["dim"], 1.0)
      mat(p + "left.g", a["heads"] * a["vdim"], d)
      mat(p + "left.o", d, a["heads"] * a["vdim"])
      H, dk, dv = r["heads"], r["dim"], r["vdim"]
      G = H if whole else r["kv_heads"]
      for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
        mat(f"{p}right.{n}", rows, d)
        if not whole:
          W[f"{p}right.{n}.conv"] = torch.randn(rows, r["conv"], generator=g) * 0.6
      mat(p + "right.o", d, H * dv)
      if whole:
        vec(p + "left.o.b", d, 0.0, 0.5)
        mat(p + "right.g", H * dv, d)
        vec(p + "left.out", d, 1.0)
        vec(p + "right.out", d, 1.0)
      else:
        ra, rg = r["_ranks"]
        mat(p + "right.b", H, d, 1.5)
        vec(p + "right.A_log", H, -1.0, 1.0)
        vec(p + "right.norm", dv, 1.0)
        mat(p + "right.a1", ra, d)
        mat(p + "right.a2", H * dk, ra, 1.5)
        vec(p + "right.dt_bias", H * dk, -1.0, 1.0)
        mat(p + "right.g1", rg, d)
        mat(p + "right.g2", H * dv, rg)
    if f is not None:
      vec(f"l{i}.norm2", d, 1.0)
      vec(f"l{i}.ls2", d, 0.8, 0.3)
      mat(f"l{i}.mlp.gate", f["ff"], d)
      mat(f"l{i}.mlp.up", f["ff"], d)
      mat(f"l{i}.mlp.down", d, f["ff"])
    mat(f"l{i}.side.gate", sp["token_side"]["dim"], d)
    mat(f"l{i}.side.proj", d, sp["token_side"]["dim"])
    vec(f"l{i}.side.norm", d, 0.7)
  vec("final.norm", d, 1.0)
  return {k: v.bfloat16().float() for k, v in W.items()}


def folder(path, sp, W):
  """`_ranks` is known from the tensors only."""
  def clean(m):
    return {k: clean(v) if isinstance(v, dict) else v for k, v in m.items() if not k.startswith("_")}
  return write_folder(path, {**sp, "layers": [clean(lay) for lay in sp["layers"]]}, W)


def oracle_logits(sp, W, tokens):
  return O.forward({k: v.double() for k, v in W.items()}, sp, tokens)


def greedy_oracle(sp, W, tokens, n):
  toks = list(tokens)
  for _ in range(n):
    toks.append(int(oracle_logits(sp, W, toks)[-1].argmax()))
  return toks[len(tokens):]


def sharpened(sp, W, query, key, score=16.0):
  """(spec, weights) in which the query of token `query` equals the key of token `key` in layer 0's softmax attention, so that the pair scores
  about `score` wherever it stands: the key's embedding is a permutation of the query's, which an RMS norm without weights passes on, and the
  query matrix is the key matrix with its columns permuted. Positions barely matter: two lanes rotate at most."""
  W, lay, d = dict(W), dict(sp["layers"][0]), sp["width"]
  pre = "l0.mix." if lay["type"] == "attention" else "l0.mix.left."
  m = dict(lay["mixer"] if lay["type"] == "attention" else lay["mixer"]["left"])
  maps = 2 if lay["type"] == "attention" else 1
  H, G, D = m["heads"], m["kv_heads"], m["dim"] * maps
  m["scale"] = score / m["dim"]
  if maps == 1:
    m["rot"] = {"base": 1e9, "dims": 2}
  else:
    m["q_temp"] = {"coef": 0.02, "every": 9}
  perm = torch.randperm(d, generator=torch.Generator().manual_seed(5))
  W["l0.norm1"], W["embed"] = torch.ones(d), W["embed"].clone()
  W["embed"][key] = W["embed"][query][perm]
  k = W[pre + "k"].view(G, D, d)
  q = torch.empty(H, D, d)
  for h in range(H):
    q[h][:, perm] = k[h // (H // G)]
  W[pre + "q"] = q.reshape(H * D, d)
  for n in ("q", "k"):
    W[f"{pre}{n}.b"] = torch.zeros_like(W[f"{pre}{n}.b"])
    if maps == 1:
      W[f"{pre}{n}.norm"] = torch.ones_like(W[f"{pre}{n}.norm"])
  W["l0.ls1"] = torch.full((d,), 2.0)
  mixer = m if lay["type"] == "attention" else {**lay["mixer"], "left": m}
  return {**sp, "layers": [{**lay, "mixer": mixer}] + sp["layers"][1:]}, {n: t.bfloat16().float() for n, t in W.items()}
