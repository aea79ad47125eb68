"""Random Gukirax models for the tests: specs of several sizes and seeded weights. How a folder is written and run is shared with the other
model-folder families (`silinex_models`)."""
import torch

import gukirax_oracle as O
from silinex_models import config, engine, prompt, rel, rel_rows, run_pieces, write_folder  # noqa: F401


def attention(heads, kv_heads, dim, rot, scale, base=700.0):
  return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, rot={"base": base, "dims": rot}, scale=scale)}


def dense(ff):
  return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
  return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def spec(layers, width, loop=None, vocab=71, eps=1e-5, logit_scale=0.7, cap=6.0):
  """layers: (mixer, feed-forward or None) pairs; loop: (start, stop, times)."""
  return {"architecture": "Gukirax", "layers": [{**m, "mlp": f} for m, f in layers], "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None,
          "logit_scale": logit_scale, "logit_softcap": cap, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every size differs from every other where the equations allow it; odd sizes take the unvectorised kernels
SPECS = {
    "heads": spec([(attention(6, 3, 20, 8, 0.3), None)], 48),
    "heads_one_key": spec([(attention(5, 1, 14, 14, 0.4), dense(36))], 44, eps=0.02),
    "heads_no_groups": spec([(attention(4, 4, 24, 2, 0.2, 40.0), None)], 40),
    "heads_odd": spec([(attention(2, 1, 11, 6, 0.5), dense(21))], 33),
    "heads_single": spec([(attention(1, 1, 32, 0, 0.3), dense(40))], 24),
    "heads_64": spec([(attention(8, 2, 64, 32, 0.12), dense(96))], 80, logit_scale=1.0),
    "heads_128": spec([(attention(6, 3, 128, 48, 0.08), None)], 96),
    "heads_20": spec([(attention(20, 5, 40, 16, 0.15), dense(64))], 64),
    "heads_many_keys": spec([(attention(12, 12, 56, 24, 0.1), None)], 72),
    "heads_wide": spec([(attention(2, 1, 200, 64, 0.05), dense(40))], 56),
    "experts": spec([(attention(2, 1, 8, 4, 0.5), moe(8, 3, 24, 40)), (attention(4, 2, 16, 8, 0.3), moe(5, 1, 40))], 48),
    "experts_all": spec([(attention(3, 3, 8, 8, 0.4), moe(4, 4, 17, 9))], 36),
    "experts_one": spec([(attention(2, 2, 16, 4, 0.3), moe(1, 1, 32, 24))], 40),
    "experts_tiles": spec([(attention(2, 1, 64, 16, 0.1), moe(2, 2, 128, 128))], 128),
    "loop_all": spec([(attention(4, 2, 16, 8, 0.3), dense(24)), (attention(3, 1, 24, 6, 0.2), None)], 40, loop=(0, 2, 3)),
    "loop_one": spec([(attention(2, 2, 8, 8, 0.5), None), (attention(4, 1, 16, 16, 0.3), moe(3, 2, 20, 12)), (attention(2, 1, 24, 4, 0.2), dense(28))], 32,
                     loop=(1, 2, 4)),
    "loop_once": spec([(attention(2, 1, 16, 8, 0.4), dense(16)), (attention(2, 1, 16, 8, 0.4), dense(16))], 24, loop=(1, 2, 1)),
    "mixed": spec([(attention(4, 2, 24, 12, 0.3), dense(70)), (attention(6, 2, 16, 16, 0.2, 90.0), moe(6, 2, 28, 36)), (attention(3, 3, 40, 8, 0.15), None),
                   (attention(2, 1, 8, 4, 0.4), moe(3, 1, 44)), (attention(5, 1, 32, 20, 0.25), dense(50))], 60, loop=(1, 4, 2), vocab=93),
    "mixed_even": spec([(attention(8, 2, 64, 32, 0.12), dense(128)), (attention(4, 4, 64, 64, 0.1), moe(4, 2, 128, 256)),
                        (attention(16, 4, 128, 64, 0.06), moe(8, 1, 256, 128))], 128, loop=(0, 2, 2), vocab=120),
}


def has_experts(sp):
  return any(lay["mlp"] is not None and lay["mlp"]["kind"] == "moe" for lay in sp["layers"])


def weights(sp, seed=0):
  """fp32 weights (values exact in bf16)."""
  g = torch.Generator().manual_seed(seed)
  W = {}

  def mat(name, out, inp, gain=1.0):
    W[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

  def vec(name, n, mean=0.0, std=0.2):
    W[name] = mean + std * torch.randn(n, generator=g)
  d = sp["width"]
  mat("embed", sp["vocab"], d, 2.0)
  vec("embed.norm", d, 1.0)
  if sp["loop"] is not None:
    mat("loop.in", d, 2 * d, 1.4)
  for i, lay in enumerate(sp["layers"]):
    m, p, f = lay["mixer"], f"l{i}.mix.", lay["mlp"]
    for q in (1, 2) if f is not None else (1,):
      vec(f"l{i}.norm{q}", d, 1.0)
      vec(f"l{i}.norm{q}b", d, 0.8)
      mat(f"l{i}.rg{q}", d, d)
      vec(f"l{i}.rg{q}.b", d, 0.3, 0.7)
    H = m["heads"]
    mat(p + "q", H * m["dim"], d)
    mat(p + "k", m["kv_heads"] * m["dim"], d)
    W[p + "talk"] = torch.eye(H) * 0.9 + torch.randn(H, H, generator=g) * 0.5 * H ** -0.5
    vec(p + "sink", H, 0.5, 1.5)
    mat(p + "o", d, H * m["vdim"])
    if f is None:
      continue
    p = f"l{i}.mlp."
    if f["kind"] == "dense":
      mat(p + "up", f["ff"], d)
      mat(p + "down", d, f["ff"])
      vec(p + "act", 2, 0.3, 0.8)
    else:
      mat(p + "router", f["router"]["experts"], d, 2.0)
      for e in range(f["router"]["experts"]):
        mat(f"{p}e{e}.up", f["expert"]["ff"], d, 1.5)
        mat(f"{p}e{e}.down", d, f["expert"]["ff"])
      if f["shared"] is not None:
        mat(p + "shared.up", f["shared"]["ff"], d)
        mat(p + "shared.down", d, f["shared"]["ff"])
  vec("final.norm", d, 1.0)
  return {k: v.bfloat16().float() for k, v in W.items()}


def oracle_logits(sp, W, tokens):
  return O.forward({k: v.double() for k, v in W.items()}, sp, tokens)


def clear_prompt(n, sp, W, seed=1, first=8):
  """A prompt whose first tokens choose their experts by clear margins. Rounding may turn a close call around, which is no fault, but an early
  token that took another expert reaches every later one."""
  while True:
    toks = prompt(n, sp, seed)
    margins = []
    O.forward(W, sp, toks[:first], margins=margins)
    if all(m > 0.12 for _, m in margins):
      return toks
    seed += 1000


def greedy_oracle(sp, W, tokens, n):
  toks = list(tokens)
  for _ in range(n):
    toks.append(int(oracle_logits(sp, W, toks)[-1].argmax()))
  return toks[len(tokens):]


def matching_heads(sp, W, query, key):
  """Weights of a first layer in which the query of token `query` equals the key of token `key` in the first head of every group, so that
  the pair scores dim * scale wherever it stands (rotation aside): the key's embedding is a permutation of the query's, which layer norms
  without weights pass on, and the query matrix is the key matrix with its columns permuted."""
  W = dict(W)
  m, d = sp["layers"][0]["mixer"], sp["width"]
  H, G, D = m["heads"], m["kv_heads"], m["dim"]
  perm = torch.randperm(d, generator=torch.Generator().manual_seed(5))
  W["embed.norm"] = W["l0.norm1"] = torch.ones(d)
  W["embed"] = W["embed"].clone()
  W["embed"][key] = W["embed"][query][perm]
  q, k = W["l0.mix.q"].clone().view(H, D, d), W["l0.mix.k"].view(G, D, d)
  for h in range(0, H, H // G):
    q[h][:, perm] = k[h // (H // G)]
  W["l0.mix.q"] = q.reshape(H * D, d)
  return W
