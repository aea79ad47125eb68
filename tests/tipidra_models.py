"""Random Tipidra models for the tests: specs of several sizes and seeded weights. How a folder is written and run is shared with the other
model-folder family (`silinex_models`)."""
import torch

import tipidra_oracle as O
from silinex_models import config, engine, prompt, rel, rel_rows, run_pieces, write_folder  # noqa: F401


def attention(heads, kv_heads, dim, vdim, rot, scale, cap, base=700.0):
  return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot={"base": base, "dims": rot}, scale=scale, softcap=cap)}


def scan(inner, state, rank, conv):
  return {"type": "mamba1", "mixer": dict(inner=inner, state=state, dt_rank=rank, conv=conv)}


def dense(ff):
  return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
  return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def spec(layers, width, streams=2, vocab=71, eps=1e-5, embed=3.0, cap=6.0):
  """layers: (mixer, feed-forward or None) pairs."""
  return {"architecture": "Tipidra", "layers": [{**m, "mlp": f} for m, f in layers], "streams": streams, "embedding": {"scale": embed},
          "logit_softcap": cap, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every size differs from every other where the equations allow it; odd sizes take the unvectorised kernels
SPECS = {
    "attention": spec([(attention(6, 3, 20, 12, 8, 0.3, 4.0), None)], 48),
    "attention_one_kv_head": spec([(attention(5, 1, 14, 18, 14, 0.5, 9.0), dense(36))], 44, streams=3, eps=0.02),
    "attention_no_groups": spec([(attention(3, 3, 16, 24, 2, 0.2, 2.0, 40.0), None)], 40, streams=1),
    "attention_odd": spec([(attention(2, 1, 11, 7, 6, 0.4, 5.0), dense(21))], 33, streams=5),
    "attention_64": spec([(attention(20, 1, 64, 64, 32, 0.1, 8.0), dense(96))], 80, embed=1.0),
    "attention_128": spec([(attention(4, 2, 128, 128, 64, 0.02, 20.0), dense(64))], 96, streams=4),
    "attention_narrow_values": spec([(attention(4, 2, 72, 40, 24, 0.15, 6.0), None)], 64),
    "attention_wide_keys": spec([(attention(3, 1, 160, 72, 40, 0.04, 3.0), dense(40))], 56),
    "attention_beyond_flash": spec([(attention(2, 1, 200, 136, 64, 0.05, 7.0), None)], 72),
    "scan": spec([(scan(40, 12, 5, 3), None)], 48),
    "scan_smallest": spec([(scan(24, 1, 1, 1), dense(20))], 32, streams=1),
    "scan_16": spec([(scan(160, 16, 8, 4), dense(64))], 72, streams=3),
    "scan_64": spec([(scan(48, 64, 20, 2), None)], 56),
    "scan_many_states": spec([(scan(12, 200, 3, 6), dense(24))], 36),
    "experts": spec([(attention(2, 1, 8, 8, 4, 0.5, 5.0), moe(8, 3, 24, 0.7)), (scan(32, 8, 4, 2), moe(5, 1, 40, 2.0))], 48),
    "experts_all": spec([(scan(24, 4, 4, 3), moe(4, 4, 17, 0.5))], 36, streams=3),
    "experts_single": spec([(scan(16, 8, 2, 2), moe(1, 1, 32, 1.5))], 40),
    "experts_tiles": spec([(attention(2, 1, 64, 64, 16, 0.1, 6.0), moe(2, 2, 128, 1.1))], 128, streams=4),
    "mixed": spec([(scan(72, 24, 10, 4), dense(70)), (attention(4, 2, 24, 16, 12, 0.3, 6.0), moe(6, 2, 28, 0.9)), (scan(56, 8, 3, 2), None),
                   (attention(3, 1, 40, 24, 40, 0.2, 11.0, 90.0), dense(50)), (scan(72, 24, 10, 4), moe(3, 1, 44, 1.7))], 60, streams=3, vocab=93),
    "mixed_even": spec([(attention(8, 2, 64, 64, 32, 0.12, 9.0), dense(128)), (scan(256, 16, 16, 4), moe(4, 2, 128, 1.0)),
                        (attention(4, 4, 128, 128, 128, 0.05, 30.0), moe(8, 1, 256, 0.8)), (scan(128, 32, 8, 3), dense(256))], 128, vocab=120),
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

  def norm(name):
    vec(name, d, 1.0)
    vec(name + ".b", d)

  def connection(p):
    n = sp["streams"]
    vec(p + "in", n, 1.0 / n, 0.3)
    vec(p + "out", n, 0.8, 0.4)
    W[p + "mix"] = torch.eye(n) * 0.8 + 0.25 * torch.randn(n, n, generator=g)
  d = sp["width"]
  mat("embed", sp["vocab"], d, d ** 0.5)
  for i, lay in enumerate(sp["layers"]):
    m, p, f = lay["mixer"], f"l{i}.mix.", lay["mlp"]
    norm(f"l{i}.norm1")
    connection(f"l{i}.hc1.")
    if lay["type"] == "attention":
      for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"]), ("g", m["heads"] * m["vdim"])):
        mat(p + n, rows, d)
      vec(p + "sink", m["heads"], 0.5, 1.5)
      mat(p + "o", d, m["heads"] * m["vdim"])
    else:
      c, n, r = m["inner"], m["state"], m["dt_rank"]
      mat(p + "in", 2 * c, d)
      W[p + "conv"] = torch.randn(c, m["conv"], generator=g) * 0.6
      vec(p + "conv.b", c)
      mat(p + "x", r + 2 * n, c, 1.5)
      mat(p + "dt", c, r)
      vec(p + "dt.b", c, -1.5, 1.5)                       # steps from a few thousandths to a few units
      W[p + "A_log"] = torch.log(torch.rand(c, n, generator=g) * 3 + 0.01)
      vec(p + "D", c, 1.0, 0.5)
      mat(p + "o", d, c)
    if f is None:
      continue
    norm(f"l{i}.norm2")
    connection(f"l{i}.hc2.")
    p = f"l{i}.mlp."
    if f["kind"] == "dense":
      mat(p + "gate", f["ff"], d)
      mat(p + "up", f["ff"], d)
      mat(p + "down", d, f["ff"])
    else:
      mat(p + "router", f["router"]["experts"], d, 2.0)
      for e in range(f["router"]["experts"]):
        mat(f"{p}e{e}.gate", f["expert"]["ff"], d, 1.5)
        mat(f"{p}e{e}.up", f["expert"]["ff"], d, 1.5)
        mat(f"{p}e{e}.down", d, f["expert"]["ff"])
  norm("final.norm")
  mat("head", sp["vocab"], d, 2.0)
  return {k: v.bfloat16().float() for k, v in W.items()}


def oracle_logits(sp, W, tokens):
  return O.forward({k: v.double() for k, v in W.items()}, sp, tokens)


def greedy_oracle(sp, W, tokens, n):
  toks = list(tokens)
  for _ in range(n):
    toks.append(int(oracle_logits(sp, W, toks)[-1].argmax()))
  return toks[len(tokens):]


def matching_heads(sp, W, query, key):
  """Weights of a first layer in which the query of token `query` equals the key of token `key` in the first head of every group, so that
  the pair scores dim * scale wherever it stands (rotation aside): the key's embedding is a permutation of the query's, which a layer norm
  without weights passes on, and the query matrix is the key matrix with its columns permuted."""
  W = dict(W)
  m, d = sp["layers"][0]["mixer"], sp["width"]
  H, G, D = m["heads"], m["kv_heads"], m["dim"]
  perm = torch.randperm(d, generator=torch.Generator().manual_seed(5))
  W["l0.norm1"], W["l0.norm1.b"] = torch.ones(d), torch.zeros(d)
  W["embed"] = W["embed"].clone()
  W["embed"][key] = W["embed"][query][perm]
  q, k = W["l0.mix.q"].clone().view(H, D, d), W["l0.mix.k"].view(G, D, d)
  for h in range(0, H, H // G):
    q[h][:, perm] = k[h // (H // G)]
  W["l0.mix.q"] = q.reshape(H * D, d)
  return W
