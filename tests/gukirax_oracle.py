"""Plain, slow definition of the Gukirax decoder: one function per mechanism, token loops, no batching, no cache.

Nothing here is shared with the product path. Weights are a dict name -> tensor with the names of the published layout;
`spec` is the parsed config.json. All arithmetic runs in the dtype of the weights handed in (use float64 for an oracle).
"""
import torch


def layer_norm(x, w, eps):
  centred = x - x.mean(-1, keepdim=True)
  return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
  return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
  return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def xielu(z, p, q):
  """Slope 1/2 at zero on both sides; grows with the square for positive z, with a bounded exponential beside the line for the others."""
  neg = torch.clamp(z, max=0)
  return torch.where(z > 0, softplus(p) * z * z + z / 2, (0.5 + softplus(q)) * (torch.exp(neg) - 1 - neg) + z / 2)


def relu_squared(z):
  return torch.clamp(z, min=0) ** 2


def soft_cap(x, c):
  return c * torch.tanh(x / c)


def rotate_halves(x, base, dims):
  """x [T, H, D]: lanes (i, i + dims/2), i < dims/2, turned by t * base^(-2i/dims) at position t; lanes from dims on stay."""
  y = x.clone()
  for i in range(dims // 2):
    ang = torch.arange(x.shape[0], dtype=torch.float64) * (float(base) ** (-2.0 * i / dims))
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., i], x[..., i + dims // 2]
    y[..., i] = u * c - v * s
    y[..., i + dims // 2] = v * c + u * s
  return y


def talking_attention(q, k, v, scale, talk, sink):
  """q [T, H, D]; k [T, G, D]; v [T, G, Dv]; talk [H, H]; sink [H]. Causal; before the softmax every head's scores become a weighted sum of
  all heads' scores; exp(sink) joins the denominator only."""
  T, H, G = q.shape[0], q.shape[1], k.shape[1]
  own = [(q[:, h] @ k[:, h // (H // G)].T) * scale for h in range(H)]
  future = torch.triu(torch.ones(T, T, dtype=torch.bool), 1)
  out = []
  for h in range(H):
    s = sum(talk[h, g] * own[g] for g in range(H)).masked_fill(future, float("-inf"))
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[h])
    p = torch.exp(s - top)
    out.append((p @ v[:, h // (H // G)]) / (p.sum(-1, keepdim=True) + torch.exp(sink[h] - top)))
  return torch.stack(out, 1)


def attention_mixer(h, w, m, eps):
  T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
  q, k = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, G, D)
  v = k.clone()
  q, k = (rms(rotate_halves(t, m["rot"]["base"], m["rot"]["dims"]), eps) for t in (q, k))
  return talking_attention(q, k, v, m["scale"], w["talk"], w["sink"]).reshape(T, H * Dv) @ w["o"].T


MIXERS = {"attention": attention_mixer}


def dense_mlp(h, w, m, margins):
  return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def expert(h, up, down):
  return relu_squared(h @ up.T) @ down.T


def moe_mlp(h, w, m, margins):
  """Softmax scores over all experts; the `top` largest weight what their experts give; one more expert runs for every token. `margins` (a list)
  collects by how much the last chosen logit of every token exceeds the next one."""
  out = torch.zeros_like(h)
  for t in range(h.shape[0]):
    z = w["router"] @ h[t]
    if margins is not None and m["router"]["top"] < m["router"]["experts"]:
      ranked = torch.sort(z, descending=True).values
      margins.append((t, float(ranked[m["router"]["top"] - 1] - ranked[m["router"]["top"]])))
    s = torch.exp(z - z.max())
    s = s / s.sum()
    for e in torch.argsort(s, descending=True)[:m["router"]["top"]].tolist():
      out[t] += s[e] * expert(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
  if m.get("shared") is not None:
    out = out + expert(h, w["shared.up"], w["shared.down"])
  return out


MLPS = {"dense": dense_mlp, "moe": moe_mlp}


def gated_sublayer(x, norm, branch, gate, gate_bias, post):
  """x + post(branch(h) * sigmoid(W h + b)), h = norm(x)."""
  h = norm(x)
  return x + post(branch(h) * sigmoid(h @ gate.T + gate_bias))


def part(weights, prefix):
  return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def layer_runs(spec):
  """[(layer, first of a pass of the loop?)] in running order."""
  n, loop = len(spec["layers"]), spec.get("loop")
  if loop is None:
    return [(i, False) for i in range(n)]
  a, b = loop["start"], loop["stop"]
  return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(weights, spec, tokens, layers_out=None, margins=None):
  """tokens: list of ids -> logits [T, vocab]; `layers_out` (a list) collects the residual stream after every layer run."""
  eps = spec["norm"]["eps"]
  x = layer_norm(weights["embed"][torch.tensor(tokens)], weights["embed.norm"], eps)
  x0 = x
  for i, opens in layer_runs(spec):
    if opens:
      x = torch.cat([x, x0], -1) @ weights["loop.in"].T
    lay = spec["layers"][i]

    def norm(which, i=i):
      return lambda t: layer_norm(t, weights[f"l{i}.{which}"], eps)
    mix = part(weights, f"l{i}.mix.")
    x = gated_sublayer(x, norm("norm1"), lambda h: MIXERS[lay["type"]](h, mix, lay["mixer"], eps), weights[f"l{i}.rg1"], weights[f"l{i}.rg1.b"], norm("norm1b"))
    if lay["mlp"] is not None:
      mlp = part(weights, f"l{i}.mlp.")
      x = gated_sublayer(x, norm("norm2"), lambda h: MLPS[lay["mlp"]["kind"]](h, mlp, lay["mlp"], margins), weights[f"l{i}.rg2"], weights[f"l{i}.rg2.b"], norm("norm2b"))
    if layers_out is not None:
      layers_out.append(x)
  h = layer_norm(x, weights["final.norm"], eps)
  return soft_cap(h @ weights["embed"].T * spec["logit_scale"], spec["logit_softcap"])
