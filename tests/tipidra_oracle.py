"""Plain, slow definition of the Tipidra decoder: one function per mechanism, token loops, no batching, no cache.

Nothing here is shared with the product path. Weights are a dict name -> tensor with the names of the published layout;
`spec` is the parsed config.json. All arithmetic runs in the dtype of the weights handed in (use float64 for an oracle).
"""
import math

import torch


def rms(x, eps):
  """x over its root mean square along the last dimension; eps joins the mean square."""
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
  centred = x - x.mean(-1, keepdim=True)
  return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(x):
  return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
  return x * sigmoid(x)


def gelu_tanh(x):
  return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def softplus(x):
  return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def soft_cap(x, c):
  return c * torch.tanh(x / c)


def causal_conv(x, w, b):
  """x [T, C], w [C, taps], b [C]; tap taps-1 multiplies the current token, tokens before the first are zero."""
  T, taps = x.shape[0], w.shape[1]
  y = b.expand_as(x).clone()
  for t in range(T):
    for j in range(taps):
      s = t - (taps - 1 - j)
      if s >= 0:
        y[t] += w[:, j] * x[s]
  return y


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


def sink_attention(q, k, v, scale, cap, sink):
  """q [T, H, D]; k [T, G, D]; v [T, G, Dv]; sink [H]: causal, capped scores, exp(sink) in the denominator only."""
  T, H, G = q.shape[0], q.shape[1], k.shape[1]
  out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
  for h in range(H):
    g = h // (H // G)
    for i in range(T):
      s = soft_cap((k[:i + 1, g] @ q[i, h]) * scale, cap)
      top = torch.maximum(s.max(), sink[h])
      p = torch.exp(s - top)
      out[i, h] = (p @ v[:i + 1, g]) / (p.sum() + torch.exp(sink[h] - top))
  return out


def selective_scan(x, dt, A, B, C, D):
  """x, dt [T, channels]; A [channels, n]; B, C [T, n]; D [channels]. Each channel decays its n states at its own rates, adds its input times
  the step size along B, and reads them out along C next to a direct path."""
  S = torch.zeros_like(A)
  out = []
  for t in range(x.shape[0]):
    S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
    out.append((S * C[t][None]).sum(-1) + D * x[t])
  return torch.stack(out)


def attention_mixer(h, w, m, eps):
  T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
  q, k, v = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, G, D), (h @ w["v"].T).view(T, G, Dv)
  q, k = (rms(rotate_halves(t, m["rot"]["base"], m["rot"]["dims"]), eps) for t in (q, k))
  o = sink_attention(q, k, v, m["scale"], m["softcap"], w["sink"]).reshape(T, H * Dv)
  return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def mamba_mixer(h, w, m, eps):
  inner, R, N = m["inner"], m["dt_rank"], m["state"]
  p = h @ w["in"].T
  x, z = silu(causal_conv(p[:, :inner], w["conv"], w["conv.b"])), p[:, inner:]
  s = x @ w["x"].T
  dt = softplus(s[:, :R] @ w["dt"].T + w["dt.b"])
  y = selective_scan(x, dt, -torch.exp(w["A_log"]), s[:, R:R + N], s[:, R + N:], w["D"])
  return (y * silu(z)) @ w["o"].T


MIXERS = {"attention": attention_mixer, "mamba1": mamba_mixer}


def dense_mlp(h, w, m):
  return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def clamped_expert(h, gate, up, down, limit):
  g = torch.clamp(h @ gate.T, max=limit)
  u = torch.clamp(h @ up.T, min=-limit, max=limit)
  return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def moe_mlp(h, w, m):
  """Sigmoid scores; the `top` largest; the score multiplies what the expert reads."""
  out = torch.zeros_like(h)
  for t in range(h.shape[0]):
    s = sigmoid(w["router"] @ h[t])
    for e in torch.argsort(s, descending=True)[:m["router"]["top"]].tolist():
      out[t] += clamped_expert(s[e] * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], m["expert"]["limit"])
  return out


MLPS = {"dense": dense_mlp, "moe": moe_mlp}


def hyper_sublayer(streams, hc, norm, branch):
  """streams: list of tensors [T, width]; hc: the weights `in` and `out`, one per stream, and `mix`, whose rows are the sources."""
  n = len(streams)
  u = sum(hc["in"][s] * streams[s] for s in range(n))
  y = branch(norm(u))
  return [sum(hc["mix"][s, t] * streams[s] for s in range(n)) + hc["out"][t] * y for t in range(n)]


def part(weights, prefix):
  return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def forward(weights, spec, tokens, layers_out=None):
  """tokens: list of ids -> logits [T, vocab]; `layers_out` (a list) collects the sum of the streams after every layer."""
  eps = spec["norm"]["eps"]
  x = weights["embed"][torch.tensor(tokens)] * spec["embedding"]["scale"]
  streams = [x.clone() for _ in range(spec["streams"])]
  for i, lay in enumerate(spec["layers"]):
    def norm(which, t, i=i):
      return layer_norm(t, weights[f"l{i}.{which}"], weights[f"l{i}.{which}.b"], eps)
    mix = part(weights, f"l{i}.mix.")
    streams = hyper_sublayer(streams, part(weights, f"l{i}.hc1."), lambda t: norm("norm1", t),
                             lambda h: MIXERS[lay["type"]](h, mix, lay["mixer"], eps))
    if lay["mlp"] is not None:
      mlp = part(weights, f"l{i}.mlp.")
      streams = hyper_sublayer(streams, part(weights, f"l{i}.hc2."), lambda t: norm("norm2", t),
                               lambda h: MLPS[lay["mlp"]["kind"]](h, mlp, lay["mlp"]))
    if layers_out is not None:
      layers_out.append(sum(streams))
  h = layer_norm(sum(streams), weights["final.norm"], weights["final.norm.b"], eps)
  return soft_cap(h @ weights["head"].T, spec["logit_softcap"])
