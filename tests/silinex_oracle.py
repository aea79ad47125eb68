"""Plain, slow definition of the Silinex decoder: one function per mechanism, token loops, no batching, no cache.

Nothing here is shared with the product path. Weights are a dict name -> tensor with the names of the published layout;
`spec` is the parsed config.json. All arithmetic runs in the dtype of the weights handed in (use float64 for an oracle).
"""
import math

import torch


def rms(x, eps):
  """RMS normalisation over the last dimension; eps is added to the mean square."""
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
  return rms(x, eps) * (1.0 + w)


def sigmoid(x):
  return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
  return x * sigmoid(x)


def gelu_erf(x):
  return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def softplus(x):
  return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def unit(x):
  return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def causal_conv(x, w):
  """x [T, C], w [C, taps]; tap taps-1 multiplies the current token, tokens before the first are zero."""
  T, C = x.shape
  taps = w.shape[1]
  y = torch.zeros_like(x)
  for t in range(T):
    for j in range(taps):
      s = t - (taps - 1 - j)
      if s >= 0:
        y[t] += w[:, j] * x[s]
  return y


def rotate_pairs(x, base):
  """x [T, ..., D]: lanes (2i, 2i+1) turned by t * base^(-2i/D) at position t."""
  T, D = x.shape[0], x.shape[-1]
  y = torch.zeros_like(x)
  for i in range(D // 2):
    ang = torch.arange(T, dtype=torch.float64) * (float(base) ** (-2.0 * i / D))
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    shape = [T] + [1] * (x.dim() - 2)
    c, s = c.view(shape), s.view(shape)
    u, v = x[..., 2 * i], x[..., 2 * i + 1]
    y[..., 2 * i] = u * c - v * s
    y[..., 2 * i + 1] = v * c + u * s
  return y


def gated_linear_recurrence(q, k, v, alpha):
  """q, k, alpha [T, H, Dk]; v [T, H, Dv]: S <- diag(alpha) S + k v^T, o = S^T q."""
  T, H, Dk = q.shape
  S = torch.zeros(H, Dk, v.shape[-1], dtype=q.dtype)
  out = []
  for t in range(T):
    S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
    out.append((S * q[t][:, :, None]).sum(1))
  return torch.stack(out)


def delta_recurrence(q, k, v, g, beta):
  """q, k [T, H, Dk] (unit / scaled already); v [T, H, Dv]; g, beta [T, H]."""
  T, H, Dk = q.shape
  S = torch.zeros(H, Dk, v.shape[-1], dtype=q.dtype)
  out = []
  for t in range(T):
    S = g[t][:, None, None] * S
    u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
    S = S + k[t][:, :, None] * u[:, None, :]
    out.append((S * q[t][:, :, None]).sum(1))
  return torch.stack(out)


def windowed_softmax_attention(q, k, v, scale, window):
  """q, k [T, H, D]; v [T, H, Dv]; query i sees keys i - window + 1 .. i."""
  T = q.shape[0]
  out = torch.zeros(T, q.shape[1], v.shape[-1], dtype=q.dtype)
  for i in range(T):
    lo = max(0, i - window + 1)
    s = torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1]) * scale
    p = torch.exp(s - s.max(-1, keepdim=True).values)
    p = p / p.sum(-1, keepdim=True)
    out[i] = torch.einsum("hj,jhd->hd", p, v[lo:i + 1])
  return out


def gla_mixer(h, w, m, eps):
  T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
  q = (h @ w["q"].T).view(T, H, dk) * dk ** -0.5
  k = (h @ w["k"].T).view(T, H, dk)
  v = (h @ w["v"].T).view(T, H, dv)
  z = ((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]).view(T, H, dk)
  o = gated_linear_recurrence(q, k, v, sigmoid(z) ** (1.0 / m["tau"]))
  o = rms(o, eps) * w["norm"]
  return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def delta_mixer(h, w, m, eps):
  T, H, Hk, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
  q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
  q, k, v = unit(q.view(T, Hk, dk)) * dk ** -0.5, unit(k.view(T, Hk, dk)), v.view(T, H, dv)
  src = torch.tensor([j // (H // Hk) for j in range(H)])
  q, k = q[:, src], k[:, src]
  beta = sigmoid(h @ w["b"].T)
  g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
  o = rms(delta_recurrence(q, k, v, g, beta), eps) * w["norm"]
  return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def latent_mixer(h, w, m, eps):
  T, H, dn, dr, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
  cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
  q = (cq @ w["uq"].T).view(T, H, dn + dr)
  kv = h @ w["dkv"].T
  c = rms(kv[:, :R], eps) * w["dkv.norm"]
  kr = rotate_pairs(kv[:, None, R:], m["rot"]["base"])
  qr = rotate_pairs(q[..., dn:], m["rot"]["base"])
  kn, v = (c @ w["uk"].T).view(T, H, dn), (c @ w["uv"].T).view(T, H, dv)
  o = windowed_softmax_attention(torch.cat([q[..., :dn], qr], -1), torch.cat([kn, kr.expand(T, H, dr)], -1), v, m["scale"],
                                 m["mask"]["size"])
  return o.reshape(T, H * dv) @ w["o"].T


MIXERS = {"gla": gla_mixer, "delta": delta_mixer, "latent_attention": latent_mixer}


def layer_weights(weights, i, part):
  pre = f"l{i}.{part}."
  return {n[len(pre):]: t for n, t in weights.items() if n.startswith(pre)}


def forward(weights, spec, tokens, layers_out=None):
  """tokens: list of ids -> logits [T, vocab]; `layers_out` (a list) collects the residual stream after every layer."""
  eps, m = spec["norm"]["eps"], spec["residual_mult"]
  x = weights["embed"][torch.tensor(tokens)]
  for i, lay in enumerate(spec["layers"]):
    n = lambda which, t, i=i: zero_centred_norm(t, weights[f"l{i}.{which}"], eps)  # noqa: E731
    y = MIXERS[lay["type"]](n("norm1", x), layer_weights(weights, i, "mix"), lay["mixer"], eps)
    x = x + m * n("norm1b", y)
    if lay["mlp"] is not None:
      w = layer_weights(weights, i, "mlp")
      x = x + m * n("norm2b", gelu_erf(n("norm2", x) @ w["up"].T) @ w["down"].T)
    if layers_out is not None:
      layers_out.append(x.clone())
  return zero_centred_norm(x, weights["final.norm"], eps) @ weights["head"].T
