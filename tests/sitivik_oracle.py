"""Plain, slow definition of the Sitivik decoder: one function per mechanism, one sequence, no cache.

Nothing here is shared with the product path. Weights are a dict name -> tensor with the names of the published layout;
`spec` is the parsed config.json. All arithmetic runs in the dtype of the weights handed in (use float64 for an oracle).
"""
import math

import torch


def rms(x, eps):
  """x over its root mean square along the last dimension; eps joins the mean square."""
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
  return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
  return x * sigmoid(x)


def gelu_tanh(x):
  return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def softplus(x):
  return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def unit(x):
  return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


# ------------------------------------------------------------------------------------------ positions
def frequencies(rot):
  """base^(-2i/dims) per rotated pair; with `scaling`, long wavelengths are slowed down by `factor`, short ones kept, those between blended."""
  out = []
  for i in range(rot["dims"] // 2):
    f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
    sc = rot.get("scaling")
    if sc:
      wave = 2.0 * math.pi / f
      if wave > sc["original"] / sc["low"]:
        f = f / sc["factor"]
      elif wave >= sc["original"] / sc["high"]:
        s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
        f = (1.0 - s) * f / sc["factor"] + s * f
    out.append(f)
  return out


def rotate(x, rot, paired, start=0):
  """x [T, H, D]; `paired`: lanes (2i, 2i+1) turn together, otherwise lanes (i, i + dims/2). Lanes from dims on stay."""
  y = x.clone()
  for i, f in enumerate(frequencies(rot)):
    a, b = (2 * i, 2 * i + 1) if paired else (i, i + rot["dims"] // 2)
    ang = (start + torch.arange(x.shape[0], dtype=torch.float64)) * f
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    y[..., a] = x[..., a] * c - x[..., b] * s
    y[..., b] = x[..., b] * c + x[..., a] * s
  return y


def temperature(T, coef, every):
  p = torch.arange(T, dtype=torch.float64)
  return 1.0 + coef * torch.log(torch.floor((p + 1.0) / every) + 1.0)


# ------------------------------------------------------------------------------------------ softmax attention
def visible(T, window=0, chunk=0):
  i, j = torch.arange(T)[:, None], torch.arange(T)[None]
  see = j <= i
  if window:
    see = see & (i - j < window)
  if chunk:
    see = see & (i // chunk == j // chunk)
  return see


def attention(q, k, v, scale, see, add_one=False):
  """q [T, H, D]; k [T, G, D]; v [T, G, Dv]; see [T, T]; `add_one`: the denominator holds a score of zero without a value."""
  H, G = q.shape[1], k.shape[1]
  outs = []
  for h in range(H):
    g = h // (H // G)
    s = (q[:, h] @ k[:, g].T) * scale
    s = s.masked_fill(~see, -math.inf)
    top = s.max(-1, keepdim=True).values
    if add_one:
      top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True) + (torch.exp(-top) if add_one else 0.0)
    outs.append((e / den) @ v[:, g])
  return torch.stack(outs, 1)


def difference(a1, a2, lam, diff, eps):
  """The two maps of each head, subtracted and normalised per head."""
  return rms(a1 - lam * a2, eps) * (1.0 - diff)


def projected(h, w, name, heads):
  y = h @ w[name].T
  if name + ".b" in w:
    y = y + w[name + ".b"]
  return y.view(h.shape[0], heads, -1)


def window_attention(h, w, m, eps):
  """Norm over all rows of q and of k, paired rotation with stretched wavelengths, a sliding window, a gate per lane."""
  T, H, G = h.shape[0], m["heads"], m["kv_heads"]
  q, k, v = projected(h, w, "q", H), projected(h, w, "k", G), projected(h, w, "v", G)
  q = (rms(q.reshape(T, -1), eps) * w["q.norm"]).view(q.shape)
  k = (rms(k.reshape(T, -1), eps) * w["k.norm"]).view(k.shape)
  q, k = rotate(q, m["rot"], True), rotate(k, m["rot"], True)
  o = attention(q, k, v, m["scale"], visible(T, window=m["mask"]["size"])).reshape(T, -1)
  return (o * sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"]


def chunk_attention(h, w, m, eps):
  """Norm per head, paired rotation, chunks, one added to the denominator, a gate per lane."""
  T, H, G = h.shape[0], m["heads"], m["kv_heads"]
  q, k, v = projected(h, w, "q", H), projected(h, w, "k", G), projected(h, w, "v", G)
  q, k = rms(q, eps) * w["q.norm"], rms(k, eps) * w["k.norm"]
  q, k = rotate(q, m["rot"], True), rotate(k, m["rot"], True)
  o = attention(q, k, v, m["scale"], visible(T, chunk=m["mask"]["size"]), add_one=True).reshape(T, -1)
  return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


def differential_attention(h, w, m, eps):
  T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
  q, k, v = projected(h, w, "q", 2 * H).view(T, H, 2, D), projected(h, w, "k", 2 * G).view(T, G, 2, D), projected(h, w, "v", G)
  q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None, None]
  a1, a2 = (attention(q[:, :, j], k[:, :, j], v, m["scale"], visible(T)) for j in (0, 1))
  lam = torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + m["diff"]
  o = difference(a1, a2, lam, m["diff"], eps) * sigmoid(h @ w["g"].T)[:, :, None]
  return o.reshape(T, -1) @ w["o"].T


# ------------------------------------------------------------------------------------------ recurrences
def causal_conv(x, w):
  """x [T, C], w [C, taps]; the last tap multiplies the current token, tokens before the first are zero."""
  T, taps = x.shape[0], w.shape[1]
  y = torch.zeros_like(x)
  for j in range(taps):
    back = taps - 1 - j
    if back < T:
      y[back:] += w[:, j] * x[:T - back]
  return y


def retention_scan(q, k, v, decay):
  """q, k [T, H, D]; v [T, H, Dv]; decay [H]."""
  S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
  out = []
  for t in range(q.shape[0]):
    S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
    out.append(torch.einsum("hkv,hk->hv", S, q[t]))
  return torch.stack(out)


def delta_scan(q, k, v, g, beta):
  """q, k [T, H, D] (unit vectors); v [T, H, Dv]; g [T, H, D] decay of every key channel; beta [T, H]."""
  S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
  out = []
  for t in range(q.shape[0]):
    S = g[t][:, :, None] * S
    u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
    S = S + k[t][:, :, None] * u[:, None, :]
    out.append(torch.einsum("hkv,hk->hv", S, q[t]))
  return torch.stack(out)


def retention(h, w, m, eps):
  T, H = h.shape[0], m["heads"]
  q, k, v = (projected(h, w, n, H) for n in ("q", "k", "v"))
  q, k = rotate(q, m["rot"], False), rotate(k, m["rot"], False) * m["dim"] ** -0.5
  o = rms(retention_scan(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)), eps).reshape(T, -1)
  return (o * silu(h @ w["g"].T)) @ w["o"].T


def gated_delta(h, w, m, eps):
  T, H, G = h.shape[0], m["heads"], m["kv_heads"]
  q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
  q, k, v = q.view(T, G, -1), k.view(T, G, -1), v.view(T, H, -1)
  q, k = unit(q) * m["dim"] ** -0.5, unit(k)
  q, k = (t.repeat_interleave(H // G, 1) for t in (q, k))
  step = softplus(h @ w["a1"].T @ w["a2"].T + w["dt_bias"]).view(T, H, -1)
  g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
  o = delta_scan(q, k, v, g, sigmoid(h @ w["b"].T))
  o = rms(o, eps) * w["norm"] * sigmoid(h @ w["g1"].T @ w["g2"].T).view(T, H, -1)
  return o.reshape(T, -1) @ w["o"].T


# ------------------------------------------------------------------------------------------ layers
def parallel(h, w, m, eps):
  left = window_attention(h, part(w, "left."), m["left"], eps)
  right = retention(h, part(w, "right."), m["right"], eps)
  return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


def parallel_2(h, w, m, eps):
  return m["left_scale"] * chunk_attention(h, part(w, "left."), m["left"], eps) + m["right_scale"] * gated_delta(h, part(w, "right."), m["right"], eps)


MIXERS = {"parallel": parallel, "attention": differential_attention, "parallel_2": parallel_2}


def dense_mlp(h, w):
  return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def token_side(x, rows, w, eps):
  """rows [T, dim]: what this layer knows about each token; a gate of the stream decides how much of it joins the stream."""
  y = (gelu_tanh(x @ w["gate"].T) * rows) @ w["proj"].T
  return rms(y, eps) * w["norm"]


def part(weights, prefix):
  return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def forward(weights, spec, tokens, layers_out=None):
  """tokens: list of ids -> logits [T, vocab]; `layers_out` (a list) collects the stream after every layer."""
  eps, dim = spec["norm"]["eps"], spec["token_side"]["dim"]
  ids = torch.tensor(tokens)
  x = weights["embed"][ids] * spec["embedding"]["scale"]
  for i, lay in enumerate(spec["layers"]):
    w = part(weights, f"l{i}.")
    x = x + w["ls1"] * MIXERS[lay["type"]](rms(x, eps) * w["norm1"], part(w, "mix."), lay["mixer"], eps)
    if lay["mlp"] is not None:
      x = x + w["ls2"] * dense_mlp(rms(x, eps) * w["norm2"], part(w, "mlp."))
    x = x + token_side(x, weights["side.embed"][ids, i * dim:(i + 1) * dim], part(w, "side."), eps)
    if layers_out is not None:
      layers_out.append(x)
  return (rms(x, eps) * weights["final.norm"]) @ weights["embed"].T
