"""Gated delta rule with a decay per key channel.

The layer of `layers.gdn` with two changes: the state's rows decay at rates of their own, from a low-rank projection of the layer input, and a
sigmoid (low-rank as well) gates the head outputs. Per value head, with q, k unit vectors and q scaled by Dk^-1/2,

  S <- diag(exp(g_t)) S,     g_t = -exp(A_log) softplus(W_a2 W_a1 x_t + dt_bias) <= 0 per key channel,
  S <- S + k_t (beta_t (v_t - S^T k_t))^T,     o_t = S^T q_t,

after a causal depthwise convolution and SiLU on q, k and v; o is RMS-normalised over Dv with one learned scale. Inference on a GPU runs the
kernels behind `ops.recurrent`; training and CPU evaluate the recurrence as written.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as tF

from ..ops import functional as F
from ..ops import recurrent
from .blocks import Builder
from .gdn import RecurrentState, l2norm


def _up8(n: int) -> int:
  return -(-int(n) // 8) * 8


@dataclass(frozen=True)
class ChannelDeltaSizes:
  """Key heads, value heads, key / value width per head, convolution taps, ranks of the decay and of the gate projection."""
  hk: int
  hv: int
  dk: int
  dv: int
  taps: int
  decay_rank: int
  gate_rank: int

  @property
  def conv_dim(self) -> int:
    return 2 * self.hk * self.dk + self.hv * self.dv

  @property
  def columns(self) -> tuple:
    """Widths of the packed input projection: q, k, v; then beta and the two low-rank inputs, each padded to a multiple of 8 rows."""
    return (self.conv_dim, _up8(self.hv), _up8(self.decay_rank), _up8(self.gate_rank))


def channel_delta_recurrent(q, k, v, g, beta, state=None):
  """q, k [B,T,H,Dk] (unit vectors, q scaled); g [B,T,H,Dk] log decays; v [B,T,H,Dv]; beta [B,T,H]. fp32. Returns (o [B,T,H,Dv], state)."""
  B, T, H, Dk = q.shape
  S = torch.zeros(B, H, Dk, v.shape[-1], dtype=torch.float32, device=q.device) if state is None else state.float()
  outs = []
  for t in range(T):
    S = S * torch.exp(g[:, t])[..., None]
    u = (v[:, t] - torch.einsum("bhkv,bhk->bhv", S, k[:, t])) * beta[:, t][..., None]
    S = S + k[:, t][..., None] * u[:, :, None, :]
    outs.append(torch.einsum("bhkv,bhk->bhv", S, q[:, t]))
  return torch.stack(outs, 1), S


class ChannelDeltaNet:
  """`in_proj` packs [q | k | v | beta | decay down-projection | gate down-projection] (`ChannelDeltaSizes.columns`)."""

  def __init__(self, b: Builder, config, name: str, sizes: ChannelDeltaSizes):
    c, s, d = config, sizes, config.emb_dim
    assert b.tp_size == 1, "the gated delta rule is not split over the tensor axis"
    self.c, self.s = c, sizes
    ab = b.sub(*name.split("/"))
    self.in_proj = ab.sub("in_proj").linear("kernel", (d,), (sum(s.columns),), ("embed", "gdn_head"))
    self.in_parts = [self.in_proj]
    self.conv = ab.sub("conv1d").table("kernel", (s.taps, 1, s.conv_dim), (None, None, "gdn_head"), init="fan_in_normal")
    self.decay = ab.sub("decay_proj").linear("kernel", (s.columns[2],), (s.hv * s.dk,), (None, "gdn_head"))
    self.dt_bias = ab.sub("decay_proj").vector("bias", s.hv * s.dk, (None,), init="ones")
    self.A_log = ab.vector("A_log", s.hv, (None,), init="log_uniform_16")
    self.gate = ab.sub("gate_proj").linear("kernel", (s.columns[3],), (s.hv * s.dv,), (None, "gdn_head"))
    self.norm = ab.sub("norm").vector("scale", s.dv, ("norm",))
    self.out = ab.sub("out_proj").linear("kernel", (s.hv * s.dv,), (d,), ("gdn_head", "embed"))

  def make_state(self, slots: int, device) -> RecurrentState:
    return RecurrentState(slots, self.s.hv, self.s.dk, self.s.dv, device, self.s.conv_dim, self.s.taps)

  def serves(self, x, ctx) -> bool:
    return recurrent.kernels_ok(x)

  def __call__(self, x, ctx, rows=None):
    B, T, _ = x.shape
    s = self.s
    p = rows[0] if rows is not None else F.linear(x, self.in_proj).view(B * T, -1)
    st = ctx.cache if isinstance(ctx.cache, RecurrentState) else None
    if self.serves(p, ctx):
      return F.linear(recurrent.channel_delta_forward(self, p, B, T, st if st is not None else self.make_state(B, x.device).fresh(B)), self.out)
    mixed, bb, a1, g1 = torch.split(p.view(B, T, -1), s.columns, dim=-1)
    hist = st.read("conv") if st is not None else torch.zeros(B, s.taps - 1, s.conv_dim, dtype=torch.float32, device=x.device)
    seq = torch.cat([hist, mixed.float()], dim=1)
    w = self.conv.leaf().float().view(s.taps, s.conv_dim)
    qkv = tF.silu(sum(seq[:, j:j + T] * w[j] for j in range(s.taps)))
    if st is not None and s.taps > 1:
      # the inputs before each row's first missing token: rows n .. n + taps - 2 of [history | new tokens]
      last = st.real(T).sum(1)[:, None] + torch.arange(s.taps - 1, device=x.device)[None]
      st.conv[st.slot_ids] = seq.gather(1, last[..., None].expand(-1, -1, s.conv_dim))
    q, k, v = torch.split(qkv, [s.hk * s.dk, s.hk * s.dk, s.hv * s.dv], dim=-1)
    q, k = (l2norm(t.view(B, T, s.hk, s.dk)).repeat_interleave(s.hv // s.hk, dim=2) for t in (q, k))
    beta = torch.sigmoid(bb[..., :s.hv].float())
    dt = tF.softplus(F.linear(a1, self.decay).float() + self.dt_bias.leaf().float()).view(B, T, s.hv, s.dk)
    g = -torch.exp(self.A_log.leaf().float())[:, None] * dt
    s0 = None
    if st is not None:
      s0 = st.read("rec")
      if st.new_lens is not None:                # padding neither decays nor writes
        keep = st.real(T)[..., None].to(g.dtype)
        g, beta = g * keep[..., None], beta * keep
    o, s1 = channel_delta_recurrent(q * s.dk ** -0.5, k, v.view(B, T, s.hv, s.dv), g, beta, s0)
    if st is not None:
      st.rec[st.slot_ids] = s1
    z = F.linear(g1, self.gate).view(B, T, s.hv, s.dv)
    o = recurrent.gated_head_norm(o, z, self.norm.leaf(), self.c.normalization_layer_epsilon, "sigmoid").to(x.dtype)
    return F.linear(o.reshape(B, T, -1), self.out)
