"""Selective scan (Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces").

A causal depthwise convolution with bias and SiLU forms x from one half of the input projection; a second projection of x gives a
low-rank step size and two vectors b and c of the state width. A channel with input u, step size d and state vector s then does, in fp32,

  s <- exp(d alpha) * s + (d u) b,      y = <s, c> + skip u,

alpha = -exp(A_log) being the channel's row of decay rates and d the softplus of its low-rank projection plus bias; SiLU of the other half of the
input projection gates y.
Inference on a GPU runs the kernels behind `ops.ssm`; training and CPU evaluate the recurrence as written.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as tF

from ..ops import functional as F
from ..ops import ssm
from .blocks import Builder
from .gdn import RecurrentState


def _up8(n: int) -> int:
  return -(-int(n) // 8) * 8


@dataclass(frozen=True)
class ScanSizes:
  """Channels, state width, rank of the step-size projection, convolution taps."""
  inner: int
  state: int
  rank: int
  taps: int

  @property
  def rank_padded(self) -> int:
    """Rows of the step size in `x_proj` (zero rows above `rank`), a multiple of 8 so that products on them stay aligned."""
    return _up8(self.rank)

  @property
  def proj_rows(self) -> int:
    return _up8(self.rank_padded + 2 * self.state)


def selective_scan(x, dt, A, B, C, D, state=None):
  """x, dt [b,T,c]; A [c,n]; B, C [b,T,n]; D [c]; state [b,c,n] or None. fp32 inside. Returns (y [b,T,c], state)."""
  S = torch.zeros(x.shape[0], x.shape[2], A.shape[1], dtype=torch.float32, device=x.device) if state is None else state.float()
  outs = []
  for t in range(x.shape[1]):
    S = torch.exp(dt[:, t, :, None] * A) * S + (dt[:, t] * x[:, t])[..., None] * B[:, t, None, :]
    outs.append((S * C[:, t, None, :]).sum(-1))
  return torch.stack(outs, 1) + D * x, S


class SelectiveScan:
  """`in_proj` packs [x | z]; `x_proj` packs [step size (rank, padded) | B | C | padding]; `dt_proj` expands the step size to the channels."""

  def __init__(self, b: Builder, config, name: str, sizes: ScanSizes):
    c = config
    assert b.tp_size == 1, "the selective scan is not split over the tensor axis"
    self.c, self.s = c, sizes
    d, s = c.emb_dim, sizes
    ab = b.sub(*name.split("/"))
    self.in_proj = ab.sub("in_proj").linear("kernel", (d,), (2 * s.inner,), ("embed", "gdn_head"))
    self.conv = ab.sub("conv1d").table("kernel", (s.taps, 1, s.inner), (None, None, "gdn_head"), init="fan_in_normal")
    self.conv_bias = ab.sub("conv1d").vector("bias", s.inner, ("gdn_head",), init="zeros")
    self.x_proj = ab.sub("x_proj").linear("kernel", (s.inner,), (s.proj_rows,), ("gdn_head", None))
    self.dt_proj = ab.sub("dt_proj").linear("kernel", (s.rank_padded,), (s.inner,), (None, "gdn_head"))
    self.dt_bias = ab.sub("dt_proj").vector("bias", s.inner, ("gdn_head",), init="zeros")
    self.A_log = ab.table("A_log", (s.inner, s.state), ("gdn_head", None), init="log_uniform_16")
    self.D = ab.vector("D", s.inner, ("gdn_head",), init="ones")
    self.out = ab.sub("out_proj").linear("kernel", (s.inner,), (d,), ("gdn_head", "embed"))

  def make_state(self, slots: int, device) -> RecurrentState:
    return RecurrentState(slots, 1, self.s.inner, self.s.state, device, self.s.inner, self.s.taps)

  def __call__(self, h, ctx):
    b, T, _ = h.shape
    s = self.s
    p = F.linear(h, self.in_proj)
    st = ctx.cache if isinstance(ctx.cache, RecurrentState) else None
    if ssm.kernels_ok(p):
      return F.linear(ssm.forward(self, p, st if st is not None else self.make_state(b, h.device).fresh(b)), self.out)
    x, z = p[..., :s.inner].float(), p[..., s.inner:]
    hist = st.read("conv") if st is not None else torch.zeros(b, s.taps - 1, s.inner, dtype=torch.float32, device=h.device)
    seq = torch.cat([hist, x], dim=1)
    w = self.conv.leaf().float().view(s.taps, s.inner)
    x = tF.silu(sum(seq[:, j:j + T] * w[j] for j in range(s.taps)) + self.conv_bias.leaf().float()).to(h.dtype)
    if st is not None and s.taps > 1:
      # the inputs before each row's first missing token: rows n .. n + taps - 2 of [history | new tokens]
      last = st.real(T).sum(1)[:, None] + torch.arange(s.taps - 1, device=h.device)[None]
      st.conv[st.slot_ids] = seq.gather(1, last[..., None].expand(-1, -1, s.inner))
    q = F.linear(x, self.x_proj)
    r, n = s.rank_padded, s.state
    dt = tF.softplus(F.linear(q[..., :r], self.dt_proj).float() + self.dt_bias.leaf().float())
    B, C = q[..., r:r + n].float(), q[..., r + n:r + 2 * n].float()
    s0 = None
    if st is not None:
      s0 = st.read("rec")[:, 0]
      if st.new_lens is not None:                # padding neither decays nor writes
        dt = dt * st.real(T)[..., None].to(dt.dtype)
    y, s1 = selective_scan(x.float(), dt, -torch.exp(self.A_log.leaf().float()), B, C, self.D.leaf().float(), s0)
    if st is not None:
      st.rec[st.slot_ids, 0] = s1
    return F.linear((y * tF.silu(z.float())).to(h.dtype), self.out)
