"""Retention (Sun et al., "Retentive Network: A Successor to Transformer for Large Language Models"): linear attention with a fixed decay per
head and no softmax or denominator.

q and k are rotated by their position; per head the layer keeps a matrix state S [Dk, Dv] and does, per token,

  S <- decay S + Dk^-1/2 k_t v_t^T,     o_t = S^T q_t.

The head outputs are RMS-normalised over Dv without a weight, gated with SiLU of a projection of the layer input, and projected back.
Inference on a GPU runs the kernels behind `ops.recurrent`; training and CPU evaluate the recurrence as written.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops import functional as F
from ..ops import recurrent
from ..ops import reference as ref
from .blocks import Builder
from .gdn import RecurrentState
from .gla import gla_recurrent


@dataclass(frozen=True)
class RetentionSizes:
  """Heads, key / value width per head, rotated lanes and their base, one decay per head."""
  heads: int
  dk: int
  dv: int
  rot: int
  base: float
  decay: tuple


class Retention:
  """`in_proj` packs [q (H Dk) | k (H Dk) | v (H Dv) | gate (H Dv)]."""

  def __init__(self, b: Builder, config, name: str, sizes: RetentionSizes, device):
    c = config
    assert b.tp_size == 1, "retention is not split over the tensor axis"
    self.c, self.heads, self.dk, self.dv, self.rot = c, sizes.heads, sizes.dk, sizes.dv, sizes.rot
    self.inv_ts = ref.rope_inv_timescale(self.rot, 1.0, sizes.base).to(device) if self.rot else None
    self.log_decay = torch.log(torch.tensor(sizes.decay, dtype=torch.float64)).float().to(device)
    d = c.emb_dim
    ab = b.sub(*name.split("/"))
    self.in_proj = ab.sub("in_proj").linear("kernel", (d,), (2 * self.heads * (self.dk + self.dv),), ("embed", "gdn_head"))
    self.in_parts = [self.in_proj]
    self.out = ab.sub("out_proj").linear("kernel", (self.heads * self.dv,), (d,), ("gdn_head", "embed"))

  def make_state(self, slots: int, device) -> RecurrentState:
    return RecurrentState(slots, self.heads, self.dk, self.dv, device)

  def serves(self, x, ctx) -> bool:
    return recurrent.kernels_ok(x)

  def __call__(self, x, ctx, rows=None):
    B, S, _ = x.shape
    H, dk, dv = self.heads, self.dk, self.dv
    p = rows[0] if rows is not None else F.linear(x, self.in_proj).view(B * S, -1)
    st = ctx.cache if isinstance(ctx.cache, RecurrentState) else None
    if self.serves(p, ctx):
      return F.linear(recurrent.retention_forward(self, p, B, S, st if st is not None else self.make_state(B, x.device).fresh(B)), self.out)
    q, k, v, z = torch.split(p.view(B, S, -1), [H * dk, H * dk, H * dv, H * dv], dim=-1)
    q, k, v = q.view(B, S, H, dk).float(), k.view(B, S, H, dk).float(), v.view(B, S, H, dv)
    if self.rot:
      q, k = (ref.apply_rope(t, ctx.positions, self.inv_ts, False, self.rot) for t in (q, k))
    log_alpha = self.log_decay.view(1, 1, H, 1).expand(B, S, H, dk)
    s0 = None
    if st is not None:
      s0 = st.read("rec")
      if st.new_lens is not None:                # padding neither decays nor writes
        keep = st.real(S)[..., None, None].float()
        log_alpha, k = log_alpha * keep, k * keep
    o, s1 = gla_recurrent(q * dk ** -0.5, k, v, log_alpha, s0)
    if st is not None:
      st.rec[st.slot_ids] = s1
    o = recurrent.gated_head_norm(o, z.view(B, S, H, dv), None, self.c.normalization_layer_epsilon).to(x.dtype)
    return F.linear(o.reshape(B, S, H * dv), self.out)
