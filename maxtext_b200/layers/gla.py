"""Gated linear attention with a decay per key channel.

Per head the layer keeps a matrix state S [Dk, Dv]; per token

  S <- diag(alpha_t) S + k_t v_t^T,     o_t = S^T q_t,     alpha_t = sigmoid(z_t)^(1 / tau),

with q scaled by Dk^-1/2 and z a low-rank projection of the layer input plus a bias. The head outputs are RMS-normalised over Dv with one
learned scale, gated with SiLU of a projection of the input, and projected back. Inference on a GPU runs the kernels behind
`ops.recurrent`; training and CPU evaluate the recurrence as written.
"""
from __future__ import annotations

import torch
import torch.nn.functional as tF

from ..ops import functional as F
from ..ops import recurrent
from .blocks import Builder
from .gdn import RecurrentState


def padded_rank(rank: int) -> int:
  """Rows the decay's down-projection takes in the fused input projection (zero rows above `rank`)."""
  return -(-int(rank) // 8) * 8


def gla_recurrent(q, k, v, log_alpha, state=None):
  """q, k, log_alpha [B,T,H,Dk] (q scaled already); v [B,T,H,Dv]; state [B,H,Dk,Dv] or None. fp32 inside. Returns (o [B,T,H,Dv], state)."""
  B, T, H, Dk = q.shape
  qf, kf, vf, al = q.float(), k.float(), v.float(), torch.exp(log_alpha.float())
  S = torch.zeros(B, H, Dk, v.shape[-1], dtype=torch.float32, device=q.device) if state is None else state.float()
  outs = []
  for t in range(T):
    S = S * al[:, t][..., None] + kf[:, t][..., None] * vf[:, t][:, :, None, :]
    outs.append(torch.einsum("bhkv,bhk->bhv", S, qf[:, t]))
  return torch.stack(outs, 1), S


class GatedLinearAttention:
  """`in_proj` packs [q (H Dk) | k (H Dk) | v (H Dv) | gate (H Dv) | decay down-projection (rank, padded)]; `decay_proj` maps the latter
  to one logit per key channel."""

  def __init__(self, b: Builder, config, name: str, heads: int, dk: int, dv: int, tau: float, decay_rank: int):
    c = config
    assert b.tp_size == 1, "gated linear attention is not split over the tensor axis"
    self.c, self.heads, self.dk, self.dv, self.tau = c, heads, dk, dv, tau
    self.rank = padded_rank(decay_rank)
    d = c.emb_dim
    ab = b.sub(*name.split("/"))
    self.in_proj = ab.sub("in_proj").linear("kernel", (d,), (2 * heads * (dk + dv) + self.rank,), ("embed", "gdn_head"))
    self.decay = ab.sub("decay_proj").linear("kernel", (self.rank,), (heads * dk,), (None, "gdn_head"))
    self.decay_bias = ab.sub("decay_proj").vector("bias", heads * dk, (None,), init="zeros")
    self.norm = ab.sub("norm").vector("scale", dv, ("norm",))
    self.out = ab.sub("out_proj").linear("kernel", (heads * dv,), (d,), ("gdn_head", "embed"))

  def make_state(self, slots: int, device) -> RecurrentState:
    return RecurrentState(slots, self.heads, self.dk, self.dv, device)

  def __call__(self, x, ctx):
    B, S, _ = x.shape
    H, dk, dv = self.heads, self.dk, self.dv
    p = F.linear(x, self.in_proj)
    st = ctx.cache if isinstance(ctx.cache, RecurrentState) else None
    if recurrent.kernels_ok(p):
      return F.linear(recurrent.gla_forward(self, p, st if st is not None else self.make_state(B, x.device).fresh(B)), self.out)
    q, k, v, z, a = torch.split(p, [H * dk, H * dk, H * dv, H * dv, self.rank], dim=-1)
    q, k, v = q.view(B, S, H, dk).float() * dk ** -0.5, k.view(B, S, H, dk), v.view(B, S, H, dv)
    logits = F.linear(a, self.decay).float() + self.decay_bias.leaf().float()
    log_alpha = (tF.logsigmoid(logits) / self.tau).view(B, S, H, dk)
    s0 = None
    if st is not None:
      s0 = st.read("rec")
      if st.new_lens is not None:                # padding neither decays nor writes
        keep = st.real(S)[..., None, None].float()
        log_alpha, k = log_alpha * keep, k.float() * keep
    o, s1 = gla_recurrent(q, k, v, log_alpha, s0)
    if st is not None:
      st.rec[st.slot_ids] = s1
    o = recurrent.gated_head_norm(o, z.view(B, S, H, dv), self.norm.leaf(), self.c.normalization_layer_epsilon).to(x.dtype)
    return F.linear(o.reshape(B, S, H * dv), self.out)
