"""Inference kernels of the selective scan (`csrc/ssm_sm100.cu`).

The kernels take the layer's input projection [x | z] and return the gated output [b, T, inner] ready for the output projection. The
convolution (with bias and SiLU, carrying its last inputs) comes first because the step size and the vectors B, C are projections of its
result; softplus, the recurrence, the read-out, the skip and the gate are one kernel, for one token per sequence and for prompts. States are
read and written in the rows `slot_ids` of the layer's `RecurrentState`; rows with `lengths` 0 start from zero, and only the first `new_lens`
tokens of a row count.
"""
from __future__ import annotations

import torch

from . import backend, functional as F


def kernels_ok(t: torch.Tensor) -> bool:
  return not torch.is_grad_enabled() and t.dtype in (torch.bfloat16, torch.float32) and backend.use_cuda_kernels(t)


def forward(layer, p, st):
  """layer: SelectiveScan; p [b, T, 2 * inner]."""
  b, T, _ = p.shape
  E = backend.ext()
  N, s = b * T, layer.s
  p2 = p.view(N, -1)
  x = torch.empty(N, s.inner, dtype=p.dtype, device=p.device)
  E.ssm_conv(p2, layer.conv.data.view(s.taps, s.inner), layer.conv_bias.data, T, st.conv, st.slot_ids, st.lengths, st.new_lens, x)
  q = F.mm(x, layer.x_proj.data, False, True)
  # the step size's fp32 accumulators go straight into softplus
  dt = F.mm(q[:, :s.rank_padded], layer.dt_proj.data, False, True, out_dtype=torch.float32)
  y = torch.empty(N, s.inner, dtype=p.dtype, device=p.device)
  E.ssm_scan(x, p2, q, dt, layer.dt_bias.data, layer.A_log.data, layer.D.data, s.rank_padded, s.state, T, st.rec, st.slot_ids, st.lengths,
             st.new_lens, y)
  return y.view(b, T, s.inner)
