"""Inference kernels of the recurrent layers (gated delta network, gated linear attention, retention, channel-wise gated delta rule):
`csrc/recurrent_sm100.cu`, `csrc/recurrent_chunk_sm100.cu`.

All of them keep a matrix state per head; the kernels take the layer's raw projections and return its gated, normalised head outputs
[B, S, H * Dv] ready for the output projection. One token per sequence is one fused launch (convolution, gates, state update,
read-out, norm); longer inputs run convolution -> recurrence -> norm. States are read and written in the rows `slot_ids` of the
layer's `RecurrentState`; rows with `lengths` 0 start from zero, and only the first `new_lens` tokens of a row count.
"""
from __future__ import annotations

import torch

from . import backend


def kernels_ok(t: torch.Tensor) -> bool:
  return not torch.is_grad_enabled() and t.dtype in (torch.bfloat16, torch.float32) and backend.use_cuda_kernels(t)


CHUNK_FROM = 24          # tokens from which the chunked kernels replace the token scan


def chunked_ok(t: torch.Tensor, S: int, dk: int, dv: int) -> bool:
  """bf16 prompts run chunk by chunk on the tensor cores; fp32, very short inputs and unusual head widths run the token scan."""
  return t.dtype == torch.bfloat16 and S >= CHUNK_FROM and backend.ext().chunk_supported(dk, dv)


def gated_head_norm(o, z, scale, eps, gate="silu"):
  """Definition: o [.., H, Dv] RMS-normalised over Dv, times scale (None: no weight), times silu(z) or sigmoid(z); fp32."""
  o = o.float()
  o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
  if scale is not None:
    o = o * scale.float()
  return o * (torch.nn.functional.silu(z.float()) if gate == "silu" else torch.sigmoid(z.float()))


def delta_forward(layer, qkvz, ba, st):
  """layer: GatedDeltaNet; qkvz [B,S,hk*(2dk+2r dv)], ba [B,S,2hv]."""
  B, S, _ = qkvz.shape
  E = backend.ext()
  N = B * S
  dev, dt = qkvz.device, qkvz.dtype
  eps = float(layer.c.normalization_layer_epsilon)
  out = torch.empty(B, S, layer.value_dim, dtype=dt, device=dev)
  q2, b2 = qkvz.view(N, -1), ba.reshape(N, -1)
  w = layer.conv.data.view(layer.K, layer.conv_dim)
  if S == 1:
    E.delta_decode(q2, b2, w, layer.A_log.data, layer.dt_bias.data, layer.norm.data, eps, layer.hk, layer.hv, layer.dk, layer.dv, st.conv,
                   st.rec, st.slot_ids, st.lengths, out.view(N, -1))
    return out
  mixed = torch.empty(N, layer.conv_dim, dtype=dt, device=dev)
  E.delta_conv(q2, w, layer.hk, layer.hv, layer.dk, layer.dv, S, st.conv, st.slot_ids, st.lengths, st.new_lens, mixed)
  o = torch.empty(N, layer.value_dim, dtype=dt, device=dev)
  scan = E.delta_chunks if chunked_ok(mixed, S, layer.dk, layer.dv) else E.delta_scan
  scan(mixed, b2, layer.A_log.data, layer.dt_bias.data, layer.hk, layer.hv, layer.dk, layer.dv, S, st.rec, st.slot_ids, st.lengths, st.new_lens, o)
  r = layer.r
  E.gated_head_norm(o, q2, layer.hv, layer.dv, r, 2 * layer.dk + r * layer.dv, 2 * layer.dk + 2 * r * layer.dv, layer.norm.data, eps,
                    out.view(N, -1))
  return out


def gla_forward(layer, p, st):
  """layer: GatedLinearAttention; p [B,S,2H(dk+dv)+rank]."""
  B, S, _ = p.shape
  E = backend.ext()
  N = B * S
  H, dk, dv = layer.heads, layer.dk, layer.dv
  eps = float(layer.c.normalization_layer_epsilon)
  out = torch.empty(B, S, H * dv, dtype=p.dtype, device=p.device)
  p2 = p.view(N, -1)
  if S == 1:
    E.gla_decode(p2, layer.decay.data, layer.decay_bias.data, layer.norm.data, eps, layer.tau, H, dk, dv, st.rec, st.slot_ids, st.lengths,
                 out.view(N, -1))
    return out
  log_alpha = torch.empty(N, H * dk, dtype=torch.float32, device=p.device)
  E.gla_decay(p2, 2 * H * (dk + dv), layer.decay.data, layer.decay_bias.data, layer.tau, log_alpha)
  o = torch.empty(N, H * dv, dtype=p.dtype, device=p.device)
  scan = E.gla_chunks if chunked_ok(p2, S, dk, dv) else E.gla_scan
  scan(p2, log_alpha, H, dk, dv, S, st.rec, st.slot_ids, st.lengths, st.new_lens, o)
  E.gated_head_norm(o, p2, H, dv, 1, 2 * H * dk + H * dv, dv, layer.norm.data, eps, out.view(N, -1))
  return out


def retention_forward(layer, p, B, S, st):
  """layer: Retention; p [B*S, >= 2H(dk+dv)] rows of the input projection."""
  E = backend.ext()
  H, dk, dv = layer.heads, layer.dk, layer.dv
  eps = float(layer.c.normalization_layer_epsilon)
  out = torch.empty(B * S, H * dv, dtype=p.dtype, device=p.device)
  turn = (layer.log_decay, layer.inv_ts, layer.rot)
  if S == 1:
    E.retention_decode(p, *turn, eps, H, dk, dv, st.rec, st.slot_ids, st.lengths, out)
    return out.view(B, S, -1)
  o = torch.empty(B * S, H * dv, dtype=p.dtype, device=p.device)
  chunked = chunked_ok(p, S, dk, dv) and p.stride(0) % 8 == 0 and p.data_ptr() % 16 == 0
  (E.retention_chunks if chunked else E.retention_scan)(p, *turn, H, dk, dv, S, st.rec, st.slot_ids, st.lengths, st.new_lens, o)
  E.gated_head_norm(o, p, H, dv, 1, 2 * H * dk + H * dv, dv, None, eps, out)
  return out.view(B, S, -1)


def channel_delta_forward(layer, p, B, S, st):
  """layer: ChannelDeltaNet; p [B*S, >= sum(columns)] rows of the input projection."""
  from . import functional as F
  E, s = backend.ext(), layer.s
  N, dev, dt = B * S, p.device, p.dtype
  eps = float(layer.c.normalization_layer_epsilon)
  qkv, beta, a1, g1 = torch.split(p, s.columns, dim=-1)
  # the decay's fp32 accumulators go straight into softplus
  da = F.mm(a1, layer.decay.data, False, True, out_dtype=torch.float32)
  z = F.mm(g1, layer.gate.data, False, True)
  out = torch.empty(N, s.hv * s.dv, dtype=dt, device=dev)
  w = layer.conv.data.view(s.taps, s.conv_dim)
  if S == 1:
    E.channel_delta_decode(qkv, beta, w, da, layer.A_log.data, layer.dt_bias.data, z, layer.norm.data, eps, s.hk, s.hv, s.dk, s.dv, st.conv, st.rec,
                           st.slot_ids, st.lengths, out)
    return out.view(B, S, -1)
  mixed = torch.empty(N, s.conv_dim, dtype=dt, device=dev)
  E.ssm_conv(qkv, w, None, S, st.conv, st.slot_ids, st.lengths, st.new_lens, mixed)
  o = torch.empty(N, s.hv * s.dv, dtype=dt, device=dev)
  E.channel_delta_scan(mixed, beta, da, layer.A_log.data, layer.dt_bias.data, s.hk, s.hv, s.dk, s.dv, S, st.rec, st.slot_ids, st.lengths, st.new_lens, o,
                       chunked_ok(mixed, S, s.dk, s.dv) and s.conv_dim % 8 == 0)
  E.gated_head_norm(o, z, s.hv, s.dv, 1, 0, s.dv, layer.norm.data, eps, out, True)
  return out.view(B, S, -1)
