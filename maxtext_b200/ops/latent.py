"""Latent attention at inference: projection epilogue, cache write, prefill and decode attention.

A token caches its normalised latent c [R] and one rotated key part [dr] shared by all heads. Prefill expands the latents to keys and
values (one GEMM) and runs the flash kernel. A decode step stays in the latent space: with W_uk, W_uv the per-head blocks of `wkv_b`,

  q_nope . (W_uk c) = (W_uk^T q_nope) . c        and        sum_j p_j (W_uv c_j) = W_uv (sum_j p_j c_j),

so all heads attend to the same [R + dr] vectors and a step reads each cached vector of the window once. On a GPU this is three
kernels (`csrc/latent_attention_sm100.cu`): absorb W_uk and rotate, attend (split over the keys), merge and apply W_uv. On CPU the
definition is evaluated. Padding tokens of a right-padded batch (`cache.new_lens`) never enter the cache.
"""
from __future__ import annotations

import torch

from . import backend, functional as F, reference as ref

FAR = 1 << 30            # position of a key slot that holds nothing: after every query, so the causal mask removes it


def _kernels(t: torch.Tensor) -> bool:
  return not torch.is_grad_enabled() and t.dtype in (torch.bfloat16, torch.float32) and backend.use_cuda_kernels(t)


def prep(qa, kva, mla, ctx):
  """qa [B,S,q_rank] or None, kva [B,S,R+dr] -> (normed query latent or None, c [B,S,R], rotated key part [B,S,dr]); the last two are
  also written to the cache rows that follow what each sequence already holds."""
  cache = ctx.cache
  B, S, _ = kva.shape
  R, dr = mla.kv_rank, mla.rope_d
  if _kernels(kva):
    N = B * S
    cq = torch.empty(B, S, mla.q_rank, dtype=kva.dtype, device=kva.device) if qa is not None else None
    lat = torch.empty(B, S, R, dtype=kva.dtype, device=kva.device)
    kr = torch.empty(B, S, dr, dtype=kva.dtype, device=kva.device)
    backend.ext().mla_prep(qa.view(N, -1) if qa is not None else None, mla.q_norm.scale.data if qa is not None else None, kva.view(N, -1),
                           mla.kv_norm.scale.data, float(mla.kv_norm.eps), ctx.positions.contiguous(), mla.inv_ts, bool(mla.interleaved),
                           cq.view(N, -1) if cq is not None else None, lat.view(N, R), kr.view(N, dr), cache.latent, cache.k_rope,
                           cache.slot_ids, cache.lengths, cache.new_lens)
    return cq, lat, kr
  cq = mla.q_norm(qa) if qa is not None else None
  lat = mla.kv_norm(kva[..., :R].contiguous())
  kr = F.rope(kva[..., R:].reshape(B, S, 1, dr), ctx.positions, mla.inv_ts, mla.interleaved).reshape(B, S, dr)
  cache.write(lat, kr)
  return cq, lat, kr


def _flash_widths(qk: int, vd: int):
  """Head widths (query/key, value) of the smallest flash variant that holds a head, or None."""
  for dq, dv in ((64, 64), (128, 128), (192, 128)):
    if qk <= dq and vd <= dv:
      return dq, dv
  return None


def attend_expanded(q, lat, kr, mla, ctx, kv_positions=None):
  """q [B,S,H,nope+dr] (not rotated yet) over keys expanded from lat [B,K,R] and kr [B,K,dr]. Without `kv_positions` the keys are
  the queries' own tokens; with it [B,K] they are any cached tokens (`FAR` marks an empty place)."""
  B, S, H, _ = q.shape
  K = lat.shape[1]
  kv = F.linear(lat, mla.wkv_b).view(B, K, H, mla.nope + mla.vd)
  seg = ctx.segment_ids if kv_positions is None else None
  widths = _flash_widths(mla.qk, mla.vd)
  if _kernels(q) and q.dtype == torch.bfloat16 and widths is not None:
    dq, dv = widths
    E = backend.ext()
    qp = torch.empty(B, S, H, dq, dtype=q.dtype, device=q.device)
    kp = torch.empty(B, K, H, dq, dtype=q.dtype, device=q.device)
    vp = torch.empty(B, K, H, dv, dtype=q.dtype, device=q.device)
    E.mla_pack(q.reshape(B * S, H, mla.qk), kv.view(B * K, H, mla.nope + mla.vd), kr.reshape(B * K, mla.rope_d), ctx.positions.contiguous(),
               mla.inv_ts, bool(mla.interleaved), mla.nope, mla.vd, qp.view(B * S, H, dq), kp.view(B * K, H, dq), vp.view(B * K, H, dv))
    out = F.attention(qp, kp, vp, ctx.positions, seg, mla.softmax_scale, 0.0, mla.window, kv_positions=kv_positions)
    return out[..., :mla.vd] if dv != mla.vd else out
  qr = F.rope(q[..., mla.nope:].contiguous(), ctx.positions, mla.inv_ts, mla.interleaved)
  q = torch.cat([q[..., :mla.nope], qr], -1)
  k = torch.cat([kv[..., :mla.nope], kr[:, :, None, :].expand(B, K, H, mla.rope_d)], dim=-1)
  return F.attention(q, k, kv[..., mla.nope:].contiguous(), ctx.positions, seg, mla.softmax_scale, 0.0, mla.window, kv_positions=kv_positions)


def decode(q, mla, cache, ctx):
  """One new token per sequence (its own latent is in the cache already): q [B,H,nope+dr] -> [B,H,vd]."""
  E = backend.ext()
  B, H = q.shape[:2]
  R, dr = mla.kv_rank, mla.rope_d
  qa = torch.empty(B, H, R + dr, dtype=q.dtype, device=q.device)
  w = mla.wkv_b.data
  E.mla_absorb(q.contiguous(), w, ctx.positions.reshape(-1).contiguous(), mla.inv_ts, bool(mla.interleaved), mla.nope, mla.vd, qa)
  span = min(cache.max_len, mla.window) if mla.window > 0 else cache.max_len
  splits = E.mla_decode_splits(B, H, span)
  part = torch.empty(B, H, splits, R, dtype=torch.float32, device=q.device)
  ml = torch.empty(B, H, splits, 2, dtype=torch.float32, device=q.device)
  E.mla_decode_attn(qa, cache.latent, cache.k_rope, cache.slot_ids, cache.lengths, float(mla.softmax_scale), int(mla.window), splits, part, ml)
  out = torch.empty(B, H, mla.vd, dtype=q.dtype, device=q.device)
  E.mla_value_up(part, ml, w, mla.nope, out)
  return out


def attend_cached(q, lat, kr, mla, cache, ctx):
  """q [B,S,H,nope+dr]; lat / kr of the S new tokens, which the cache holds by now."""
  B, S = q.shape[:2]
  if S == 1 and _kernels(q):
    return decode(q[:, 0], mla, cache, ctx)[:, None]
  if ctx.mode == "prefill":
    return attend_expanded(q, lat, kr, mla, ctx)                          # nothing was cached before this call
  # a later portion of a prompt: the cached tokens it can see (the window before it, or everything) and its own
  if mla.window > 0:
    idx = cache.lengths[:, None] - (mla.window - 1) + torch.arange(mla.window - 1 + S, device=q.device)[None]
  else:
    idx = torch.arange(int((cache.lengths.max() + S).item()), device=q.device)[None].expand(B, -1)
  kv_pos = torch.where((idx < 0) | (idx >= (cache.lengths + S)[:, None]), torch.full_like(idx, FAR), idx)
  rows = idx.clamp(0, cache.max_len - 1)
  slots = cache.slot_ids[:, None].expand_as(rows)
  return attend_expanded(q, cache.latent[slots, rows], cache.k_rope[slots, rows], mla, ctx, kv_positions=kv_pos)
