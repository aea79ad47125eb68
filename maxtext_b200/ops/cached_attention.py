"""Attention over a slot-indexed key/value cache on the inference kernels (`csrc/cached_attention_sm100.cu`).

`serve` is the whole attention part of a layer with sizes of its own (`layers.blocks.HeadSizes`): one kernel adds biases, normalises, rotates,
fills the cache and lays the operands out for what follows; prompts run the flash kernel (head widths padded to the next variant), one new
token per sequence runs the split decode kernel, and everything else (fp32, unusual widths) a plain kernel that reads the cache. Sinks,
soft caps, windows, chunks, a query temperature, a second map per head (differential attention) and a sigmoid output gate are parameters. Where
the heads mix their scores (`layer.talk`) the first kernel folds the mixing into the queries, which then meet the keys of all key heads side by side
(`wide`). `attend` is the same for layers that prepare q, k and v themselves (`inference.kvcache.LayerKVCache.attend`).
"""
from __future__ import annotations

import torch

from . import backend, functional as F

FAR = 1 << 30            # position of a key row that holds nothing: after every query, so the causal mask removes it


def kernels_ok(t: torch.Tensor) -> bool:
  return not torch.is_grad_enabled() and t.dtype in (torch.bfloat16, torch.float32) and backend.use_cuda_kernels(t)


def servable(x, layer, ctx) -> bool:
  """Can this call of a `layers.blocks.Attention` with sizes of its own run `serve`?"""
  from ..inference.kvcache import LayerKVCache
  c = ctx.cache
  return (kernels_ok(x) and type(c) is LayerKVCache and c.quant is None and c.seq_size == 1 and c.k.dtype == x.dtype and ctx.tp_size == 1
          and ctx.positions3 is None and ctx.bidir is None and layer.vn is None and (not layer.share_kv or layer.sizes is not None)
          and not (layer.qk_norm and (layer.l2_qk_norm or layer.qn.scale is None or layer.qn.offset != 0))
          and not (ctx.segment_ids is not None and (x.dtype != torch.bfloat16 or not prompt_kernel(layer))))


def flash_widths(qk: int, vd: int):
  """Head widths (query/key, value) of the smallest flash variant that holds a head, or None."""
  for dq, dv in ((64, 64), (128, 128), (192, 128)):
    if qk <= dq and vd <= dv:
      return dq, dv
  return None


def wide_flash_ok(D: int, Dv: int, scale: float) -> bool:
  return D % 8 == 0 and Dv % 8 == 0 and Dv <= 128 and scale > 0.0


def prompt_kernel(layer) -> bool:
  """Does a flash kernel hold this layer's heads?"""
  if layer.talk is not None:
    return wide_flash_ok(layer.dh, layer.dv, float(layer.query_scalar))
  return flash_widths(layer.kw, layer.dv) is not None


def attends(q, cache, ctx) -> bool:
  """Can `attend` take q [B, S, H, D] over this cache? (bf16 caches that are neither quantised nor split, no image blocks)"""
  B, S, H, D = q.shape
  return (q.dtype == torch.bfloat16 and kernels_ok(q) and cache.quant is None and cache.k.dtype == q.dtype and H % cache.k.shape[2] == 0
          and getattr(ctx, "bidir", None) is None and max(D, cache.v.shape[3]) <= 512 and (S == 1 or ctx.segment_ids is None or ctx.mode == "prefill")
          and (S == 1 or ctx.segment_ids is None or flash_widths(D, cache.v.shape[3]) is not None))


def attend(q, k, v, cache, ctx, window, soft_cap, sinks, chunk=0):
  """q [B, S, H, D] (scaled) and the S new tokens' k, v, which the cache holds by now -> [B, S, H, Dv]."""
  B, S, H, D = q.shape
  Dv = v.shape[3]
  cap, win, sk = float(soft_cap or 0.0), int(window or 0), sinks.data.to(q.dtype) if sinks is not None else None
  widths = flash_widths(D, Dv)
  if S == 1:
    out = decode(q[:, 0].contiguous(), cache, 1.0, cap, win, sk, chunk=chunk)
  elif widths is None:
    out = plain(q.reshape(B * S, H, D).contiguous(), cache, S, 1.0, cap, win, sk, chunk=chunk)
  else:
    def wide(t, n):
      return t if t.shape[3] == n else torch.nn.functional.pad(t, (0, n - t.shape[3]))
    q = wide(q, widths[0]).contiguous()
    if ctx.mode == "prefill":
      out = _flash(q, wide(k, widths[0]).contiguous(), wide(v, widths[1]).contiguous(), ctx.positions, ctx.segment_ids, 1.0, cap, win, sk, F.CAP_EXACT,
                   chunk=chunk)
    else:
      out = _portion(q, cache, ctx, 1.0, cap, win, sk, F.CAP_EXACT, D, Dv, chunk)
    out = out[..., :Dv]
  return out.reshape(B, S, H, Dv)


def _gate(o, g, H, dv, layer=None):
  """o [N, H * maps, >= dv] -> [N, H * dv]: the maps of a differential layer joined, then times sigmoid(g), one gate per lane or per head
  (g None: no gate)."""
  per_head = layer is not None and layer.gate_per_head
  if g is None and (layer is None or layer.maps == 1):
    return o[..., :dv].reshape(o.shape[0], H * dv)
  out = torch.empty(o.shape[0], H * dv, dtype=o.dtype, device=o.device)
  if layer is not None and layer.maps == 2:
    backend.ext().diff_combine(o, [p.data for p in layer.lam], float(layer.sizes.diff), float(layer.config.normalization_layer_epsilon), g, dv, out, per_head)
  else:
    backend.ext().head_gate(o, g, dv, out, per_head)
  return out


def serve(layer, q, k, v, g, ctx):
  """q [N, H*maps*D], k [N, G*maps*D], v [N, G*Dv] rows of the projections (no bias, not rotated yet), g the logits of the gate or None
  -> [N, H*Dv]."""
  E, cache = backend.ext(), ctx.cache
  B, S = ctx.positions.shape
  N, H, G, D, Dv, maps = B * S, layer.hq_l, layer.hkv_l, layer.dh, layer.dv, layer.maps
  bf = q.dtype == torch.bfloat16
  scale, cap, win, chunk = float(layer.query_scalar or 1.0) * layer.logit_scale, float(layer.soft_cap), int(layer.window), int(layer.chunk)
  sinks = layer.sink_data(q.dtype)
  rot = (int(layer.rotary_dim or D) if layer.use_rope else 0)
  bias = [b.data if b is not None else None for b in (layer.bq, layer.bk, layer.bv)]
  norms = (layer.qn.scale.data, layer.kn.scale.data) if layer.qk_norm else (None, None)
  eps = float(layer.config.normalization_layer_epsilon) if layer.l2_qk_norm or layer.qk_norm else -1.0
  temp = layer.q_temp or (0.0, 0.0)
  if layer.talk is not None:
    return _serve_mixed(layer, q, k, v, ctx, scale, win, chunk, sinks, rot, eps, bias, norms, temp)
  kw = layer.kw                                          # width of a cached key: the maps' keys side by side
  widths = flash_widths(kw, Dv) if bf and S > 1 else None
  # two maps whose keys are too wide together run the flash kernel one after the other
  apart = flash_widths(D, Dv) if bf and S > 1 and maps == 2 and widths is None and ctx.mode == "prefill" else None
  fresh = ctx.mode == "prefill"
  dq, dvp = widths or (kw, apart[1] if apart is not None else Dv)
  pack_k = (widths is not None or apart is not None) and fresh         # later portions read their keys from the cache
  qp = torch.empty(N, H * maps, dq, dtype=q.dtype, device=q.device)
  kp = torch.empty(N, G, dq, dtype=q.dtype, device=q.device) if pack_k else None
  copy_v = pack_k and (dvp != Dv or bias[2] is not None or v.stride(0) % 8 != 0 or v.data_ptr() % 16 != 0)
  vp = torch.empty(N, G, dvp, dtype=q.dtype, device=q.device) if copy_v else None
  E.qkv_prep(q, k, v, D, Dv, ctx.positions.contiguous(), layer.inv_ts if rot else None, rot, eps, qp, kp, vp, cache.k, cache.v, cache.slot_ids,
             cache.lengths, cache.new_lens, *bias, *norms, layer.interleaved, maps, *temp)
  if S == 1:
    return decode(qp, cache, scale, cap, win, sinks, g, chunk, layer)
  if apart is not None:
    vs = vp.view(B, S, G, dvp) if vp is not None else _rows(v, B, S, G, Dv)
    o = torch.stack([_flash(*(torch.nn.functional.pad(t, (0, apart[0] - D)).contiguous() for t in (
        qp[:, m::2, m * D:(m + 1) * D].reshape(B, S, H, D), kp[:, :, m * D:(m + 1) * D].reshape(B, S, G, D))), vs, ctx.positions, ctx.segment_ids, scale, cap,
                            win, sinks, F.CAP_EXACT, chunk=chunk) for m in (0, 1)], 3)
    return _gate(o.reshape(N, H * maps, dvp), g, H, Dv, layer)
  if widths is None:
    return plain(qp, cache, S, scale, cap, win, sinks, g, chunk, layer)
  # normalised q and k bound every score by D * scale
  mode = F.CAP_SMALL if layer.l2_qk_norm and D * abs(scale) <= 0.3 * cap else F.CAP_EXACT
  if fresh:
    o = _flash(qp.view(B, S, H * maps, dq), kp.view(B, S, G, dq), vp.view(B, S, G, dvp) if vp is not None else _rows(v, B, S, G, Dv), ctx.positions,
               ctx.segment_ids, scale, cap, win, sinks, mode, chunk=chunk)
  else:
    o = _portion(qp.view(B, S, H * maps, dq), cache, ctx, scale, cap, win, sinks, mode, kw, Dv, chunk)
  return _gate(o.view(N, H * maps, dvp), g, H, Dv, layer)


def _serve_mixed(layer, q, k, v, ctx, scale, win, chunk, sinks, rot, eps, bias, norms, temp):
  """`serve` for heads that mix their scores."""
  E, cache = backend.ext(), ctx.cache
  B, S = ctx.positions.shape
  N, H, G, D, Dv = B * S, layer.hq_l, layer.hkv_l, layer.dh, layer.dv
  flash = q.dtype == torch.bfloat16 and S > 1 and prompt_kernel(layer)
  fresh = ctx.mode == "prefill"
  qp = torch.empty(N, H, G * D, dtype=q.dtype, device=q.device)
  kp = torch.empty(N, G, D, dtype=q.dtype, device=q.device) if flash and fresh else None
  copy_v = flash and fresh and (bias[2] is not None or v.stride(0) % 8 != 0 or v.data_ptr() % 16 != 0)
  vp = torch.empty(N, G, Dv, dtype=q.dtype, device=q.device) if copy_v else None
  E.qkv_prep(q, k, v, D, Dv, ctx.positions.contiguous(), layer.inv_ts if rot else None, rot, eps, qp, kp, vp, cache.k, cache.v, cache.slot_ids,
             cache.lengths, cache.new_lens, *bias, *norms, layer.interleaved, 1, *temp, talk=layer.talk.data)
  if S == 1 and decode_widths_ok(D, Dv, q.dtype) and wide_decode_ok(G, D, Dv):
    splits = E.cached_decode_splits(B, H, 1, min(x for x in (cache.max_len, win, chunk) if x > 0))
    part = torch.empty(B, H, splits, Dv, dtype=torch.float32, device=q.device)
    ml = torch.empty(B, H, splits, 2, dtype=torch.float32, device=q.device)
    out = torch.empty(B, H * Dv, dtype=q.dtype, device=q.device)
    E.wide_decode(qp, cache.k, cache.v, cache.slot_ids, cache.lengths, scale, win, chunk, sinks, splits, part, ml, out)
    return out
  out = torch.empty(N, H * Dv, dtype=q.dtype, device=q.device)
  if not flash:
    E.wide_attention(qp, cache.k, cache.v, cache.slot_ids, cache.lengths, S, scale, win, chunk, sinks, out)
    return out
  qw = qp.view(B, S, H, G * D)
  if fresh:
    seg = F._i32(ctx.segment_ids)
    pos = F._i32(ctx.positions) if seg is not None and chunk else None
    E.wide_flash(qw, kp.view(B, S, G, D), vp.view(B, S, G, Dv) if vp is not None else _rows(v, B, S, G, Dv), out, seg, seg, pos, pos, sinks, scale, win, chunk, 0)
  else:
    kc, vc, kv_pos = _cached_rows(cache, S, win)
    E.wide_flash(qw, kc, vc, out, None, None, F._i32(ctx.positions), F._i32(kv_pos), sinks, scale, win, chunk, 0)
  return out


def wide_decode_ok(G: int, D: int, Dv: int) -> bool:
  """Do the wide queries of 16 heads and the ring fit in shared memory?"""
  w = next(x for x in (64, 128, 256) if max(D, Dv) <= x)
  return (16 * (G * -(-D // 16) * 16 + 8) + 4 * 4 * 16 * (w + 8)) * 2 <= 227 * 1024


def _rows(v, B, S, G, Dv):
  """[N, G*Dv] rows of a wider matrix as [B, S, G, Dv] without a copy."""
  return v.as_strided((B, S, G, Dv), (S * v.stride(0), v.stride(0), Dv, 1), v.storage_offset())


def _flash(q, k, v, positions, segment_ids, scale, cap, win, sinks, mode, kv_positions=None, chunk=0):
  return F.attention_fwd(q, k, v, positions, segment_ids, scale, cap, win, kv_positions=kv_positions, sinks=sinks, cap_mode=mode, chunk=chunk)[0]


def _cached_rows(cache, S, win):
  """What S new tokens per sequence can see of the cache: keys, values and their positions."""
  dev = cache.lengths.device
  if win > 0:
    idx = cache.lengths[:, None] - (win - 1) + torch.arange(win - 1 + S, device=dev)[None]
  else:
    idx = torch.arange(int((cache.lengths.max() + S).item()), device=dev)[None].expand(cache.lengths.numel(), -1)
  kv_pos = torch.where((idx < 0) | (idx >= (cache.lengths + S)[:, None]), torch.full_like(idx, FAR), idx)
  rows = idx.clamp(0, cache.max_len - 1)
  slots = cache.slot_ids[:, None].expand_as(rows)
  return cache.k[slots, rows], cache.v[slots, rows], kv_pos


def _portion(q, cache, ctx, scale, cap, win, sinks, mode, D, Dv, chunk=0):
  """Queries that follow cached tokens: the keys they can see are gathered from the cache (padded to the flash widths)."""
  B, S, H, dq = q.shape
  dvp = flash_widths(D, Dv)[1]
  k, v, kv_pos = _cached_rows(cache, S, win)
  k = torch.nn.functional.pad(k, (0, dq - D)) if dq != D else k
  v = torch.nn.functional.pad(v, (0, dvp - Dv)) if dvp != Dv else v
  return _flash(q, k, v, ctx.positions, None, scale, cap, win, sinks, mode, kv_pos, chunk)


def decode_widths_ok(D: int, Dv: int, dtype) -> bool:
  return dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0 and max(D, Dv) <= 256


def decode(q, cache, scale, cap, win, sinks, g=None, chunk=0, layer=None):
  """One new token per sequence (its own key is in the cache already): q [B, H, D] -> [B, H*Dv] (heads of a differential layer: H / 2),
  gated by sigmoid(g) if given."""
  E = backend.ext()
  B, H, D = q.shape
  G, Dv = cache.k.shape[2], cache.v.shape[3]
  if not decode_widths_ok(D, Dv, q.dtype):
    return plain(q, cache, 1, scale, cap, win, sinks, g, chunk, layer)
  span = min(x for x in (cache.max_len, win, chunk) if x > 0)
  splits = E.cached_decode_splits(B, H, G, span)
  part = torch.empty(B, H, splits, Dv, dtype=torch.float32, device=q.device)
  ml = torch.empty(B, H, splits, 2, dtype=torch.float32, device=q.device)
  maps = layer.maps if layer is not None else 1
  out = torch.empty(B, H // maps * Dv, dtype=q.dtype, device=q.device)
  diff = dict(lam=[p.data for p in layer.lam], diff=float(layer.sizes.diff), eps=float(layer.config.normalization_layer_epsilon)) if maps == 2 else {}
  E.cached_decode(q, cache.k, cache.v, cache.slot_ids, cache.lengths, scale, cap, win, sinks, g, splits, part, ml, out, chunk=chunk,
                  per_head=layer is not None and layer.gate_per_head, **diff)
  return out


def plain(q, cache, S, scale, cap, win, sinks, g=None, chunk=0, layer=None):
  """Any widths up to 512, fp32 or bf16, any number of new tokens: q [B*S, H, D] over the cache -> [B*S, H*Dv]."""
  H, Dv = q.shape[1], cache.v.shape[3]
  o = torch.empty(q.shape[0], H, Dv, dtype=q.dtype, device=q.device)
  backend.ext().cached_attention(q, cache.k, cache.v, cache.slot_ids, cache.lengths, S, scale, cap, win, sinks, o, chunk)
  return _gate(o, g, H // (layer.maps if layer is not None else 1), Dv, layer)
