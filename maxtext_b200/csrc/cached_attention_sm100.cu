// Softmax attention over a slot-indexed key/value cache at inference: [slots, max_len, G, D] keys, [slots, max_len, G, Dv] values, any head
// widths, with soft-capped scores, a per-head sink in the denominator, a sliding window or chunks, and a sigmoid output gate per lane or head.
//
//   qkv_prep   projections (plus bias) -> RMS-normalised and rotated q and k (first `rot` lanes; halves or neighbours paired; the norm after the
//              rotation without a weight, or before it with one, per head or over the whole projection), a query temperature, cache rows,
//              operands of the flash kernel
//              where heads mix their scores, s_h <- sum_g T[h, g] s_g, the mixing moves to the queries: q_h becomes one query over the keys of all
//              key heads side by side, whose part for key head c is the sum of T[h, g] q_g over the query heads g of c
//   decode     one new token per sequence: keys split over CTAs and, inside a CTA, over four warps that each stream their own 16-key tiles
//              through a cp.async ring; up to 16 query heads of a key head sit in the M position of mma.sync m16n8k16; softmax in registers,
//              weights as (high, low) bf16 pairs. No barrier between tiles. tcgen05 has no use here: a step is bound by reading the cache
//              and its 128-row accumulators would be at most one eighth full
//   merge      joins the splits, adds the sink, applies the gate
//   wide       decode for such wide queries: all query heads of a block read all key heads, whose 16-key tiles pass through the ring one head after
//              the other; each row of the weights meets the values of its own group
//   plain      fp32 arithmetic on CUDA cores over the cache, any widths up to 512 (wide queries: any) and any number of new tokens
//   head_gate  gate of the prompt path, drops the flash kernel's width padding
//   diff       differential attention: a head's two maps share the values. The cache holds the head's two keys side by side as one key, and each
//              map's query is zero over the other map's half, so that the kernels above see two query heads of ordinary grouped attention;
//              here the second result is subtracted from the first, times lambda, normalised per head, scaled and gated
#include "cached_attention.h"
#include "serving_common.cuh"
#include "warp_mma.cuh"
#include <type_traits>

namespace mt {
namespace cattn {

// cap * tanh(s / cap) from one exponential: the error is relative to cap, a few units of fp32
__device__ __forceinline__ float capped(float s, float cap, float two_over_cap) {
  return cap - __fdividef(2.f * cap, 1.f + __expf(s * two_over_cap));
}

// ------------------------------------------------------------------------------------------------ prep
// Wide queries of a token: sq [H][D] its normalised, rotated heads, st [H][H] the transposed mixing matrix. A thread forms VEC neighbouring lanes
// of eight heads at a time.
template <typename T, int VEC>
__device__ __forceinline__ void fold_heads(const PrepArgs& a, const float* sq, const float* st, long n) {
  const int grp = a.H / a.G, per = a.G * a.D / VEC, blocks = (a.H + 7) / 8, LT = blocks * 8;
  T* out = static_cast<T*>(a.qp) + n * a.H * a.G * a.D;
  for (int i = threadIdx.x; i < per * blocks; i += 128) {
    const int col = (i % per) * VEC, h0 = (i / per) * 8, c = col / a.D, d = col % a.D;
    float acc[8][VEC];
#pragma unroll
    for (int h = 0; h < 8; ++h)
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[h][e] = 0.f;
    for (int j = 0; j < grp; ++j) {
      float x[VEC], t[8];
      load_vec<VEC>(sq + (c * grp + j) * a.D + d, x);
      load_vec<8>(st + (c * grp + j) * LT + h0, t);
#pragma unroll
      for (int h = 0; h < 8; ++h)
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[h][e] = fmaf(t[h], x[e], acc[h][e]);
    }
#pragma unroll
    for (int h = 0; h < 8; ++h)
      if (h0 + h < a.H) store_vec<VEC>(out + (long)(h0 + h) * a.G * a.D + col, acc[h]);
  }
}

template <typename T>
__device__ __forceinline__ void load_talk(const PrepArgs& a, float* st) {
  const int LT = (a.H + 7) / 8 * 8;
  for (int i = threadIdx.x; i < a.H * LT; i += 128) {
    const int g = i / LT, h = i % LT;
    st[i] = h < a.H ? to_f(static_cast<const T*>(a.talk)[h * a.H + g]) : 0.f;
  }
}

// floats of shared memory in front of the mixing operands (a multiple of four)
__host__ __device__ __forceinline__ int angle_floats(int rot) { return (rot + 2 + 3) / 4 * 4; }

// One CTA per token; a warp per head and map. Lanes hold VEC neighbouring elements, ITER times.
template <typename T, int VEC, int ITER, bool TALK>
__global__ void __launch_bounds__(128)
qkv_prep_kernel(const PrepArgs a) {
  extern __shared__ __align__(16) float2 cs[];              // (cos, sin) of the rot / 2 angles
  float* sq = reinterpret_cast<float*>(cs) + angle_floats(a.rot);
  float* st = sq + (a.H * a.D + 3) / 4 * 4;
  if constexpr (TALK) load_talk<T>(a, st);
  __shared__ float red[2][4];
  const long n = blockIdx.x;
  const int b = (int)(n / a.S), s = (int)(n % a.S), half = a.rot / 2, D = a.D, HM = a.H * a.maps, GM = a.G * a.maps;
  const float p = (float)a.pos[n];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    sincosf(p * a.inv_ts[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  const float warm = a.temp_every > 0.f ? 1.f + a.temp_coef * logf(floorf((p + 1.f) / a.temp_every) + 1.f) : 1.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // raw elements of a head (with its bias), at lane offset e0
  auto raw = [&](bool key, int head, int e0, float (&x)[VEC]) {
    load_vec<VEC>(static_cast<const T*>(key ? a.k : a.q) + n * (key ? a.ldk : a.ldq) + (long)head * D + e0, x);
    const T* bias = static_cast<const T*>(key ? a.bk : a.bq);
    if (bias) {
      float y[VEC];
      load_vec<VEC>(bias + (long)head * D + e0, y);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] += y[e];
    }
  };
  float rstd_q = 1.f, rstd_k = 1.f;
  if (a.norm == NORM_ALL) {
    float ss[2] = {0.f, 0.f};
    for (int h = warp; h < HM + GM; h += 4) {
      const bool key = h >= HM;
      float t = 0.f;
#pragma unroll
      for (int it = 0; it < ITER; ++it) {
        const int e0 = (it * 32 + lane) * VEC;
        if (e0 < D) {
          float x[VEC];
          raw(key, key ? h - HM : h, e0, x);
#pragma unroll
          for (int e = 0; e < VEC; ++e) t += x[e] * x[e];
        }
      }
      if (key) ss[1] += t; else ss[0] += t;
    }
    ss[0] = warp_add(ss[0]);
    ss[1] = warp_add(ss[1]);
    if (lane == 0) { red[0][warp] = ss[0]; red[1][warp] = ss[1]; }
  }
  __syncthreads();
  if (a.norm == NORM_ALL) {
    rstd_q = rsqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / (float)(HM * D) + a.eps);
    rstd_k = rsqrtf((red[1][0] + red[1][1] + red[1][2] + red[1][3]) / (float)(GM * D) + a.eps);
  }
  const long at = a.lengths[b] + s;
  const bool keep = at < a.max_len && s < (a.new_lens ? a.new_lens[b] : (int64_t)a.S);
  const long row = a.slots[b] * a.max_len + at;
  for (int h = warp; h < HM + GM; h += 4) {
    const bool key = h >= HM;
    const int head = key ? h - HM : h;
    const T* w = a.norm >= NORM_HEAD ? static_cast<const T*>(key ? a.wk : a.wq) + (a.norm == NORM_ALL ? (long)head * D : 0) : nullptr;
    float x[ITER][VEC], ss = 0.f, r = key ? rstd_k : rstd_q;
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int e0 = (it * 32 + lane) * VEC;
      if (e0 < D) {
        raw(key, head, e0, x[it]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += x[it][e] * x[it][e];
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[it][e] = 0.f;
      }
    }
    if (a.norm == NORM_HEAD || a.norm == NORM_AFTER) r = rsqrtf(warp_add(ss) / (float)D + a.eps);   // a rotation leaves the norm as it is
    // the factor of an element in front of the rotation
    auto scaled = [&](int e0, float (&y)[VEC]) {
      float g[VEC];
      if (w) load_vec<VEC>(w + e0, g);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] *= w ? r * g[e] : r;
    };
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int e0 = (it * 32 + lane) * VEC;
      if (e0 >= D) continue;
      scaled(e0, x[it]);
      if (e0 < a.rot) {
        if (!a.paired) {
          const bool low = e0 < half;
          const int o0 = low ? e0 + half : e0 - half;
          float y[VEC];
          raw(key, head, o0, y);
          scaled(o0, y);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            const float2 c = cs[(low ? e0 : e0 - half) + e];
            x[it][e] = x[it][e] * c.x + (low ? -y[e] : y[e]) * c.y;
          }
        } else if constexpr (VEC > 1) {
#pragma unroll
          for (int e = 0; e < VEC; e += 2) {
            const float2 c = cs[(e0 + e) / 2];
            const float u = x[it][e], v = x[it][e + 1];
            x[it][e] = u * c.x - v * c.y;
            x[it][e + 1] = v * c.x + u * c.y;
          }
        } else {
          float y[VEC];
          raw(key, head, e0 ^ 1, y);
          scaled(e0 ^ 1, y);
          const float2 c = cs[e0 / 2];
          x[it][0] = x[it][0] * c.x + (e0 & 1 ? y[0] : -y[0]) * c.y;
        }
      }
      if (!key) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[it][e] *= warm;
      }
    }
    const int m = head % a.maps;                            // this map's lanes of the head
    T* dst = key ? (a.kp ? static_cast<T*>(a.kp) + (n * a.G + head / a.maps) * (TALK ? D : a.dq) : nullptr) : static_cast<T*>(a.qp) + (n * HM + head) * a.dq;
    T* cache = key && keep ? static_cast<T*>(a.kc) + (row * GM + head) * D : nullptr;
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int e0 = (it * 32 + lane) * VEC;
      if (e0 < D) {
        if (TALK && !key) store_vec<VEC>(sq + head * D + e0, x[it]);
        else if (dst) store_vec<VEC>(dst + m * D + e0, x[it]);
        if (cache) store_vec<VEC>(cache + e0, x[it]);
      }
    }
    // zeros: a query's other lanes, and what pads a key to the operand's width
    if (!TALK && dst && (key ? m == a.maps - 1 && a.dq > a.maps * D : a.dq > D)) {
      const float zero[VEC] = {};
      for (int e0 = lane * VEC; e0 < a.dq; e0 += 32 * VEC)
        if (e0 >= (m + 1) * D || (!key && e0 < m * D)) store_vec<VEC>(dst + e0, zero);
    }
  }
  if (keep || a.vp) {
    T *vc = static_cast<T*>(a.vc), *vp = static_cast<T*>(a.vp);
    for (int i = threadIdx.x * VEC; i < a.G * a.Dv; i += blockDim.x * VEC) {
      float x[VEC];
      load_vec<VEC>(static_cast<const T*>(a.v) + n * a.ldv + i, x);
      if (a.bv) {
        float y[VEC];
        load_vec<VEC>(static_cast<const T*>(a.bv) + i, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += y[e];
      }
      if (keep) store_vec<VEC>(vc + row * a.G * a.Dv + i, x);
      if (vp) store_vec<VEC>(vp + (n * a.G + i / a.Dv) * a.dvp + i % a.Dv, x);
    }
    if (vp && a.dvp > a.Dv) {
      const int pad = a.dvp - a.Dv;
      for (int i = threadIdx.x; i < a.G * pad; i += blockDim.x) vp[(n * a.G + i / pad) * a.dvp + a.Dv + i % pad] = from_f<T>(0.f);
    }
  }
  if constexpr (TALK) {
    __syncthreads();
    fold_heads<T, VEC>(a, sq, st, n);
  }
}

// The same for head widths up to 8 * LPH that are multiples of 8: LPH lanes share a head, a warp takes 32 / LPH heads at a time, and the lanes that
// rotate together meet by a shuffle. (Halves that are paired begin at a multiple of 8.)
template <typename T, int LPH, bool TALK>
__global__ void __launch_bounds__(128, TALK ? 4 : 12)
qkv_prep_wide_kernel(const PrepArgs a) {
  constexpr int VEC = 8, STEP = 4 * (32 / LPH);
  extern __shared__ __align__(16) float2 cs[];              // (cos, sin) of the rot / 2 angles
  float* sq = reinterpret_cast<float*>(cs) + angle_floats(a.rot);
  float* st = sq + a.H * a.D;
  if constexpr (TALK) load_talk<T>(a, st);
  __shared__ float red[2][4];
  const long n = blockIdx.x;
  const int b = (int)(n / a.S), s = (int)(n % a.S), half = a.rot / 2, D = a.D, HM = a.H * a.maps, GM = a.G * a.maps, all = HM + GM;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, e0 = (lane % LPH) * VEC, first = warp * (32 / LPH) + lane / LPH;
  const bool on = e0 < D;
  auto raw = [&](int h, float (&x)[VEC]) {                  // elements of head h (keys follow the queries) with their bias
    const bool key = h >= HM;
    const int head = key ? h - HM : h;
    if (on && h < all) {
      load_vec<VEC>(static_cast<const T*>(key ? a.k : a.q) + n * (key ? a.ldk : a.ldq) + (long)head * D + e0, x);
      const T* bias = static_cast<const T*>(key ? a.bk : a.bq);
      if (bias) {
        float y[VEC];
        load_vec<VEC>(bias + (long)head * D + e0, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += y[e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] = 0.f;
    }
  };
  float x[VEC];
  raw(first, x);
  const float p = (float)a.pos[n];
  const long at = a.lengths[b] + s;
  const bool keep = at < a.max_len && s < (a.new_lens ? a.new_lens[b] : (int64_t)a.S);
  const long row = a.slots[b] * a.max_len + at;
  if (keep || a.vp) {
    T *vc = static_cast<T*>(a.vc), *vp = static_cast<T*>(a.vp);
    for (int i = threadIdx.x * VEC; i < a.G * a.Dv; i += 128 * VEC) {
      float v[VEC];
      load_vec<VEC>(static_cast<const T*>(a.v) + n * a.ldv + i, v);
      if (a.bv) {
        float y[VEC];
        load_vec<VEC>(static_cast<const T*>(a.bv) + i, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] += y[e];
      }
      if (keep) store_vec<VEC>(vc + row * a.G * a.Dv + i, v);
      if (vp) store_vec<VEC>(vp + (n * a.G + i / a.Dv) * a.dvp + i % a.Dv, v);
    }
    if (vp && a.dvp > a.Dv) {
      const int pad = (a.dvp - a.Dv) / VEC;
      const float zero[VEC] = {};
      for (int i = threadIdx.x; i < a.G * pad; i += 128) store_vec<VEC>(vp + (n * a.G + i / pad) * a.dvp + a.Dv + (i % pad) * VEC, zero);
    }
  }
  for (int i = threadIdx.x; i < half; i += 128) {
    float sn, c;
    sincosf(p * a.inv_ts[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  const float warm = a.temp_every > 0.f ? 1.f + a.temp_coef * logf(floorf((p + 1.f) / a.temp_every) + 1.f) : 1.f;
  if (a.norm == NORM_ALL) {
    float sq = 0.f, sk = 0.f;
    for (int h = first; h < all; h += STEP) {
      float y[VEC], t = 0.f;
      raw(h, y);
#pragma unroll
      for (int e = 0; e < VEC; ++e) t += y[e] * y[e];
      if (h >= HM) sk += t; else sq += t;
    }
    sq = warp_add(sq);
    sk = warp_add(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  }
  __syncthreads();
  float rstd_q = 1.f, rstd_k = 1.f;
  if (a.norm == NORM_ALL) {
    rstd_q = rsqrtf((red[0][0] + red[0][1] + red[0][2] + red[0][3]) / (float)(HM * D) + a.eps);
    rstd_k = rsqrtf((red[1][0] + red[1][1] + red[1][2] + red[1][3]) / (float)(GM * D) + a.eps);
  }
  for (int h0 = 0; h0 < all; h0 += STEP) {                  // every lane takes part in the shuffles
    const int h = h0 + first;
    const bool key = h >= HM, live = on && h < all;
    const int head = key ? h - HM : h;
    float next[VEC];
    raw(h + STEP, next);
    float r = key ? rstd_k : rstd_q;
    if (a.norm == NORM_HEAD || a.norm == NORM_AFTER) {      // a rotation leaves the norm as it is
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += x[e] * x[e];
#pragma unroll
      for (int w = LPH / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
      r = rsqrtf(ss / (float)D + a.eps);
    }
    if (a.norm >= NORM_HEAD && live) {
      float g[VEC];
      load_vec<VEC>(static_cast<const T*>(key ? a.wk : a.wq) + (a.norm == NORM_ALL ? (long)head * D : 0) + e0, g);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] *= r * g[e];
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] *= r;
    }
    if (a.rot && a.paired) {
#pragma unroll
      for (int e = 0; e < VEC; e += 2) {
        if (e0 + e < a.rot) {
          const float2 c = cs[(e0 + e) / 2];
          const float u = x[e], v = x[e + 1];
          x[e] = u * c.x - v * c.y;
          x[e + 1] = v * c.x + u * c.y;
        }
      }
    } else if (a.rot) {
      const bool turn = e0 < a.rot, low = e0 < half;
      const int src = (lane & ~(LPH - 1)) | ((turn ? (low ? e0 + half : e0 - half) : e0) / VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float y = __shfl_sync(0xffffffffu, x[e], src);
        if (turn) {
          const float2 c = cs[(low ? e0 : e0 - half) + e];
          x[e] = x[e] * c.x + (low ? -y : y) * c.y;
        }
      }
    }
    const int m = head % a.maps;                            // this map's lanes of the head
    if (live) {
      if (!key) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] *= warm;
      }
      T* dst = key ? (a.kp ? static_cast<T*>(a.kp) + (n * a.G + head / a.maps) * (TALK ? D : a.dq) : nullptr) : static_cast<T*>(a.qp) + (n * HM + head) * a.dq;
      if (TALK && !key) store_vec<VEC>(sq + head * D + e0, x);
      else if (dst) store_vec<VEC>(dst + m * D + e0, x);
      if (key && keep) store_vec<VEC>(static_cast<T*>(a.kc) + (row * GM + head) * D + e0, x);
    }
    if (!TALK && h < all && (key ? a.kp && m == a.maps - 1 && a.dq > a.maps * D : a.dq > D)) {
      T* dst = key ? static_cast<T*>(a.kp) + (n * a.G + head / a.maps) * a.dq : static_cast<T*>(a.qp) + (n * HM + head) * a.dq;
      const float zero[VEC] = {};
      for (int z = e0; z < a.dq; z += LPH * VEC)
        if (z >= (m + 1) * D || (!key && z < m * D)) store_vec<VEC>(dst + z, zero);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = next[e];
  }
  if constexpr (TALK) {
    __syncthreads();
    fold_heads<T, VEC>(a, sq, st, n);
  }
}

// ------------------------------------------------------------------------------------------------ decode
struct DecodeArgs {
  const __nv_bfloat16 *q, *k, *v;      // q [B, H, D]
  const int64_t *slots, *lengths;      // lengths without the new token
  long max_len;
  int H, G, D, Dv, window, chunk, splits, head_blocks;
  float scale, cap;
  float *part, *ml;                    // part [B, H, splits, Dv], ml [B, H, splits, 2]
};

constexpr int KEYS = 16, RING = 3;     // keys of a warp's tile, tiles in flight

template <int DK, int DVT>             // widths rounded up to the template: DK, DVT multiples of 16
__global__ void __launch_bounds__(128)
decode_kernel(const DecodeArgs a) {
  constexpr int LK = DK + 8, LV = DVT + 8, TILE = KEYS * (LK + LV);
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sq = sm;                                   // [16][LK]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __nv_bfloat16* ring = sm + 16 * LK + warp * RING * TILE;
  const int split = blockIdx.x, g = blockIdx.y / a.head_blocks, hb = blockIdx.y % a.head_blocks, b = blockIdx.z;
  const int grp = a.H / a.G, h0 = g * grp + hb * 16, nh = min(16, grp - hb * 16);
  const int D16 = (a.D + 15) / 16, V16 = (a.Dv + 15) / 16;
  const long len = min(a.lengths[b] + 1, (int64_t)a.max_len);
  int first = (a.window > 0 && len > a.window) ? (int)(len - a.window) : 0;
  if (a.chunk > 0) first = max(first, (int)((len - 1) / a.chunk) * a.chunk);
  const int per = ((int)((len - first + a.splits - 1) / a.splits) + KEYS - 1) / KEYS * KEYS;
  const int lo = first + split * per, hi = (int)min((long)lo + per, len);
  const __nv_bfloat16* kb = a.k + (a.slots[b] * a.max_len * a.G + g) * a.D;
  const __nv_bfloat16* vb = a.v + (a.slots[b] * a.max_len * a.G + g) * a.Dv;
  const long ldk = (long)a.G * a.D, ldv = (long)a.G * a.Dv;
  for (int i = threadIdx.x; i < 16 * D16 * 2; i += 128) {   // 8-element pieces
    const int r = i / (D16 * 2), c = (i % (D16 * 2)) * 8;
    uint4 t = make_uint4(0, 0, 0, 0);
    if (r < nh && c < a.D) t = *reinterpret_cast<const uint4*>(a.q + ((long)b * a.H + h0 + r) * a.D + c);
    *reinterpret_cast<uint4*>(sq + r * LK + c) = t;
  }
  __syncthreads();
  const int n_tiles = hi > lo ? (hi - lo + KEYS - 1) / KEYS : 0;
  // a lane keeps its 16-byte column of a row and walks down the keys; columns beyond the width are filled with zeros once per tile
  constexpr int KP = DK / 8, VP = DVT / 8, KR = 32 / KP, VR = 32 / VP;
  const int kr = lane / KP, kcol = (lane % KP) * 8, vr = lane / VP, vcol = (lane % VP) * 8;
  const bool kin = kcol < a.D, vin = vcol < a.Dv, kpad = kcol < D16 * 16, vpad = vcol < V16 * 16;
  const __nv_bfloat16 *kp = kb + (kin ? (lo + kr) * ldk + kcol : 0), *vp = vb + (vin ? (lo + vr) * ldv + vcol : 0);
  auto load = [&](int tile, int stage) {
    __nv_bfloat16* sk = ring + stage * TILE + kr * LK + kcol;
    __nv_bfloat16* sv = ring + stage * TILE + KEYS * LK + vr * LV + vcol;
    const int left = hi - lo - tile * KEYS;
    const __nv_bfloat16 *kt = kp + (kin ? (long)tile * KEYS * ldk : 0), *vt = vp + (vin ? (long)tile * KEYS * ldv : 0);
    if (kpad) {
#pragma unroll
      for (int j = 0; j < KEYS / KR; ++j) {
        const bool ok = kin && kr + j * KR < left;
        la_cp_async16(sk + j * KR * LK, ok ? kt + j * KR * ldk : kb, ok ? 16 : 0);
      }
    }
    if (vpad) {
#pragma unroll
      for (int j = 0; j < KEYS / VR; ++j) {
        const bool ok = vin && vr + j * VR < left;
        la_cp_async16(sv + j * VR * LV, ok ? vt + j * VR * ldv : vb, ok ? 16 : 0);
      }
    }
  };
  float o[DVT / 8][4];
#pragma unroll
  for (int j = 0; j < DVT / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // rows lane / 4 and lane / 4 + 8
  const float two_over_cap = a.cap > 0.f ? 2.f / a.cap : 0.f;
  int fetch = warp;
#pragma unroll
  for (int s = 0; s < RING - 1; ++s, fetch += 4) {
    if (fetch < n_tiles) load(fetch, s);
    la_commit();
  }
  int stage = 0;
  for (int tile = warp; tile < n_tiles; tile += 4) {
    la_wait<RING - 2>();
    __syncwarp();
    if (fetch < n_tiles) load(fetch, (stage + RING - 1) % RING);
    fetch += 4;
    la_commit();
    const __nv_bfloat16* sk = ring + stage * TILE;
    const __nv_bfloat16* sv = sk + KEYS * LK;
    float s[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      if (kk < D16) {
        unsigned aq[4], bk[4];
        la_ldm4(aq, sq + (lane & 15) * LK + kk * 16 + (lane >> 4) * 8);
        la_ldm4(bk, sk + ((lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
        la_mma(s[0], aq, bk[0], bk[1]);
        la_mma(s[1], aq, bk[2], bk[3]);
      }
    }
    const int left = hi - lo - tile * KEYS;                  // keys of the tile that exist
    float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float x = s[j][e] * a.scale;
        if (a.cap > 0.f) x = capped(x, a.cap, two_over_cap);
        if (j * 8 + (lane & 3) * 2 + (e & 1) >= left) x = -INFINITY;
        s[j][e] = x;
        if (e < 2) t0 = fmaxf(t0, x); else t1 = fmaxf(t1, x);
      }
#pragma unroll
    for (int d = 1; d < 4; d <<= 1) {
      t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, d));
      t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, d));
    }
    const float n0 = fmaxf(m0, t0), n1 = fmaxf(m1, t1);      // finite: a tile holds at least one key
    if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {
      const float c0 = __expf(m0 - n0), c1 = __expf(m1 - n1);
      l0 *= c0;
      l1 *= c1;
#pragma unroll
      for (int j = 0; j < DVT / 8; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
      m0 = n0;
      m1 = n1;
    }
    unsigned ph[4], pl[4];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float p0 = __expf(s[j][0] - m0), p1 = __expf(s[j][1] - m0), p2 = __expf(s[j][2] - m1), p3 = __expf(s[j][3] - m1);
      l0 += p0 + p1;
      l1 += p2 + p3;
      __nv_bfloat162 hi2, lo2;
      la_split2(p0, p1, hi2, lo2);
      ph[2 * j] = *reinterpret_cast<unsigned*>(&hi2); pl[2 * j] = *reinterpret_cast<unsigned*>(&lo2);
      la_split2(p2, p3, hi2, lo2);
      ph[2 * j + 1] = *reinterpret_cast<unsigned*>(&hi2); pl[2 * j + 1] = *reinterpret_cast<unsigned*>(&lo2);
    }
#pragma unroll
    for (int j = 0; j < DVT / 16; ++j) {
      if (j < V16) {
        unsigned bv[4];
        la_ldm4t(bv, sv + (lane & 15) * LV + j * 16 + (lane >> 4) * 8);
        la_mma(o[2 * j], ph, bv[0], bv[1]);
        la_mma(o[2 * j], pl, bv[0], bv[1]);
        la_mma(o[2 * j + 1], ph, bv[2], bv[3]);
        la_mma(o[2 * j + 1], pl, bv[2], bv[3]);
      }
    }
    __syncwarp();
    stage = (stage + 1) % RING;
  }
  la_wait<0>();
#pragma unroll
  for (int d = 1; d < 4; d <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, d);
    l1 += __shfl_xor_sync(0xffffffffu, l1, d);
  }
  __syncthreads();
  // join the four warps: [4][16][DVT + 2] fp32 over the ring's memory
  constexpr int LO = DVT + 4;
  float* so = reinterpret_cast<float*>(sm) + warp * 16 * LO;
  const int r = lane >> 2;
#pragma unroll
  for (int j = 0; j < DVT / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) so[(r + (e >> 1) * 8) * LO + j * 8 + (lane & 3) * 2 + (e & 1)] = o[j][e];
  if ((lane & 3) == 0) {
    so[r * LO + DVT] = m0; so[r * LO + DVT + 1] = l0;
    so[(r + 8) * LO + DVT] = m1; so[(r + 8) * LO + DVT + 1] = l1;
  }
  __syncthreads();
  const float* all = reinterpret_cast<const float*>(sm);
  for (int i = threadIdx.x; i < nh * a.Dv; i += 128) {
    const int h = i / a.Dv, d = i % a.Dv;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, all[(w * 16 + h) * LO + DVT]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float c = m == -INFINITY ? 0.f : __expf(all[(w * 16 + h) * LO + DVT] - m);
      num += c * all[(w * 16 + h) * LO + d];
      den += c * all[(w * 16 + h) * LO + DVT + 1];
    }
    const long at = ((long)b * a.H + h0 + h) * a.splits + split;
    a.part[at * a.Dv + d] = num;
    if (d == 0) { a.ml[at * 2] = m; a.ml[at * 2 + 1] = den; }
  }
}

// ------------------------------------------------------------------------------------------------ decode with wide queries
struct WideArgs {
  const __nv_bfloat16 *q, *k, *v;      // q [B, H, G * D]
  const int64_t *slots, *lengths;
  long max_len;
  int H, G, D, Dv, window, chunk, splits, head_blocks;
  float scale;
  float *part, *ml;
};

constexpr int WIDE_RING = 4;           // pieces in flight per warp; a piece is 16 keys (or values) of one key head

template <int DW>                      // max(D, Dv) rounded up
__global__ void __launch_bounds__(128)
wide_decode_kernel(const WideArgs a) {
  constexpr int LW = DW + 8, PIECE = KEYS * LW, RING_ = WIDE_RING, P = DW / 8, PR = 32 / P;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int D16 = (a.D + 15) / 16, V16 = (a.Dv + 15) / 16, DP = D16 * 16, LQ = a.G * DP + 8;
  __nv_bfloat16* sq = sm;                                   // [16][LQ]
  __nv_bfloat16* ring = sm + 16 * LQ + warp * RING_ * PIECE;
  const int split = blockIdx.x, hb = blockIdx.y, b = blockIdx.z;
  const int grp = a.H / a.G, h0 = hb * 16, nh = min(16, a.H - h0), g0 = h0 / grp, pieces = a.G + (h0 + nh - 1) / grp - g0 + 1;
  const long len = min(a.lengths[b] + 1, (int64_t)a.max_len);
  int first = (a.window > 0 && len > a.window) ? (int)(len - a.window) : 0;
  if (a.chunk > 0) first = max(first, (int)((len - 1) / a.chunk) * a.chunk);
  const int per = ((int)((len - first + a.splits - 1) / a.splits) + KEYS - 1) / KEYS * KEYS;
  const int lo = first + split * per, hi = (int)min((long)lo + per, len);
  const long ldk = (long)a.G * a.D, ldv = (long)a.G * a.Dv;
  const __nv_bfloat16 *kb = a.k + a.slots[b] * a.max_len * ldk, *vb = a.v + a.slots[b] * a.max_len * ldv;
  for (int i = threadIdx.x; i < 16 * a.G * D16 * 2; i += 128) {              // 8-element pieces
    const int r = i / (a.G * D16 * 2), c = i % (a.G * D16 * 2) / (D16 * 2), d = i % (D16 * 2) * 8;
    uint4 t = make_uint4(0, 0, 0, 0);
    if (r < nh && d < a.D) t = *reinterpret_cast<const uint4*>(a.q + ((long)b * a.H + h0 + r) * ldk + c * a.D + d);
    *reinterpret_cast<uint4*>(sq + r * LQ + c * DP + d) = t;
  }
  __syncthreads();
  const int n_tiles = hi > lo ? (hi - lo + KEYS - 1) / KEYS : 0;
  const int pr = lane / P, pcol = (lane % P) * 8;           // a lane keeps its column of a piece and walks down the rows
  int f_tile = warp, f_piece = 0, f_stage = 0;
  auto fetch = [&]() {
    if (f_tile < n_tiles) {
      const bool key = f_piece < a.G;
      const int width = key ? a.D : a.Dv, left = hi - lo - f_tile * KEYS;
      if (pcol < (key ? DP : V16 * 16)) {                   // columns beyond the width are filled with zeros
        const long ld = key ? ldk : ldv;
        const __nv_bfloat16* base = key ? kb : vb;
        const __nv_bfloat16* src = base + (long)(lo + f_tile * KEYS + pr) * ld + (key ? f_piece * a.D : (g0 + f_piece - a.G) * a.Dv) + pcol;
        __nv_bfloat16* dst = ring + f_stage * PIECE + pr * LW + pcol;
#pragma unroll
        for (int j = 0; j < KEYS / PR; ++j) {
          const bool ok = pcol < width && pr + j * PR < left;
          la_cp_async16(dst + j * PR * LW, ok ? src + j * PR * ld : base, ok ? 16 : 0);
        }
      }
      if (++f_piece == pieces) { f_piece = 0; f_tile += 4; }
    }
    f_stage = f_stage + 1 == RING_ ? 0 : f_stage + 1;
    la_commit();
  };
#pragma unroll
  for (int s = 0; s < RING_ - 1; ++s) fetch();
  int stage = 0;
  auto next = [&]() {                                       // the piece that is due; its predecessor's place is refilled
    la_wait<RING_ - 2>();
    __syncwarp();
    const __nv_bfloat16* p = ring + stage * PIECE;
    fetch();
    stage = stage + 1 == RING_ ? 0 : stage + 1;
    return p;
  };
  float o[DW / 8][4];
#pragma unroll
  for (int j = 0; j < DW / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;  // rows lane / 4 and lane / 4 + 8
  const int r0 = lane >> 2, c0 = (h0 + r0) / grp, c1 = (h0 + r0 + 8) / grp;     // their groups
  for (int tile = warp; tile < n_tiles; tile += 4) {
    float s[2][4] = {};
    for (int c = 0; c < a.G; ++c) {
      const __nv_bfloat16* sk = next();
#pragma unroll
      for (int kk = 0; kk < DW / 16; ++kk) {
        if (kk < D16) {
          unsigned aq[4], bk[4];
          la_ldm4(aq, sq + (lane & 15) * LQ + c * DP + kk * 16 + (lane >> 4) * 8);
          la_ldm4(bk, sk + ((lane & 7) + ((lane >> 4) << 3)) * LW + kk * 16 + ((lane >> 3) & 1) * 8);
          la_mma(s[0], aq, bk[0], bk[1]);
          la_mma(s[1], aq, bk[2], bk[3]);
        }
      }
    }
    const int left = hi - lo - tile * KEYS;                  // keys of the tile that exist
    float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[j][e] = j * 8 + (lane & 3) * 2 + (e & 1) >= left ? -INFINITY : s[j][e] * a.scale;
        if (e < 2) t0 = fmaxf(t0, s[j][e]); else t1 = fmaxf(t1, s[j][e]);
      }
#pragma unroll
    for (int d = 1; d < 4; d <<= 1) {
      t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, d));
      t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, d));
    }
    const float n0 = fmaxf(m0, t0), n1 = fmaxf(m1, t1);      // finite: a tile holds at least one key
    if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {
      const float f0 = __expf(m0 - n0), f1 = __expf(m1 - n1);
      l0 *= f0;
      l1 *= f1;
#pragma unroll
      for (int j = 0; j < DW / 8; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
      m0 = n0;
      m1 = n1;
    }
    unsigned ph[4], pl[4];                                   // even entries: row r0, odd ones: row r0 + 8
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float p0 = __expf(s[j][0] - m0), p1 = __expf(s[j][1] - m0), p2 = __expf(s[j][2] - m1), p3 = __expf(s[j][3] - m1);
      l0 += p0 + p1;
      l1 += p2 + p3;
      __nv_bfloat162 hi2, lo2;
      la_split2(p0, p1, hi2, lo2);
      ph[2 * j] = *reinterpret_cast<unsigned*>(&hi2); pl[2 * j] = *reinterpret_cast<unsigned*>(&lo2);
      la_split2(p2, p3, hi2, lo2);
      ph[2 * j + 1] = *reinterpret_cast<unsigned*>(&hi2); pl[2 * j + 1] = *reinterpret_cast<unsigned*>(&lo2);
    }
    for (int c = g0; c < g0 + pieces - a.G; ++c) {
      const __nv_bfloat16* sv = next();
      unsigned wh[4], wl[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const bool mine = (e & 1 ? c1 : c0) == c;
        wh[e] = mine ? ph[e] : 0u;
        wl[e] = mine ? pl[e] : 0u;
      }
#pragma unroll
      for (int j = 0; j < DW / 16; ++j) {
        if (j < V16) {
          unsigned bv[4];
          la_ldm4t(bv, sv + (lane & 15) * LW + j * 16 + (lane >> 4) * 8);
          la_mma(o[2 * j], wh, bv[0], bv[1]);
          la_mma(o[2 * j], wl, bv[0], bv[1]);
          la_mma(o[2 * j + 1], wh, bv[2], bv[3]);
          la_mma(o[2 * j + 1], wl, bv[2], bv[3]);
        }
      }
    }
  }
  la_wait<0>();
#pragma unroll
  for (int d = 1; d < 4; d <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, d);
    l1 += __shfl_xor_sync(0xffffffffu, l1, d);
  }
  __syncthreads();
  // join the four warps: [4][16][DW + 4] fp32 over the whole buffer
  constexpr int LO = DW + 4;
  float* so = reinterpret_cast<float*>(sm) + warp * 16 * LO;
#pragma unroll
  for (int j = 0; j < DW / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) so[(r0 + (e >> 1) * 8) * LO + j * 8 + (lane & 3) * 2 + (e & 1)] = o[j][e];
  if ((lane & 3) == 0) {
    so[r0 * LO + DW] = m0; so[r0 * LO + DW + 1] = l0;
    so[(r0 + 8) * LO + DW] = m1; so[(r0 + 8) * LO + DW + 1] = l1;
  }
  __syncthreads();
  const float* all = reinterpret_cast<const float*>(sm);
  for (int i = threadIdx.x; i < nh * a.Dv; i += 128) {
    const int h = i / a.Dv, d = i % a.Dv;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, all[(w * 16 + h) * LO + DW]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float c = m == -INFINITY ? 0.f : __expf(all[(w * 16 + h) * LO + DW] - m);
      num += c * all[(w * 16 + h) * LO + d];
      den += c * all[(w * 16 + h) * LO + DW + 1];
    }
    const long at = ((long)b * a.H + h0 + h) * a.splits + split;
    a.part[at * a.Dv + d] = num;
    if (d == 0) { a.ml[at * 2] = m; a.ml[at * 2 + 1] = den; }
  }
}

// out [B, H * Dv] = (splits joined, sink in the denominator) * sigmoid(gate)
template <typename T>
__global__ void merge_kernel(const float* __restrict__ part, const float* __restrict__ ml, int H, int Dv, int splits, const T* __restrict__ sinks,
                             const T* __restrict__ gate, long ldg, int per_head, T* __restrict__ out) {
  const int h = blockIdx.x, b = blockIdx.y;
  const long at = ((long)b * H + h) * splits;
  float m = sinks ? to_f(sinks[h]) : -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[(at + s) * 2]);
  float den = sinks ? __expf(to_f(sinks[h]) - m) : 0.f;
  for (int s = 0; s < splits; ++s) den += ml[(at + s) * 2] == -INFINITY ? 0.f : ml[(at + s) * 2 + 1] * __expf(ml[(at + s) * 2] - m);
  const float inv = den > 0.f ? 1.f / den : 0.f;
  for (int d = threadIdx.x; d < Dv; d += blockDim.x) {
    float o = 0.f;
    for (int s = 0; s < splits; ++s)
      if (ml[(at + s) * 2] != -INFINITY) o += part[(at + s) * Dv + d] * __expf(ml[(at + s) * 2] - m);
    o *= inv;
    if (gate) o *= sigmoid_f(to_f(gate[b * ldg + (per_head ? h : (long)h * Dv + d)]));
    out[(long)b * H * Dv + (long)h * Dv + d] = from_f<T>(o);
  }
}

// ------------------------------------------------------------------------------------------------ differential attention
template <typename T>
__device__ __forceinline__ float diff_lambda(const DiffArgs& a, int lane) {
  float s1 = 0.f, s2 = 0.f;
  for (int i = lane; i < a.D; i += 32) {
    s1 += to_f(static_cast<const T*>(a.lq1)[i]) * to_f(static_cast<const T*>(a.lk1)[i]);
    s2 += to_f(static_cast<const T*>(a.lq2)[i]) * to_f(static_cast<const T*>(a.lk2)[i]);
  }
  return expf(warp_add(s1)) - expf(warp_add(s2)) + a.diff;
}

// decode: grid (heads, B), 128 threads. The maps of head h are the query heads 2 h and 2 h + 1 of `part`
template <typename T>
__global__ void __launch_bounds__(128)
diff_merge_kernel(const float* __restrict__ part, const float* __restrict__ ml, const DiffArgs a, int H, int Dv, int splits, const T* __restrict__ gate,
                  long ldg, int per_head, T* __restrict__ out) {
  __shared__ float red[4], top[4], den[4], wt[2][64];
  const int h = blockIdx.x, b = blockIdx.y, t = threadIdx.x, warp = t >> 5;
  const float lam = diff_lambda<T>(a, t & 31);
  // the weights of the splits: 64 threads per map
  const long at0 = ((long)b * 2 * H + 2 * h) * splits;
  float mx = -INFINITY, l = 0.f;
  if ((t & 63) < splits) {
    const float2 v = *reinterpret_cast<const float2*>(ml + (at0 + (t >> 6) * splits + (t & 63)) * 2);
    mx = v.x;
    l = v.y;
  }
  float wm = mx;
#pragma unroll
  for (int d = 16; d > 0; d >>= 1) wm = fmaxf(wm, __shfl_xor_sync(0xffffffffu, wm, d));
  if ((t & 31) == 0) top[warp] = wm;
  __syncthreads();
  const float c = mx == -INFINITY ? 0.f : __expf(mx - fmaxf(top[warp & 2], top[warp | 1]));
  l = warp_add(c * l);
  if ((t & 31) == 0) den[warp] = l;
  wt[t >> 6][t & 63] = c;
  __syncthreads();
  float x[2] = {0.f, 0.f};                                  // Dv up to 256
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const float* p = part + (at0 + m * splits) * Dv;
    const float sum = den[2 * m] + den[2 * m + 1], f = sum > 0.f ? (m ? -lam : 1.f) / sum : 0.f;
    float o[2] = {0.f, 0.f};
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (t + j * 128 < Dv && wt[m][s] != 0.f) o[j] += p[(long)s * Dv + t + j * 128] * wt[m][s];
    }
    x[0] += f * o[0];
    x[1] += f * o[1];
  }
  const float r = rsqrtf(block_add(x[0] * x[0] + x[1] * x[1], red) / (float)Dv + a.eps) * (1.f - a.diff);
  const T* g = gate ? gate + b * ldg + (per_head ? h : (long)h * Dv) : nullptr;
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int d = t + j * 128;
    if (d < Dv) out[((long)b * H + h) * Dv + d] = from_f<T>(x[j] * r * (g ? sigmoid_f(to_f(g[per_head ? 0 : d])) : 1.f));
  }
}

// prompts: LPR lanes per token and head, VEC neighbouring elements each, NV times; o [N, 2 H, dvp] -> out [N, H * Dv]
template <typename T, int VEC, int LPR, int NV>
__global__ void __launch_bounds__(256)
diff_combine_kernel(const T* __restrict__ o, int dvp, const DiffArgs a, long N, int H, int Dv, const T* __restrict__ gate, long ldg, int per_head,
                    T* __restrict__ out) {
  const int lane = threadIdx.x & 31, t = lane % LPR;
  const float lam = diff_lambda<T>(a, lane);
  const long rows = N * H, step = gridDim.x * (256l / LPR);
  for (long i = (blockIdx.x * 256l + threadIdx.x) / LPR; i - lane / LPR < rows; i += step) {         // a warp leaves the loop together
    const bool in = i < rows;
    const long n = in ? i / H : 0;
    const int h = in ? (int)(i % H) : 0;
    const T* o1 = o + (n * 2 * H + 2 * h) * dvp;
    float x[NV][VEC], ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = (j * LPR + t) * VEC;
      if (d < Dv) {
        float y[VEC];
        load_vec<VEC>(o1 + d, x[j]);
        load_vec<VEC>(o1 + dvp + d, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          x[j][e] -= lam * y[e];
          ss += x[j][e] * x[j][e];
        }
      }
    }
#pragma unroll
    for (int w = LPR / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    if (!in) continue;
    float r = rsqrtf(ss / (float)Dv + a.eps) * (1.f - a.diff);
    const T* g = gate ? gate + n * ldg + (per_head ? h : (long)h * Dv) : nullptr;
    if (g && per_head) r *= sigmoid_f(to_f(g[0]));
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = (j * LPR + t) * VEC;
      if (d < Dv) {
        float z[VEC];
        if (g && !per_head) load_vec<VEC>(g + d, z);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[j][e] *= g && !per_head ? r * sigmoid_f(z[e]) : r;
        store_vec<VEC>(out + i * Dv + d, x[j]);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ plain
// 16 queries of one head against tiles of 32 keys. Eight threads per query: four scores each per tile, then Dv / 8 output columns each.
constexpr int PQ = 16, PK = 32;

template <typename T, int NV>          // NV * 8 >= Dv
__global__ void __launch_bounds__(128)
plain_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long max_len, const int64_t* __restrict__ slots,
             const int64_t* __restrict__ lengths, int S, int H, int G, int D, int Dv, float scale, float cap, int window, int chunk,
             const T* __restrict__ sinks, T* __restrict__ out) {
  extern __shared__ __align__(16) float smf[];
  const int LD = D + 1, LV = Dv + 1;
  float* sq = smf;                     // [PQ][LD]
  float* sk = sq + PQ * LD;            // [PK][LD]
  float* sv = sk + PK * LD;            // [PK][LV]
  float* sp = sv + PK * LV;            // [PQ][PK + 1]
  const int s0 = blockIdx.x * PQ, h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
  const int tid = threadIdx.x, r = tid >> 3, l8 = tid & 7;
  const long base = lengths[b];
  for (int i = tid; i < PQ * D; i += 128) {
    const int t = i / D, d = i % D;
    sq[t * LD + d] = s0 + t < S ? to_f(q[(((long)b * S + s0 + t) * H + h) * D + d]) : 0.f;
  }
  const long last = min(base + min(S, s0 + PQ) - 1, max_len - 1);               // position of the last query
  const long mine = base + s0 + r;
  long firstk = window > 0 ? max(0l, base + s0 - window + 1) : 0l;
  if (chunk > 0) firstk = max(firstk, (base + s0) / chunk * chunk);
  const long from = max(window > 0 ? mine - window + 1 : 0l, chunk > 0 ? mine / chunk * chunk : 0l);      // first key this query sees
  float acc[NV], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) acc[j] = 0.f;
  for (long t0 = firstk; t0 <= last; t0 += PK) {
    __syncthreads();
    for (int i = tid; i < PK * D; i += 128) {
      const int t = i / D, d = i % D;
      sk[t * LD + d] = t0 + t <= last ? to_f(k[((slots[b] * max_len + t0 + t) * G + g) * D + d]) : 0.f;
    }
    for (int i = tid; i < PK * Dv; i += 128) {
      const int t = i / Dv, d = i % Dv;
      sv[t * LV + d] = t0 + t <= last ? to_f(v[((slots[b] * max_len + t0 + t) * G + g) * Dv + d]) : 0.f;
    }
    __syncthreads();
    float sc[4], tm = -INFINITY;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = l8 + j * 8;
      float x = 0.f;
      for (int d = 0; d < D; ++d) x = fmaf(sq[r * LD + d], sk[t * LD + d], x);
      x *= scale;
      if (cap > 0.f) x = cap * tanhf(x / cap);
      const long p = t0 + t;
      if (p > mine || p > last || p < from) x = -INFINITY;
      sc[j] = x;
      tm = fmaxf(tm, x);
    }
#pragma unroll
    for (int d = 1; d < 8; d <<= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, d));
    const float n = fmaxf(m, tm), c = n == -INFINITY ? 1.f : expf(m - n);
    m = n;
    float ts = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float p = sc[j] == -INFINITY ? 0.f : expf(sc[j] - n);
      sp[r * (PK + 1) + l8 + j * 8] = p;
      ts += p;
    }
#pragma unroll
    for (int d = 1; d < 8; d <<= 1) ts += __shfl_xor_sync(0xffffffffu, ts, d);
    l = l * c + ts;
    __syncwarp();
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = l8 + j * 8;
      if (d < Dv) {
        float o = 0.f;
        for (int t = 0; t < PK; ++t) o = fmaf(sp[r * (PK + 1) + t], sv[t * LV + d], o);
        acc[j] = acc[j] * c + o;
      }
    }
  }
  if (s0 + r >= S) return;
  float inv = 0.f;
  if (sinks) {
    const float sk_ = to_f(sinks[h]), n = fmaxf(m, sk_);
    const float c = m == -INFINITY ? 0.f : expf(m - n);
    inv = c / (l * c + expf(sk_ - n));
  } else if (l > 0.f) {
    inv = 1.f / l;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int d = l8 + j * 8;
    if (d < Dv) out[(((long)b * S + s0 + r) * H + h) * Dv + d] = from_f<T>(acc[j] * inv);
  }
}

// The same for wide queries, q [B * S, H, G * D] against the keys of all key heads side by side; the contraction passes 64 lanes at a time.
constexpr int WK = 64;

template <typename T, int NV>
__global__ void __launch_bounds__(128)
wide_plain_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long max_len, const int64_t* __restrict__ slots,
                  const int64_t* __restrict__ lengths, int S, int H, int G, int W, int Dv, float scale, int window, int chunk, const T* __restrict__ sinks,
                  T* __restrict__ out) {
  extern __shared__ __align__(16) float smf[];
  constexpr int LD = WK + 1;
  const int LV = Dv + 1;
  float* sq = smf;                     // [PQ][LD]
  float* sk = sq + PQ * LD;            // [PK][LD]
  float* sv = sk + PK * LD;            // [PK][LV]
  float* sp = sv + PK * LV;            // [PQ][PK + 1]
  const int s0 = blockIdx.x * PQ, h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
  const int tid = threadIdx.x, r = tid >> 3, l8 = tid & 7;
  const long base = lengths[b], rows = slots[b] * max_len;
  const long last = min(base + min(S, s0 + PQ) - 1, max_len - 1);               // position of the last query
  const long mine = base + s0 + r;
  long firstk = window > 0 ? max(0l, base + s0 - window + 1) : 0l;
  if (chunk > 0) firstk = max(firstk, (base + s0) / chunk * chunk);
  const long from = max(window > 0 ? mine - window + 1 : 0l, chunk > 0 ? mine / chunk * chunk : 0l);      // first key this query sees
  float acc[NV], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) acc[j] = 0.f;
  for (long t0 = firstk; t0 <= last; t0 += PK) {
    float sc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int w0 = 0; w0 < W; w0 += WK) {
      __syncthreads();
      for (int i = tid; i < PQ * WK; i += 128) {
        const int t = i / WK, d = w0 + i % WK;
        sq[t * LD + i % WK] = s0 + t < S && d < W ? to_f(q[(((long)b * S + s0 + t) * H + h) * W + d]) : 0.f;
      }
      for (int i = tid; i < PK * WK; i += 128) {
        const int t = i / WK, d = w0 + i % WK;
        sk[t * LD + i % WK] = t0 + t <= last && d < W ? to_f(k[(rows + t0 + t) * W + d]) : 0.f;
      }
      if (w0 == 0) {
        for (int i = tid; i < PK * Dv; i += 128) {
          const int t = i / Dv, d = i % Dv;
          sv[t * LV + d] = t0 + t <= last ? to_f(v[((rows + t0 + t) * G + g) * Dv + d]) : 0.f;
        }
      }
      __syncthreads();
#pragma unroll 8
      for (int d = 0; d < WK; ++d) {
        const float x = sq[r * LD + d];
#pragma unroll
        for (int j = 0; j < 4; ++j) sc[j] = fmaf(x, sk[(l8 + j * 8) * LD + d], sc[j]);
      }
    }
    float tm = -INFINITY;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const long p = t0 + l8 + j * 8;
      sc[j] = p > mine || p > last || p < from ? -INFINITY : sc[j] * scale;
      tm = fmaxf(tm, sc[j]);
    }
#pragma unroll
    for (int d = 1; d < 8; d <<= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, d));
    const float n = fmaxf(m, tm), c = n == -INFINITY ? 1.f : expf(m - n);
    m = n;
    float ts = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float p = sc[j] == -INFINITY ? 0.f : expf(sc[j] - n);
      sp[r * (PK + 1) + l8 + j * 8] = p;
      ts += p;
    }
#pragma unroll
    for (int d = 1; d < 8; d <<= 1) ts += __shfl_xor_sync(0xffffffffu, ts, d);
    l = l * c + ts;
    __syncwarp();
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = l8 + j * 8;
      if (d < Dv) {
        float o = 0.f;
        for (int t = 0; t < PK; ++t) o = fmaf(sp[r * (PK + 1) + t], sv[t * LV + d], o);
        acc[j] = acc[j] * c + o;
      }
    }
  }
  if (s0 + r >= S) return;
  float inv = 0.f;
  if (sinks) {
    const float sk_ = to_f(sinks[h]), n = fmaxf(m, sk_);
    const float c = m == -INFINITY ? 0.f : expf(m - n);
    inv = c / (l * c + expf(sk_ - n));
  } else if (l > 0.f) {
    inv = 1.f / l;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int d = l8 + j * 8;
    if (d < Dv) out[(((long)b * S + s0 + r) * H + h) * Dv + d] = from_f<T>(acc[j] * inv);
  }
}

// ------------------------------------------------------------------------------------------------ gate
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
head_gate_kernel(const T* __restrict__ o, int dvp, const T* __restrict__ g, long ldg, long rows, int HD, int Dv, int per_head,
                 T* __restrict__ out) {
  const long per = HD / VEC;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < rows * per; i += gridDim.x * 256l) {
    const long r = i / per;
    const int c = (int)(i % per) * VEC, h = c / Dv, d = c % Dv;
    float x[VEC], y[VEC];
    load_vec<VEC>(o + (r * (HD / Dv) + h) * dvp + d, x);
    if (per_head) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = to_f(g[r * ldg + h]);
    } else {
      load_vec<VEC>(g + r * ldg + c, y);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] *= sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-y[e])) : sigmoid_f(y[e]);
    store_vec<VEC>(out + r * HD + c, x);
  }
}

template <typename T>
int prep_t(const PrepArgs& a, long N, cudaStream_t st) {
  uintptr_t bits = 0;
  for (const void* p : {a.q, a.k, a.v, a.bq, a.bk, a.bv, a.wq, a.wk}) bits |= reinterpret_cast<uintptr_t>(p);
  const bool v4 = a.D % 4 == 0 && a.Dv % 4 == 0 && a.rot % (a.paired ? 4 : 8) == 0 && a.dq % 4 == 0 && a.ldq % 4 == 0 && a.ldk % 4 == 0 && a.ldv % 4 == 0 &&
                  (!a.vp || a.dvp % 4 == 0) && bits % (4 * sizeof(T)) == 0;
  const int extra = a.talk ? ((a.H * a.D + 3) / 4 * 4 + a.H * ((a.H + 7) / 8 * 8)) * 4 : 0, smem = angle_floats(a.rot) * 4 + extra;
  if (a.D > 512 || smem > 200 * 1024 || (a.talk && a.maps != 1)) return -1;
  auto launch = [&](auto kernel) {
    if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
    kernel<<<(unsigned)N, 128, smem, st>>>(a);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  const bool v8 = a.D % 8 == 0 && a.Dv % 8 == 0 && (a.paired || a.rot % 16 == 0) && a.dq % 8 == 0 && a.ldq % 8 == 0 && a.ldk % 8 == 0 && a.ldv % 8 == 0 &&
                  (!a.vp || a.dvp % 8 == 0) && bits % 16 == 0;
  auto pick = [&](auto talk) {
    constexpr bool K = decltype(talk)::value;
    if (v8 && a.D <= 64) return launch(qkv_prep_wide_kernel<T, 8, K>);
    if (v8 && a.D <= 128) return launch(qkv_prep_wide_kernel<T, 16, K>);
    if (v8 && a.D <= 256) return launch(qkv_prep_wide_kernel<T, 32, K>);
    if (!v4) return launch(qkv_prep_kernel<T, 1, 16, K>);
    if (a.D <= 128) return launch(qkv_prep_kernel<T, 4, 1, K>);
    if (a.D <= 256) return launch(qkv_prep_kernel<T, 4, 2, K>);
    return launch(qkv_prep_kernel<T, 4, 4, K>);
  };
  return a.talk ? pick(std::true_type{}) : pick(std::false_type{});
}

template <int DK, int DVT>
int decode_run(const DecodeArgs& a, int B, cudaStream_t st) {
  constexpr int ring = (16 * (DK + 8) + 4 * RING * KEYS * (DK + 8 + DVT + 8)) * 2, join = 4 * 16 * (DVT + 4) * 4;
  constexpr int smem = ring > join ? ring : join;
  auto k = decode_kernel<DK, DVT>;
  if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  k<<<dim3(a.splits, a.G * a.head_blocks, B), 128, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
template <int DK>
int decode_dv(const DecodeArgs& a, int B, cudaStream_t st) {
  if (a.Dv <= 64) return decode_run<DK, 64>(a, B, st);
  if (a.Dv <= 128) return decode_run<DK, 128>(a, B, st);
  return decode_run<DK, 256>(a, B, st);
}

template <typename T>
int plain_t(const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S, int H, int G, int D, int Dv,
            float scale, float cap, int window, int chunk, const void* sinks, void* out, cudaStream_t st) {
  const int smem = ((PQ + PK) * (D + 1) + PK * (Dv + 1) + PQ * (PK + 1)) * 4;
  if (Dv > 512 || smem > 227 * 1024) return -1;
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
    kernel<<<dim3((S + PQ - 1) / PQ, H, B), 128, smem, st>>>((const T*)q, (const T*)k, (const T*)v, max_len, slots, lengths, S, H, G, D, Dv, scale, cap, window, chunk,
                                                             (const T*)sinks, (T*)out);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  if (Dv <= 64) return launch(plain_kernel<T, 8>);
  if (Dv <= 128) return launch(plain_kernel<T, 16>);
  if (Dv <= 256) return launch(plain_kernel<T, 32>);
  return launch(plain_kernel<T, 64>);
}

template <int DW>
int wide_decode_run(const WideArgs& a, int B, cudaStream_t st) {
  const int LQ = a.G * ((a.D + 15) / 16 * 16) + 8;
  const int pipe = (16 * LQ + 4 * WIDE_RING * KEYS * (DW + 8)) * 2, join = 4 * 16 * (DW + 4) * 4, smem = pipe > join ? pipe : join;
  if (smem > 227 * 1024) return -1;
  auto k = wide_decode_kernel<DW>;
  if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  k<<<dim3(a.splits, a.head_blocks, B), 128, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
int wide_plain_t(const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S, int H, int G, int D,
                 int Dv, float scale, int window, int chunk, const void* sinks, void* out, cudaStream_t st) {
  const int smem = ((PQ + PK) * (WK + 1) + PK * (Dv + 1) + PQ * (PK + 1)) * 4;
  if (Dv > 512 || smem > 227 * 1024) return -1;
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
    kernel<<<dim3((S + PQ - 1) / PQ, H, B), 128, smem, st>>>((const T*)q, (const T*)k, (const T*)v, max_len, slots, lengths, S, H, G, G * D, Dv, scale, window,
                                                             chunk, (const T*)sinks, (T*)out);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  if (Dv <= 64) return launch(wide_plain_kernel<T, 8>);
  if (Dv <= 128) return launch(wide_plain_kernel<T, 16>);
  if (Dv <= 256) return launch(wide_plain_kernel<T, 32>);
  return launch(wide_plain_kernel<T, 64>);
}

template <typename T>
int gate_t(const void* o, int dvp, const void* g, long ldg, long rows, int HD, int Dv, int per_head, void* out, int sms, cudaStream_t st) {
  const bool v8 = Dv % 8 == 0 && dvp % 8 == 0 && (per_head || (ldg % 8 == 0 && reinterpret_cast<uintptr_t>(g) % 16 == 0));
  const long blocks = (rows * (HD / (v8 ? 8 : 1)) + 255) / 256;
  const unsigned grid = (unsigned)(blocks < sms * 16l ? (blocks < 1 ? 1 : blocks) : sms * 16l);
  if (v8) head_gate_kernel<T, 8><<<grid, 256, 0, st>>>((const T*)o, dvp, (const T*)g, ldg, rows, HD, Dv, per_head, (T*)out);
  else head_gate_kernel<T, 1><<<grid, 256, 0, st>>>((const T*)o, dvp, (const T*)g, ldg, rows, HD, Dv, per_head, (T*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cattn
}  // namespace mt

using namespace mt::cattn;
using bf16 = __nv_bfloat16;

extern "C" int mt_qkv_prep(int f32, const PrepArgs* a, long N, cudaStream_t st) {
  if (N <= 0) return 0;
  return f32 ? prep_t<float>(*a, N, st) : prep_t<bf16>(*a, N, st);
}

// diff (or null): q holds two maps per head, H counts both, out is [B, H / 2 * Dv]
extern "C" int mt_cached_decode(const void* q, const void* k, const void* v, const int64_t* slots, const int64_t* lengths, long max_len, int B, int H, int G,
                                int D, int Dv, float scale, float cap, int window, int chunk, const void* sinks, const void* gate, long ldg, int per_head,
                                const DiffArgs* diff, int splits, float* part, float* ml, void* out, cudaStream_t st) {
  if (B <= 0) return 0;
  if (D % 8 || Dv % 8 || D > 256 || Dv > 256 || H % G || splits < 1 || (diff && (H % 2 || sinks || splits > 64))) return -1;
  DecodeArgs a{(const bf16*)q, (const bf16*)k, (const bf16*)v, slots, lengths, max_len, H, G, D, Dv, window, chunk, splits, (H / G + 15) / 16, scale, cap,
               part, ml};
  const int rc = D <= 64 ? decode_dv<64>(a, B, st) : (D <= 128 ? decode_dv<128>(a, B, st) : decode_dv<256>(a, B, st));
  if (rc) return rc;
  if (diff)
    diff_merge_kernel<bf16><<<dim3(H / 2, B), 128, 0, st>>>(part, ml, *diff, H / 2, Dv, splits, (const bf16*)gate, ldg, per_head, (bf16*)out);
  else
    merge_kernel<bf16><<<dim3(H, B), Dv <= 64 ? 64 : 128, 0, st>>>(part, ml, H, Dv, splits, (const bf16*)sinks, (const bf16*)gate, ldg, per_head, (bf16*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

// q [B, H, G * D]: every head reads the keys of all key heads (a mixing matrix has been folded into the queries)
extern "C" int mt_wide_decode(const void* q, const void* k, const void* v, const int64_t* slots, const int64_t* lengths, long max_len, int B, int H, int G, int D,
                              int Dv, float scale, int window, int chunk, const void* sinks, int splits, float* part, float* ml, void* out, cudaStream_t st) {
  if (B <= 0) return 0;
  if (D % 8 || Dv % 8 || D > 256 || Dv > 256 || H % G || splits < 1) return -1;
  const WideArgs a{(const bf16*)q, (const bf16*)k, (const bf16*)v, slots, lengths, max_len, H, G, D, Dv, window, chunk, splits, (H + 15) / 16, scale, part, ml};
  const int w = D > Dv ? D : Dv, rc = w <= 64 ? wide_decode_run<64>(a, B, st) : w <= 128 ? wide_decode_run<128>(a, B, st) : wide_decode_run<256>(a, B, st);
  if (rc) return rc;
  merge_kernel<bf16><<<dim3(H, B), Dv <= 64 ? 64 : 128, 0, st>>>(part, ml, H, Dv, splits, (const bf16*)sinks, (const bf16*)nullptr, 0, 0, (bf16*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_wide_attention(int f32, const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S,
                                 int H, int G, int D, int Dv, float scale, int window, int chunk, const void* sinks, void* out, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  return f32 ? wide_plain_t<float>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, window, chunk, sinks, out, st)
             : wide_plain_t<bf16>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, window, chunk, sinks, out, st);
}

extern "C" int mt_cached_attention(int f32, const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S,
                                   int H, int G, int D, int Dv, float scale, float cap, int window, int chunk, const void* sinks, void* out, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  return f32 ? plain_t<float>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, cap, window, chunk, sinks, out, st)
             : plain_t<bf16>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, cap, window, chunk, sinks, out, st);
}

extern "C" int mt_head_gate(int f32, const void* o, int dvp, const void* g, long ldg, long rows, int HD, int Dv, int per_head, void* out, int sms,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? gate_t<float>(o, dvp, g, ldg, rows, HD, Dv, per_head, out, sms, st) : gate_t<bf16>(o, dvp, g, ldg, rows, HD, Dv, per_head, out, sms, st);
}

extern "C" int mt_diff_combine(int f32, const void* o, int dvp, const DiffArgs* a, long N, int H, int Dv, const void* gate, long ldg, int per_head, void* out,
                               int sms, cudaStream_t st) {
  if (N <= 0) return 0;
  if (Dv > 256) return -1;
  const bool v8 = Dv % 8 == 0 && dvp % 8 == 0 && (per_head || !gate || (ldg % 8 == 0 && reinterpret_cast<uintptr_t>(gate) % 16 == 0));
  auto grid = [&](int lpr) {
    const long blocks = (N * H * lpr + 255) / 256;
    return (unsigned)(blocks < sms * 16l ? blocks : sms * 16l);
  };
#define GO(T, VEC, LPR, NV) diff_combine_kernel<T, VEC, LPR, NV><<<grid(LPR), 256, 0, st>>>((const T*)o, dvp, *a, N, H, Dv, (const T*)gate, ldg, per_head, (T*)out)
#define BY(VEC, LPR, NV) do { if (f32) GO(float, VEC, LPR, NV); else GO(bf16, VEC, LPR, NV); } while (0)
  if (!v8) BY(1, 32, 8);
  else if (Dv <= 64) BY(8, 8, 1);
  else if (Dv <= 128) BY(8, 16, 1);
  else BY(8, 32, 1);
#undef BY
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
