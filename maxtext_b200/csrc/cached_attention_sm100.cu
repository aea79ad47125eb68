// Softmax attention over a slot-indexed key/value cache at inference: [slots, max_len, G, D] keys, [slots, max_len, G, Dv] values, any head
// widths, with soft-capped scores, a per-head sink in the denominator, a sliding window and a sigmoid output gate.
//
//   qkv_prep   projections -> rotated (first `rot` lanes, halves paired) and RMS-normalised q and k, cache rows, operands of the flash kernel
//   decode     one new token per sequence: keys split over CTAs and, inside a CTA, over four warps that each stream their own 16-key tiles
//              through a cp.async ring; up to 16 query heads of a key head sit in the M position of mma.sync m16n8k16; softmax in registers,
//              weights as (high, low) bf16 pairs. No barrier between tiles. tcgen05 has no use here: a step is bound by reading the cache
//              and its 128-row accumulators would be at most one eighth full
//   merge      joins the splits, adds the sink, applies the gate
//   plain      fp32 arithmetic on CUDA cores over the cache, any widths up to 512 and any number of new tokens
//   head_gate  gate of the prompt path, drops the flash kernel's width padding
#include "serving_common.cuh"
#include "warp_mma.cuh"

namespace mt {
namespace cattn {

// cap * tanh(s / cap) from one exponential: the error is relative to cap, a few units of fp32
__device__ __forceinline__ float capped(float s, float cap, float two_over_cap) {
  return cap - __fdividef(2.f * cap, 1.f + __expf(s * two_over_cap));
}

// ------------------------------------------------------------------------------------------------ prep
// One CTA per token; a warp per head. Lanes hold VEC neighbouring elements, ITER times.
template <typename T, int VEC, int ITER>
__global__ void __launch_bounds__(128)
qkv_prep_kernel(const T* __restrict__ q, long ldq, const T* __restrict__ k, long ldk, const T* __restrict__ v, long ldv, int H, int G, int D, int Dv,
                const int64_t* __restrict__ pos, const float* __restrict__ inv_ts, int rot, float eps, int S, T* __restrict__ qp, int dq, T* __restrict__ kp,
                T* __restrict__ vp, int dvp, T* __restrict__ kc, T* __restrict__ vc, long max_len, const int64_t* __restrict__ slots,
                const int64_t* __restrict__ lengths, const int64_t* __restrict__ new_lens) {
  extern __shared__ float2 cs[];                            // (cos, sin) of the rot / 2 angles
  const long n = blockIdx.x;
  const int b = (int)(n / S), s = (int)(n % S), half = rot / 2;
  const float p = (float)pos[n];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    sincosf(p * inv_ts[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  __syncthreads();
  const long at = lengths[b] + s;
  const bool keep = at < max_len && s < (new_lens ? new_lens[b] : (int64_t)S);
  const long row = slots[b] * max_len + at;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = warp; h < H + G; h += 4) {
    const bool key = h >= H;
    const T* src = key ? k + n * ldk + (long)(h - H) * D : q + n * ldq + (long)h * D;
    float x[ITER][VEC], ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int e0 = (it * 32 + lane) * VEC;
      if (e0 < D) {
        load_vec<VEC>(src + e0, x[it]);
        if (e0 < rot) {
          const bool low = e0 < half;
          float y[VEC];
          load_vec<VEC>(src + (low ? e0 + half : e0 - half), y);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            const float2 a = cs[(low ? e0 : e0 - half) + e];
            x[it][e] = x[it][e] * a.x + (low ? -y[e] : y[e]) * a.y;
          }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += x[it][e] * x[it][e];
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[it][e] = 0.f;
      }
    }
    if (eps >= 0.f) {
      const float r = rsqrtf(warp_add(ss) / (float)D + eps);
#pragma unroll
      for (int it = 0; it < ITER; ++it)
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[it][e] *= r;
    }
    T* dst = key ? (kp ? kp + (n * G + h - H) * dq : nullptr) : qp + (n * H + h) * dq;
    T* cache = key && keep ? kc + (row * G + h - H) * D : nullptr;
#pragma unroll
    for (int it = 0; it < ITER; ++it) {
      const int e0 = (it * 32 + lane) * VEC;
      if (dst && e0 < dq) store_vec<VEC>(dst + e0, x[it]);
      if (cache && e0 < D) store_vec<VEC>(cache + e0, x[it]);
    }
  }
  if (keep || vp) {
    for (int i = threadIdx.x * VEC; i < G * Dv; i += blockDim.x * VEC) {
      float x[VEC];
      load_vec<VEC>(v + n * ldv + i, x);
      if (keep) store_vec<VEC>(vc + row * G * Dv + i, x);
      if (vp) store_vec<VEC>(vp + (n * G + i / Dv) * dvp + i % Dv, x);
    }
    if (vp && dvp > Dv) {
      const int pad = dvp - Dv;
      for (int i = threadIdx.x; i < G * pad; i += blockDim.x) vp[(n * G + i / pad) * dvp + Dv + i % pad] = from_f<T>(0.f);
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode
struct DecodeArgs {
  const __nv_bfloat16 *q, *k, *v;      // q [B, H, D]
  const int64_t *slots, *lengths;      // lengths without the new token
  long max_len;
  int H, G, D, Dv, window, splits, head_blocks;
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
  const int first = (a.window > 0 && len > a.window) ? (int)(len - a.window) : 0;
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

// out [B, H * Dv] = (splits joined, sink in the denominator) * sigmoid(gate)
template <typename T>
__global__ void merge_kernel(const float* __restrict__ part, const float* __restrict__ ml, int H, int Dv, int splits, const T* __restrict__ sinks,
                             const T* __restrict__ gate, long ldg, T* __restrict__ out) {
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
    if (gate) o *= sigmoid_f(to_f(gate[b * ldg + (long)h * Dv + d]));
    out[(long)b * H * Dv + (long)h * Dv + d] = from_f<T>(o);
  }
}

// ------------------------------------------------------------------------------------------------ plain
// 16 queries of one head against tiles of 32 keys. Eight threads per query: four scores each per tile, then Dv / 8 output columns each.
constexpr int PQ = 16, PK = 32;

template <typename T, int NV>          // NV * 8 >= Dv
__global__ void __launch_bounds__(128)
plain_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long max_len, const int64_t* __restrict__ slots,
             const int64_t* __restrict__ lengths, int S, int H, int G, int D, int Dv, float scale, float cap, int window, const T* __restrict__ sinks,
             T* __restrict__ out) {
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
  const long firstk = window > 0 ? max(0l, base + s0 - window + 1) : 0l;
  const long mine = base + s0 + r;
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
      if (p > mine || p > last || (window > 0 && p <= mine - window)) x = -INFINITY;
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

// ------------------------------------------------------------------------------------------------ gate
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
head_gate_kernel(const T* __restrict__ o, int dvp, const T* __restrict__ g, long ldg, long rows, int HD, int Dv, T* __restrict__ out) {
  const long per = HD / VEC;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < rows * per; i += gridDim.x * 256l) {
    const long r = i / per;
    const int c = (int)(i % per) * VEC, h = c / Dv, d = c % Dv;
    float x[VEC], y[VEC];
    load_vec<VEC>(o + (r * (HD / Dv) + h) * dvp + d, x);
    load_vec<VEC>(g + r * ldg + c, y);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] *= sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-y[e])) : sigmoid_f(y[e]);
    store_vec<VEC>(out + r * HD + c, x);
  }
}

template <typename T>
int prep_t(const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, int H, int G, int D, int Dv, const int64_t* pos, const float* inv_ts,
           int rot, float eps, int S, void* qp, int dq, void* kp, void* vp, int dvp, void* kc, void* vc, long max_len, const int64_t* slots,
           const int64_t* lengths, const int64_t* new_lens, long N, cudaStream_t st) {
  const bool v4 = D % 4 == 0 && Dv % 4 == 0 && rot % 8 == 0 && dq % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 && (!vp || dvp % 4 == 0) &&
                  (reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) % (4 * sizeof(T)) == 0;
  const int wide = dq > D ? dq : D;
  auto launch = [&](auto kernel) {
    kernel<<<(unsigned)N, 128, (rot / 2) * 8 + 8, st>>>((const T*)q, ldq, (const T*)k, ldk, (const T*)v, ldv, H, G, D, Dv, pos, inv_ts, rot, eps, S, (T*)qp, dq,
                                                        (T*)kp, (T*)vp, dvp, (T*)kc, (T*)vc, max_len, slots, lengths, new_lens);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  if (wide > 512) return -1;
  if (!v4) return launch(qkv_prep_kernel<T, 1, 16>);
  if (wide <= 128) return launch(qkv_prep_kernel<T, 4, 1>);
  if (wide <= 256) return launch(qkv_prep_kernel<T, 4, 2>);
  return launch(qkv_prep_kernel<T, 4, 4>);
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
            float scale, float cap, int window, const void* sinks, void* out, cudaStream_t st) {
  const int smem = ((PQ + PK) * (D + 1) + PK * (Dv + 1) + PQ * (PK + 1)) * 4;
  if (Dv > 512 || smem > 227 * 1024) return -1;
  auto launch = [&](auto kernel) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
    kernel<<<dim3((S + PQ - 1) / PQ, H, B), 128, smem, st>>>((const T*)q, (const T*)k, (const T*)v, max_len, slots, lengths, S, H, G, D, Dv, scale, cap, window,
                                                             (const T*)sinks, (T*)out);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  if (Dv <= 64) return launch(plain_kernel<T, 8>);
  if (Dv <= 128) return launch(plain_kernel<T, 16>);
  if (Dv <= 256) return launch(plain_kernel<T, 32>);
  return launch(plain_kernel<T, 64>);
}

template <typename T>
int gate_t(const void* o, int dvp, const void* g, long ldg, long rows, int HD, int Dv, void* out, int sms, cudaStream_t st) {
  const bool v8 = Dv % 8 == 0 && dvp % 8 == 0 && ldg % 8 == 0 && reinterpret_cast<uintptr_t>(g) % 16 == 0;
  const long blocks = (rows * (HD / (v8 ? 8 : 1)) + 255) / 256;
  const unsigned grid = (unsigned)(blocks < sms * 16l ? (blocks < 1 ? 1 : blocks) : sms * 16l);
  if (v8) head_gate_kernel<T, 8><<<grid, 256, 0, st>>>((const T*)o, dvp, (const T*)g, ldg, rows, HD, Dv, (T*)out);
  else head_gate_kernel<T, 1><<<grid, 256, 0, st>>>((const T*)o, dvp, (const T*)g, ldg, rows, HD, Dv, (T*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace cattn
}  // namespace mt

using namespace mt::cattn;
using bf16 = __nv_bfloat16;

extern "C" int mt_qkv_prep(int f32, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, int H, int G, int D, int Dv, const int64_t* pos,
                           const float* inv_ts, int rot, float eps, int S, void* qp, int dq, void* kp, void* vp, int dvp, void* kc, void* vc, long max_len,
                           const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, long N, cudaStream_t st) {
  if (N <= 0) return 0;
  return f32 ? prep_t<float>(q, ldq, k, ldk, v, ldv, H, G, D, Dv, pos, inv_ts, rot, eps, S, qp, dq, kp, vp, dvp, kc, vc, max_len, slots, lengths, new_lens, N, st)
             : prep_t<bf16>(q, ldq, k, ldk, v, ldv, H, G, D, Dv, pos, inv_ts, rot, eps, S, qp, dq, kp, vp, dvp, kc, vc, max_len, slots, lengths, new_lens, N, st);
}

extern "C" int mt_cached_decode(const void* q, const void* k, const void* v, const int64_t* slots, const int64_t* lengths, long max_len, int B, int H, int G,
                                int D, int Dv, float scale, float cap, int window, const void* sinks, const void* gate, long ldg, int splits, float* part,
                                float* ml, void* out, cudaStream_t st) {
  if (B <= 0) return 0;
  if (D % 8 || Dv % 8 || D > 256 || Dv > 256 || H % G || splits < 1) return -1;
  DecodeArgs a{(const bf16*)q, (const bf16*)k, (const bf16*)v, slots, lengths, max_len, H, G, D, Dv, window, splits, (H / G + 15) / 16, scale, cap, part, ml};
  const int rc = D <= 64 ? decode_dv<64>(a, B, st) : (D <= 128 ? decode_dv<128>(a, B, st) : decode_dv<256>(a, B, st));
  if (rc) return rc;
  merge_kernel<bf16><<<dim3(H, B), Dv <= 64 ? 64 : 128, 0, st>>>(part, ml, H, Dv, splits, (const bf16*)sinks, (const bf16*)gate, ldg, (bf16*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_cached_attention(int f32, const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S,
                                   int H, int G, int D, int Dv, float scale, float cap, int window, const void* sinks, void* out, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  return f32 ? plain_t<float>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, cap, window, sinks, out, st)
             : plain_t<bf16>(q, k, v, max_len, slots, lengths, B, S, H, G, D, Dv, scale, cap, window, sinks, out, st);
}

extern "C" int mt_head_gate(int f32, const void* o, int dvp, const void* g, long ldg, long rows, int HD, int Dv, void* out, int sms, cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? gate_t<float>(o, dvp, g, ldg, rows, HD, Dv, out, sms, st) : gate_t<bf16>(o, dvp, g, ldg, rows, HD, Dv, out, sms, st);
}
