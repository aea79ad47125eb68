// Latent attention at inference. A token caches its normalised latent c [R] and a rotated key part kr [dr] shared by all heads.
//  * mla_prep: after the down-projections, per token: RMS norm of the query latent, RMS norm of c, rotation of kr, cache write.
//  * mla_pack: prompts: per-head q | k | v in the widths of the flash kernel, rotation applied, the rest zero.
//  * decode, three kernels: mla_absorb (q' = [W_uk^T q_nope | rotated q_rope]), mla_attn (all heads against the same cached vectors, the key range
//    of a sequence split over CTAs), mla_value_up (merge the splits, apply W_uv). The attention reads every cached vector of the window once:
//    it is a stream of [R + dr] rows through shared memory (cp.async), with the heads in the M = 16 position of mma.sync for both products. The
//    softmax weights enter the second product as a bf16 pair (high + low part), so they keep 16 bits of mantissa. Types and sizes that do not
//    fit that form (fp32, latents not a multiple of 64) take a plain kernel with fp32 arithmetic.
// Lengths and slots are device memory: nothing synchronises with the host, so a decode step can be captured in a graph.
#include "serving_common.cuh"
#include "warp_mma.cuh"

namespace mt {

// cos / sin of the dr / 2 rotation angles at position pos, into shared memory [dr / 2][2]
__device__ __forceinline__ void rotation_table(float* cs, long pos, const float* __restrict__ inv_ts, int half) {
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf((float)pos * inv_ts[i], &s, &c);
    cs[2 * i] = c;
    cs[2 * i + 1] = s;
  }
}
// lane e of the rotated vector x [dr]
template <typename T>
__device__ __forceinline__ float rotated(const T* x, const float* cs, int e, int half, bool interleaved) {
  const int i = interleaved ? e >> 1 : (e < half ? e : e - half);
  const bool first = interleaved ? !(e & 1) : e < half;
  const float u = to_f(x[interleaved ? 2 * i : i]), v = to_f(x[interleaved ? 2 * i + 1 : i + half]);
  return first ? u * cs[2 * i] - v * cs[2 * i + 1] : v * cs[2 * i] + u * cs[2 * i + 1];
}

// ------------------------------------------------------------------------------------------------ projection epilogue
// rms norm of p [n] times w, VEC elements per access; the result also goes to `also` when that is not null
template <typename T, int VEC>
__device__ __forceinline__ void norm_row(const T* __restrict__ p, const T* __restrict__ w, int n, float eps, float* red, T* __restrict__ y, T* __restrict__ also) {
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(p + i, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
  }
  const float rstd = rsqrtf(block_add(ss, red) / (float)n + eps);
  for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
    float v[VEC], g[VEC];
    load_vec<VEC>(p + i, v);
    load_vec<VEC>(w + i, g);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * rstd * g[e];
    store_vec<VEC>(y + i, v);
    if (also) store_vec<VEC>(also + i, v);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128) mla_prep_kernel(const T* __restrict__ qa, long ldq, const T* __restrict__ qw, int Q, const T* __restrict__ kva,
                                                       long ldk, const T* __restrict__ kw, int R, int dr, float eps, const int64_t* __restrict__ pos,
                                                       const float* __restrict__ inv_ts, int interleaved, int S, T* __restrict__ cq, T* __restrict__ lat,
                                                       T* __restrict__ kr, T* __restrict__ cache_lat, T* __restrict__ cache_kr, long max_len,
                                                       const int64_t* __restrict__ slots, const int64_t* __restrict__ lengths,
                                                       const int64_t* __restrict__ new_lens) {
  extern __shared__ float cs[];
  __shared__ float red[32];
  const long n = blockIdx.x;
  const int b = (int)(n / S), t = (int)(n % S);
  rotation_table(cs, pos[n], inv_ts, dr / 2);
  if (qa) norm_row<T, VEC>(qa + n * ldq, qw, Q, eps, red, cq + n * Q, (T*)nullptr);
  const T* p = kva + n * ldk;
  const long at = lengths[b] + t;
  const bool real = (!new_lens || t < new_lens[b]) && at < max_len;
  const long row = slots[b] * max_len + at;
  norm_row<T, VEC>(p, kw, R, eps, red, lat + n * R, real ? cache_lat + row * R : (T*)nullptr);       // its barriers also publish the rotation table
  for (int e = threadIdx.x; e < dr; e += blockDim.x) {
    const T v = from_f<T>(rotated(p + R, cs, e, dr / 2, interleaved));
    kr[n * dr + e] = v;
    if (real) cache_kr[row * dr + e] = v;
  }
}

// ------------------------------------------------------------------------------------------------ operands of the flash kernel
// q [N, H, nope + dr] -> qp [N, H, DQ]: nope | rotated | zeros. One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) mla_pack_q_kernel(const T* __restrict__ q, const int64_t* __restrict__ pos, const float* __restrict__ inv_ts,
                                                         int interleaved, int H, int nope, int dr, int DQ, T* __restrict__ qp) {
  extern __shared__ float cs[];
  const long n = blockIdx.x;
  rotation_table(cs, pos[n], inv_ts, dr / 2);
  __syncthreads();
  const int qk = nope + dr, C = DQ / 8;
  const bool vec = interleaved && nope % 8 == 0 && dr % 8 == 0;
  for (int i = threadIdx.x; i < H * C; i += blockDim.x) {
    const int h = i / C, e0 = (i % C) * 8;
    const T* x = q + (n * H + h) * qk;
    float v[8];
    if (vec) {
      if (e0 < qk) {
        load_vec<8>(x + e0, v);
        if (e0 >= nope) {
          const float* t = cs + (e0 - nope);             // (cos, sin) of four pairs
#pragma unroll
          for (int j = 0; j < 8; j += 2) {
            const float u = v[j], w = v[j + 1];
            v[j] = u * t[j] - w * t[j + 1];
            v[j + 1] = w * t[j] + u * t[j + 1];
          }
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = 0.f;
      }
      store_vec<8>(qp + (n * H + h) * DQ + e0, v);
      continue;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = e0 + j;
      v[j] = e < nope ? to_f(x[e]) : (e < qk ? rotated(x + nope, cs, e - nope, dr / 2, interleaved) : 0.f);
    }
    store_vec<8>(qp + (n * H + h) * DQ + e0, v);
  }
}

// kv [N, H, nope + vd], kr [N, dr] -> kp [N, H, DQ]: nope | kr | zeros, vp [N, H, DV]: v | zeros. VEC = 8 when the parts are multiples of 8.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) mla_pack_kv_kernel(const T* __restrict__ kv, const T* __restrict__ kr, int H, int nope, int dr, int vd, int DQ,
                                                          int DV, T* __restrict__ kp, T* __restrict__ vp) {
  const long n = blockIdx.x;
  const int qk = nope + dr, C = (DQ + DV) / VEC;
  for (int i = threadIdx.x; i < H * C; i += blockDim.x) {
    const int h = i / C, e = (i % C) * VEC;
    const T* x = kv + (n * H + h) * (long)(nope + vd);
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    if (e < DQ) {
      if (e < nope) load_vec<VEC>(x + e, v);
      else if (e < qk) load_vec<VEC>(kr + n * dr + (e - nope), v);
      store_vec<VEC>(kp + (n * H + h) * (long)DQ + e, v);
    } else {
      if (e - DQ < vd) load_vec<VEC>(x + nope + (e - DQ), v);
      store_vec<VEC>(vp + (n * H + h) * (long)DV + (e - DQ), v);
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode: absorb W_uk
// qa[b, h, j] = sum_d q[b, h, d] W[h * (nope + vd) + d, j] for j < R; qa[b, h, R + e] = rotated q_rope. grid (H, ceil(B / 4), ceil(R / 256)):
// warp w takes the rows d = w, w + 8, ... of a 256-column block, lane l eight columns; the warps' sums meet in shared memory.
constexpr int AB_BT = 4;

template <typename T, bool ALIGNED>
__global__ void __launch_bounds__(256) mla_absorb_kernel(const T* __restrict__ q, const T* __restrict__ w, const int64_t* __restrict__ pos,
                                                         const float* __restrict__ inv_ts, int interleaved, int B, int H, int nope, int dr, int vd, int R,
                                                         T* __restrict__ qa) {
  extern __shared__ __align__(16) float sm[];            // [8][AB_BT][256] partial sums, then the rotation table
  const int h = blockIdx.x, b0 = blockIdx.y * AB_BT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int j = blockIdx.z * 256 + lane * 8, qk = nope + dr;
  float acc[AB_BT][8];
#pragma unroll
  for (int i = 0; i < AB_BT; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[i][e] = 0.f;
  const T* wb = w + (long)h * (nope + vd) * R;
#pragma unroll 8
  for (int d = warp; d < nope; d += 8) {
    float wv[8];
    if (ALIGNED) {
#pragma unroll
      for (int e = 0; e < 8; ++e) wv[e] = 0.f;
      if (j < R) load_vec<8>(wb + (long)d * R + j, wv);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) wv[e] = j + e < R ? to_f(wb[(long)d * R + j + e]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < AB_BT; ++i) {
      const float x = b0 + i < B ? to_f(q[((long)(b0 + i) * H + h) * qk + d]) : 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[i][e] += x * wv[e];
    }
  }
#pragma unroll
  for (int i = 0; i < AB_BT; ++i) store_vec<8>(sm + (warp * AB_BT + i) * 256 + lane * 8, acc[i]);
  __syncthreads();
  for (int i = tid; i < AB_BT * 256; i += 256) {
    const int bi = i >> 8, c = i & 255, jj = blockIdx.z * 256 + c;
    if (b0 + bi < B && jj < R) {
      float s = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) s += sm[(g * AB_BT + bi) * 256 + c];
      qa[((long)(b0 + bi) * H + h) * (R + dr) + jj] = from_f<T>(s);
    }
  }
  if (blockIdx.z == 0) {
    float* cs = sm + 8 * AB_BT * 256;
    for (int i = 0; i < AB_BT && b0 + i < B; ++i) {
      __syncthreads();
      rotation_table(cs, pos[b0 + i], inv_ts, dr / 2);
      __syncthreads();
      const T* x = q + ((long)(b0 + i) * H + h) * qk + nope;
      for (int e = tid; e < dr; e += 256) qa[((long)(b0 + i) * H + h) * (R + dr) + R + e] = from_f<T>(rotated(x, cs, e, dr / 2, interleaved));
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode: attention in the latent space
struct AttnArgs {
  int H, R, dr, window, splits;
  long max_len;
  float scale;
  const int64_t* slots;
  const int64_t* lengths;        // tokens cached before this one
};

// keys of split `s` of sequence b: [lo, hi)
__device__ __forceinline__ void key_range(const AttnArgs& a, int b, int s, int& lo, int& hi) {
  const int len = (int)min(a.lengths[b] + 1, (int64_t)a.max_len);
  const int first = (a.window > 0 && len > a.window) ? len - a.window : 0;
  const int per = (((len - first + a.splits - 1) / a.splits) + 15) & ~15;
  lo = min(len, first + s * per);
  hi = min(len, lo + per);
}

// Plain form: grid (splits, ceil(H / HG), B), 256 threads; part [B, H, splits, R] unnormalised sums, ml [B, H, splits, 2] (maximum, sum).
constexpr int PL_HG = 4, PL_TILE = 16, PL_CMAX = 4;

template <typename T>
__global__ void __launch_bounds__(256) mla_attn_plain_kernel(AttnArgs a, const T* __restrict__ qa, const T* __restrict__ lat, const T* __restrict__ kr,
                                                             float* __restrict__ part, float* __restrict__ ml) {
  extern __shared__ __align__(16) float sm[];
  const int D = a.R + a.dr, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * PL_HG, b = blockIdx.z;
  float* qs = sm;                                        // [HG][D]
  float* xs = qs + PL_HG * D;                            // [TILE][D]
  float* ps = xs + PL_TILE * D;                          // [HG][TILE]
  int lo, hi;
  key_range(a, b, split, lo, hi);
  const long base = a.slots[b] * a.max_len;
  for (int i = tid; i < PL_HG * D; i += 256) qs[i] = h0 + i / D < a.H ? to_f(qa[((long)b * a.H + h0) * D + i]) * a.scale : 0.f;
  float acc[PL_HG][PL_CMAX], m[PL_HG], l[PL_HG];
#pragma unroll
  for (int g = 0; g < PL_HG; ++g) {
    m[g] = -INFINITY; l[g] = 0.f;
#pragma unroll
    for (int c = 0; c < PL_CMAX; ++c) acc[g][c] = 0.f;
  }
  for (int t0 = lo; t0 < hi; t0 += PL_TILE) {
    const int n = min(PL_TILE, hi - t0);
    __syncthreads();
    for (int i = tid; i < n * D; i += 256) {
      const int r = i / D, e = i % D;
      xs[i] = e < a.R ? to_f(lat[(base + t0 + r) * a.R + e]) : to_f(kr[(base + t0 + r) * a.dr + (e - a.R)]);
    }
    __syncthreads();
    for (int i = warp; i < n * PL_HG; i += 8) {
      const int r = i / PL_HG, g = i % PL_HG;
      float s = 0.f;
      for (int e = lane; e < D; e += 32) s += qs[g * D + e] * xs[r * D + e];
      s = warp_add(s);
      if (lane == 0) ps[g * PL_TILE + r] = s;
    }
    __syncthreads();
#pragma unroll
    for (int g = 0; g < PL_HG; ++g) {
      float mx = m[g];
      for (int r = 0; r < n; ++r) mx = fmaxf(mx, ps[g * PL_TILE + r]);
      const float f = expf(m[g] - mx);
      m[g] = mx;
      l[g] *= f;
#pragma unroll
      for (int c = 0; c < PL_CMAX; ++c) acc[g][c] *= f;
      for (int r = 0; r < n; ++r) {
        const float p = expf(ps[g * PL_TILE + r] - mx);
        l[g] += p;
#pragma unroll
        for (int c = 0; c < PL_CMAX; ++c)
          if (tid + c * 256 < a.R) acc[g][c] += p * xs[r * D + tid + c * 256];
      }
    }
  }
#pragma unroll
  for (int g = 0; g < PL_HG; ++g) {
    if (h0 + g >= a.H) continue;
    const long o = ((long)b * a.H + h0 + g) * a.splits + split;
#pragma unroll
    for (int c = 0; c < PL_CMAX; ++c)
      if (tid + c * 256 < a.R) part[o * a.R + tid + c * 256] = acc[g][c];
    if (tid == 0) { ml[o * 2] = m[g]; ml[o * 2 + 1] = l[g]; }
  }
}

// Tensor-core form (bf16): grid (splits, ceil(H / 16), B), 256 threads. Tiles of 64 keys, two in flight. Warp w: scores of keys 8 w .. 8 w + 7
// for 16 heads; then columns [w * R / 8, (w + 1) * R / 8) of the weighted sum. CT = R / 64 column tiles of 8 per warp.
constexpr int TC_KEYS = 64, TC_NT = 256, TC_PLD = TC_KEYS + 8;

template <int CT>
__global__ void __launch_bounds__(TC_NT) mla_attn_tc_kernel(AttnArgs a, const __nv_bfloat16* __restrict__ qa, const __nv_bfloat16* __restrict__ lat,
                                                            const __nv_bfloat16* __restrict__ kr, float* __restrict__ part, float* __restrict__ ml) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int R = CT * 64, D = R + a.dr, LD = D + 8;       // row padding of 16 bytes: the eight rows of an ldmatrix start in different banks
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(raw);                     // [16][LD]
  __nv_bfloat16* xs = qs + 16 * LD;                                              // [2][64][LD]
  __nv_bfloat16* ph = xs + 2 * TC_KEYS * LD;                                     // [16][PLD] high part of the weights
  __nv_bfloat16* pl = ph + 16 * TC_PLD;                                          // low part
  float* wmax = reinterpret_cast<float*>(pl + 16 * TC_PLD);                      // [8][16]
  float* wsum = wmax + 128;                                                      // [8][16]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * 16, b = blockIdx.z;
  int lo, hi;
  key_range(a, b, split, lo, hi);
  const long base = a.slots[b] * a.max_len;
  const int vec_row = D / 8, vec_lat = R / 8;
  auto issue = [&](int t0, int buf) {
    for (int r = warp; r < TC_KEYS; r += TC_NT / 32) {
      const bool in = t0 + r < hi;
      const long row = base + (in ? t0 + r : lo);
      __nv_bfloat16* dst = xs + ((long)buf * TC_KEYS + r) * LD;
      const int bytes = in ? 16 : 0;                                                         // rows past the end are zero-filled
#pragma unroll
      for (int v = lane; v < CT * 8; v += 32) la_cp_async16(dst + v * 8, lat + row * R + v * 8, bytes);
      for (int v = lane; v < vec_row - vec_lat; v += 32) la_cp_async16(dst + R + v * 8, kr + row * a.dr + v * 8, bytes);
    }
    la_commit();
  };
  if (lo < hi) issue(lo, 0);
  for (int i = tid; i < 16 * vec_row; i += TC_NT) {
    const int g = i / vec_row, v = i % vec_row;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (h0 + g < a.H) x = *reinterpret_cast<const uint4*>(qa + ((long)b * a.H + h0 + g) * D + v * 8);
    *reinterpret_cast<uint4*>(qs + g * LD + v * 8) = x;
  }
  float acc[CT][4];
#pragma unroll
  for (int c = 0; c < CT; ++c)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[c][e] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;                    // heads lane / 4 and lane / 4 + 8
  const int gr = lane >> 2, kc = (lane & 3) * 2;
  int buf = 0;
  for (int t0 = lo; t0 < hi; t0 += TC_KEYS, buf ^= 1) {
    if (t0 + TC_KEYS < hi) { issue(t0 + TC_KEYS, buf ^ 1); la_wait<1>(); } else { la_wait<0>(); }
    __syncthreads();
    const __nv_bfloat16* xt = xs + (long)buf * TC_KEYS * LD;
    // scores of 8 keys: A = q (16 x 16 pieces), B = keys (8 rows); one ldmatrix.x4 of the keys covers two k-steps
    float sc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[i][e] = 0.f;
    const __nv_bfloat16* qrow = qs + (lane & 15) * LD + (lane >> 4) * 8;
    const __nv_bfloat16* krow = xt + (warp * 8 + (lane & 7)) * LD + (lane >> 3) * 8;
    int k = 0;
#pragma unroll 2
    for (; k + 64 <= D; k += 64) {
      unsigned fa[4][4], fb[2][4];
      la_ldm4(fb[0], krow + k);
      la_ldm4(fb[1], krow + k + 32);
#pragma unroll
      for (int i = 0; i < 4; ++i) la_ldm4(fa[i], qrow + k + 16 * i);
#pragma unroll
      for (int i = 0; i < 4; ++i) la_mma(sc[i], fa[i], fb[i >> 1][2 * (i & 1)], fb[i >> 1][2 * (i & 1) + 1]);
    }
    for (; k + 32 <= D; k += 32) {
      unsigned fa[4], fb[4];
      la_ldm4(fb, krow + k);
      la_ldm4(fa, qrow + k);
      la_mma(sc[0], fa, fb[0], fb[1]);
      la_ldm4(fa, qrow + k + 16);
      la_mma(sc[1], fa, fb[2], fb[3]);
    }
    if (k < D) {                                         // D is a multiple of 16: one k-step is left
      unsigned fa[4], fb[2];
      const unsigned p = (unsigned)__cvta_generic_to_shared(xt + (warp * 8 + (lane & 7)) * LD + k + ((lane >> 3) & 1) * 8);
      asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(fb[0]), "=r"(fb[1]) : "r"(p));
      la_ldm4(fa, qrow + k);
      la_mma(sc[2], fa, fb[0], fb[1]);
    }
    float s[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = (sc[0][e] + sc[1][e]) + (sc[2][e] + sc[3][e]);
    const int key = t0 + warp * 8 + kc;
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = key + (e & 1) < hi ? s[e] * a.scale : -INFINITY;
    float x0 = fmaxf(s[0], s[1]), x1 = fmaxf(s[2], s[3]);
#pragma unroll
    for (int o = 1; o <= 2; o <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, o));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, o));
    }
    if ((lane & 3) == 0) { wmax[warp * 16 + gr] = x0; wmax[warp * 16 + gr + 8] = x1; }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < 8; ++w) { n0 = fmaxf(n0, wmax[w * 16 + gr]); n1 = fmaxf(n1, wmax[w * 16 + gr + 8]); }
    const float f0 = expf(m0 - n0), f1 = expf(m1 - n1);  // the first tile holds at least one key: n is finite
    m0 = n0; m1 = n1;
    const float p[4] = {expf(s[0] - n0), expf(s[1] - n0), expf(s[2] - n1), expf(s[3] - n1)};
    l0 = l0 * f0 + p[0] + p[1];                          // this lane's keys only; summed over lanes and warps at the end
    l1 = l1 * f1 + p[2] + p[3];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const __nv_bfloat16 a0 = __float2bfloat16_rn(p[2 * e]), a1 = __float2bfloat16_rn(p[2 * e + 1]);
      const int at = (gr + 8 * e) * TC_PLD + warp * 8 + kc;
      *reinterpret_cast<__nv_bfloat162*>(ph + at) = __nv_bfloat162(a0, a1);
      *reinterpret_cast<__nv_bfloat162*>(pl + at) = __floats2bfloat162_rn(p[2 * e] - __bfloat162float(a0), p[2 * e + 1] - __bfloat162float(a1));
    }
#pragma unroll
    for (int c = 0; c < CT; ++c) { acc[c][0] *= f0; acc[c][1] *= f0; acc[c][2] *= f1; acc[c][3] *= f1; }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < TC_KEYS; ks += 16) {
      unsigned fh[4], fl[4];
      la_ldm4(fh, ph + (lane & 15) * TC_PLD + ks + (lane >> 4) * 8);
      la_ldm4(fl, pl + (lane & 15) * TC_PLD + ks + (lane >> 4) * 8);
      const __nv_bfloat16* vrow = xt + (ks + (lane & 15)) * LD + warp * CT * 8 + (lane >> 4) * 8;
#pragma unroll
      for (int c = 0; c + 1 < CT; c += 2) {
        unsigned fb[4];
        la_ldm4t(fb, vrow + c * 8);
        la_mma(acc[c], fh, fb[0], fb[1]);
        la_mma(acc[c], fl, fb[0], fb[1]);
        la_mma(acc[c + 1], fh, fb[2], fb[3]);
        la_mma(acc[c + 1], fl, fb[2], fb[3]);
      }
      if constexpr (CT & 1) {
        unsigned fb[2];
        la_ldm2t(fb, xt + (ks + (lane & 15)) * LD + warp * CT * 8 + (CT - 1) * 8);
        la_mma(acc[CT - 1], fh, fb[0], fb[1]);
        la_mma(acc[CT - 1], fl, fb[0], fb[1]);
      }
    }
    __syncthreads();                                     // the tile and the weights are free again
  }
#pragma unroll
  for (int o = 1; o <= 2; o <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, o);
    l1 += __shfl_xor_sync(0xffffffffu, l1, o);
  }
  if ((lane & 3) == 0) { wsum[warp * 16 + gr] = l0; wsum[warp * 16 + gr + 8] = l1; }
  __syncthreads();
  auto out_row = [&](int g) { return ((long)b * a.H + h0 + g) * a.splits + split; };
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int g = gr + 8 * e;
    if (h0 + g < a.H) {
      float* o = part + out_row(g) * R + warp * CT * 8 + kc;
#pragma unroll
      for (int c = 0; c < CT; ++c) *reinterpret_cast<float2*>(o + c * 8) = make_float2(acc[c][2 * e], acc[c][2 * e + 1]);
      if (warp == 0 && (lane & 3) == 0) {
        float l = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) l += wsum[w * 16 + g];
        ml[out_row(g) * 2] = e ? m1 : m0;
        ml[out_row(g) * 2 + 1] = l;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode: merge the splits, apply W_uv
// out[b, h, e] = sum_j ctx[b, h, j] W[h * (nope + vd) + nope + e, j]. grid (H, ceil(B / 4), ceil(vd / 64)); a warp takes one row e at a time.
template <typename T, bool ALIGNED>
__global__ void __launch_bounds__(256) mla_value_up_kernel(const float* __restrict__ part, const float* __restrict__ ml, const T* __restrict__ w, int B,
                                                           int H, int nope, int vd, int R, int splits, T* __restrict__ out) {
  extern __shared__ __align__(16) float ctx[];           // [AB_BT][Rp], Rp = R rounded up to 4
  __shared__ float wt[AB_BT][64];
  const int h = blockIdx.x, b0 = blockIdx.y * AB_BT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int Rp = (R + 3) & ~3;
  if (tid < AB_BT && b0 + tid < B) {
    const float* p = ml + ((long)(b0 + tid) * H + h) * splits * 2;
    float m = -INFINITY, den = 0.f;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, p[2 * s]);
    for (int s = 0; s < splits; ++s) den += p[2 * s + 1] > 0.f ? p[2 * s + 1] * expf(p[2 * s] - m) : 0.f;
    for (int s = 0; s < splits; ++s) wt[tid][s] = p[2 * s + 1] > 0.f ? expf(p[2 * s] - m) / den : 0.f;
  }
  __syncthreads();
  for (int i = tid; i < AB_BT * R; i += 256) {
    const int bi = i / R, j = i % R;
    float v = 0.f;
    if (b0 + bi < B) {
      const float* p = part + (((long)(b0 + bi) * H + h) * splits) * R + j;
      for (int s = 0; s < splits; ++s) v += wt[bi][s] > 0.f ? wt[bi][s] * p[(long)s * R] : 0.f;
    }
    ctx[bi * Rp + j] = v;
  }
  __syncthreads();
  const int e1 = min(vd, (int)(blockIdx.z + 1) * 64);
  for (int e = blockIdx.z * 64 + warp; e < e1; e += 8) {
    const T* wr = w + ((long)h * (nope + vd) + nope + e) * R;
    float acc[AB_BT];
#pragma unroll
    for (int i = 0; i < AB_BT; ++i) acc[i] = 0.f;
    if (ALIGNED) {
      for (int j = lane * 8; j < R; j += 256) {
        float wv[8];
        load_vec<8>(wr + j, wv);
#pragma unroll
        for (int i = 0; i < AB_BT; ++i) {
          float c[8];
          load_vec<8>(ctx + i * Rp + j, c);
#pragma unroll
          for (int x = 0; x < 8; ++x) acc[i] += c[x] * wv[x];
        }
      }
    } else {
      for (int j = lane; j < R; j += 32) {
        const float wv = to_f(wr[j]);
#pragma unroll
        for (int i = 0; i < AB_BT; ++i) acc[i] += ctx[i * Rp + j] * wv;
      }
    }
#pragma unroll
    for (int i = 0; i < AB_BT; ++i) {
      const float v = warp_add(acc[i]);
      if (lane == 0 && b0 + i < B) out[((long)(b0 + i) * H + h) * vd + e] = from_f<T>(v);
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode: the two per-head products on tensor cores
// bf16, batches of eight and more. Batch rows in the M position, 64 columns per CTA.
constexpr int HB = 64;                                   // batch rows per absorb CTA
constexpr int VB = 32;                                   // batch rows per value CTA

// grid (H, R / 64, ceil(B / 64)), 128 threads; warp w: columns 16 w .. 16 w + 15, four row tiles
__global__ void __launch_bounds__(128) mla_absorb_tc_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ w,
                                                            const int64_t* __restrict__ pos, const float* __restrict__ inv_ts, int interleaved, int B, int H,
                                                            int nope, int dr, int vd, int R, __nv_bfloat16* __restrict__ qa) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int h = blockIdx.x, j0 = blockIdx.y * 64, b0 = blockIdx.z * HB, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qk = nope + dr, QL = nope + 8, nb = min(HB, B - b0);
  __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(raw);                     // [nope][72]
  __nv_bfloat16* qs = ws + nope * 72;                                            // [64][QL]
  const __nv_bfloat16* wb = w + (long)h * (nope + vd) * R + j0;
  for (int i = tid; i < nope * 8; i += 128) la_cp_async16(ws + (i >> 3) * 72 + (i & 7) * 8, wb + (long)(i >> 3) * R + (i & 7) * 8, 16);
  for (int r = warp; r < HB; r += 4)
    for (int v = lane; v < nope / 8; v += 32)
      la_cp_async16(qs + r * QL + v * 8, q + ((long)(b0 + (r < nb ? r : 0)) * H + h) * qk + v * 8, r < nb ? 16 : 0);
  la_commit();
  if (blockIdx.y == 0) {                                 // the rotated part, while the copies run
    const int half = dr / 2;
    for (int i = tid; i < nb * half; i += 128) {
      const int r = i / half, p = i % half;
      float s, c;
      sincosf((float)pos[b0 + r] * inv_ts[p], &s, &c);
      const __nv_bfloat16* x = q + ((long)(b0 + r) * H + h) * qk + nope;
      __nv_bfloat16* y = qa + ((long)(b0 + r) * H + h) * (R + dr) + R;
      const int iu = interleaved ? 2 * p : p, iv = interleaved ? 2 * p + 1 : p + half;
      const float u = to_f(x[iu]), v = to_f(x[iv]);
      y[iu] = __float2bfloat16_rn(u * c - v * s);
      y[iv] = __float2bfloat16_rn(v * c + u * s);
    }
  }
  float acc[4][2][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  la_wait<0>();
  __syncthreads();
#pragma unroll 2
  for (int k = 0; k < nope; k += 16) {
    unsigned fb[4];
    la_ldm4t(fb, ws + (k + (lane & 15)) * 72 + warp * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      if (m * 16 < nb) {
        unsigned fa[4];
        la_ldm4(fa, qs + (m * 16 + (lane & 15)) * QL + k + (lane >> 4) * 8);
        la_mma(acc[m][0], fa, fb[0], fb[1]);
        la_mma(acc[m][1], fa, fb[2], fb[3]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int r = m * 16 + (lane >> 2) + (e ? 8 : 0);
      if (r < nb) {
        __nv_bfloat16* y = qa + ((long)(b0 + r) * H + h) * (R + dr) + j0 + warp * 16 + (lane & 3) * 2;
        *reinterpret_cast<__nv_bfloat162*>(y) = __floats2bfloat162_rn(acc[m][0][e], acc[m][0][e + 1]);
        *reinterpret_cast<__nv_bfloat162*>(y + 8) = __floats2bfloat162_rn(acc[m][1][e], acc[m][1][e + 1]);
      }
    }
}

// grid (H, ceil(vd / 64), ceil(B / 32)), 256 threads; warp: columns 16 (w & 3) .., row tile w >> 2. The merged latent sums enter as bf16 pairs.
__global__ void __launch_bounds__(256) mla_value_up_tc_kernel(const float* __restrict__ part, const float* __restrict__ ml, const __nv_bfloat16* __restrict__ w,
                                                              int B, int H, int nope, int vd, int R, int splits, __nv_bfloat16* __restrict__ out) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float wt[VB][64];
  const int h = blockIdx.x, e0 = blockIdx.y * 64, b0 = blockIdx.z * VB, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int LD = R + 8, nb = min(VB, B - b0), ne = min(64, vd - e0);
  __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(raw);                     // [64][LD]
  __nv_bfloat16* ch = ws + 64 * LD;                                              // [32][LD] high, low
  __nv_bfloat16* cl = ch + VB * LD;
  const __nv_bfloat16* wb = w + ((long)h * (nope + vd) + nope + e0) * R;
  for (int r = warp; r < 64; r += 8)
    for (int v = lane; v < R / 8; v += 32) la_cp_async16(ws + r * LD + v * 8, wb + (long)(r < ne ? r : 0) * R + v * 8, r < ne ? 16 : 0);
  la_commit();
  if (tid < nb) {
    const float* p = ml + ((long)(b0 + tid) * H + h) * splits * 2;
    float m = -INFINITY, den = 0.f;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, p[2 * s]);
    for (int s = 0; s < splits; ++s) den += p[2 * s + 1] > 0.f ? p[2 * s + 1] * expf(p[2 * s] - m) : 0.f;
    for (int s = 0; s < splits; ++s) wt[tid][s] = p[2 * s + 1] > 0.f ? expf(p[2 * s] - m) / den : 0.f;
  }
  __syncthreads();
  for (int r = warp; r < VB; r += 8) {
    const float* p = part + ((long)(b0 + (r < nb ? r : 0)) * H + h) * splits * R;
    for (int j = lane * 4; j < R; j += 128) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < nb)
        for (int s = 0; s < splits; ++s) {
          const float f = wt[r][s];
          if (f > 0.f) {
            const float4 x = *reinterpret_cast<const float4*>(p + (long)s * R + j);
            v.x += f * x.x; v.y += f * x.y; v.z += f * x.z; v.w += f * x.w;
          }
        }
      __nv_bfloat162 hi, lo;
      la_split2(v.x, v.y, hi, lo);
      *reinterpret_cast<__nv_bfloat162*>(ch + r * LD + j) = hi;
      *reinterpret_cast<__nv_bfloat162*>(cl + r * LD + j) = lo;
      la_split2(v.z, v.w, hi, lo);
      *reinterpret_cast<__nv_bfloat162*>(ch + r * LD + j + 2) = hi;
      *reinterpret_cast<__nv_bfloat162*>(cl + r * LD + j + 2) = lo;
    }
  }
  la_wait<0>();
  __syncthreads();
  const int n0 = (warp & 3) * 16, m0 = (warp >> 2) * 16;
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}}, low[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
  for (int k = 0; k < R; k += 16) {
    unsigned fb[4], fh[4], fl[4];
    la_ldm4(fb, ws + (n0 + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8);
    la_ldm4(fh, ch + (m0 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    la_ldm4(fl, cl + (m0 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    la_mma(acc[0], fh, fb[0], fb[1]);
    la_mma(acc[1], fh, fb[2], fb[3]);
    la_mma(low[0], fl, fb[0], fb[1]);
    la_mma(low[1], fl, fb[2], fb[3]);
  }
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = m0 + (lane >> 2) + (e >> 1) * 8, c = n0 + n * 8 + (lane & 3) * 2 + (e & 1);
      if (r < nb && c < ne) out[((long)(b0 + r) * H + h) * vd + e0 + c] = __float2bfloat16_rn(acc[n][e] + low[n][e]);
    }
}

template <typename K>
int raise_smem(K k, size_t smem) {
  if (smem > 227 * 1024) return -1;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
  return 0;
}

size_t tc_smem(int R, int dr) {
  const size_t LD = R + dr + 8;
  return 2 * (16 * LD + 2 * TC_KEYS * LD + 2 * 16 * TC_PLD) + 4 * 256;
}
bool tc_form(int f32, int R, int dr) { return !f32 && R % 64 == 0 && R <= 512 && dr % 16 == 0 && tc_smem(R, dr) <= 227 * 1024; }

}  // namespace mt

using namespace mt;
typedef __nv_bfloat16 bf16;

extern "C" int mt_mla_prep(int f32, const void* qa, long ldq, const void* qw, int Q, const void* kva, long ldk, const void* kw, int R, int dr, float eps,
                           const int64_t* pos, const float* inv_ts, int interleaved, int S, void* cq, void* lat, void* kr, void* cache_lat, void* cache_kr,
                           long max_len, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, long N, cudaStream_t st) {
  if (N <= 0) return 0;
  const size_t smem = sizeof(float) * dr;
  const bool v4 = Q % 4 == 0 && R % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0;
#define CALL(T, V) mla_prep_kernel<T, V><<<(unsigned)N, 128, smem, st>>>((const T*)qa, ldq, (const T*)qw, Q, (const T*)kva, ldk, (const T*)kw, R, dr, eps, pos, \
                                                                        inv_ts, interleaved, S, (T*)cq, (T*)lat, (T*)kr, (T*)cache_lat, (T*)cache_kr, \
                                                                        max_len, slots, lengths, new_lens)
  if (f32) { if (v4) CALL(float, 4); else CALL(float, 1); }
  else { if (v4) CALL(bf16, 4); else CALL(bf16, 1); }
#undef CALL
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_mla_pack(const void* q, const void* kv, const void* kr, const int64_t* pos, const float* inv_ts, int interleaved, long NQ, long NK, int H,
                           int nope, int dr, int vd, int DQ, int DV, void* qp, void* kp, void* vp, cudaStream_t st) {
  if (NQ <= 0 || NK <= 0) return 0;
  if (DQ % 8 || DV % 8) return -1;
  mla_pack_q_kernel<bf16><<<(unsigned)NQ, 256, sizeof(float) * dr, st>>>((const bf16*)q, pos, inv_ts, interleaved, H, nope, dr, DQ, (bf16*)qp);
  auto k8 = mla_pack_kv_kernel<bf16, 8>;
  auto k1 = mla_pack_kv_kernel<bf16, 1>;
  (nope % 8 || dr % 8 || vd % 8 ? k1 : k8)<<<(unsigned)NK, 256, 0, st>>>((const bf16*)kv, (const bf16*)kr, H, nope, dr, vd, DQ, DV, (bf16*)kp, (bf16*)vp);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_mla_absorb(int f32, const void* q, const void* w, const int64_t* pos, const float* inv_ts, int interleaved, int B, int H, int nope, int dr,
                             int vd, int R, void* qa, cudaStream_t st) {
  if (B <= 0) return 0;
  if (!f32 && B >= 8 && R % 64 == 0 && nope % 16 == 0 && dr % 8 == 0 && nope <= 512) {
    const size_t smem = 2 * ((size_t)nope * 72 + HB * (nope + 8));
    if (int rc = raise_smem(mla_absorb_tc_kernel, smem)) return rc;
    mla_absorb_tc_kernel<<<dim3(H, R / 64, (B + HB - 1) / HB), 128, smem, st>>>((const bf16*)q, (const bf16*)w, pos, inv_ts, interleaved, B, H, nope, dr, vd, R,
                                                                             (bf16*)qa);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  const size_t smem = sizeof(float) * (8 * AB_BT * 256 + dr);
  const dim3 grid(H, (B + AB_BT - 1) / AB_BT, (R + 255) / 256);
#define GO(T, AL) { if (int rc = raise_smem(mla_absorb_kernel<T, AL>, smem)) return rc; \
    mla_absorb_kernel<T, AL><<<grid, 256, smem, st>>>((const T*)q, (const T*)w, pos, inv_ts, interleaved, B, H, nope, dr, vd, R, (T*)qa); }
  if (f32) { if (R % 8 == 0) GO(float, true) else GO(float, false) }
  else { if (R % 8 == 0) GO(bf16, true) else GO(bf16, false) }
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_mla_decode_attn(int f32, const void* qa, const void* lat, const void* kr, long max_len, const int64_t* slots, const int64_t* lengths, int B,
                                  int H, int R, int dr, float scale, int window, int splits, float* part, float* ml, cudaStream_t st) {
  if (B <= 0) return 0;
  if (splits < 1 || splits > 64) return -1;
  const AttnArgs a{H, R, dr, window, splits, max_len, scale, slots, lengths};
  if (tc_form(f32, R, dr)) {
    const size_t smem = tc_smem(R, dr);
    const dim3 grid(splits, (H + 15) / 16, B);
#define GO(CT) case CT: { if (int rc = raise_smem(mla_attn_tc_kernel<CT>, smem)) return rc; \
    mla_attn_tc_kernel<CT><<<grid, TC_NT, smem, st>>>(a, (const bf16*)qa, (const bf16*)lat, (const bf16*)kr, part, ml); break; }
    switch (R / 64) { GO(1) GO(2) GO(3) GO(4) GO(5) GO(6) GO(7) GO(8) default: return -1; }
#undef GO
  } else {
    if (R > 256 * PL_CMAX) return -1;
    const size_t smem = sizeof(float) * ((PL_HG + PL_TILE) * (size_t)(R + dr) + PL_HG * PL_TILE);
    const dim3 grid(splits, (H + PL_HG - 1) / PL_HG, B);
    if (f32) {
      if (int rc = raise_smem(mla_attn_plain_kernel<float>, smem)) return rc;
      mla_attn_plain_kernel<float><<<grid, 256, smem, st>>>(a, (const float*)qa, (const float*)lat, (const float*)kr, part, ml);
    } else {
      if (int rc = raise_smem(mla_attn_plain_kernel<bf16>, smem)) return rc;
      mla_attn_plain_kernel<bf16><<<grid, 256, smem, st>>>(a, (const bf16*)qa, (const bf16*)lat, (const bf16*)kr, part, ml);
    }
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_mla_value_up(int f32, const float* part, const float* ml, const void* w, int B, int H, int nope, int vd, int R, int splits, void* out,
                               cudaStream_t st) {
  if (B <= 0) return 0;
  if (splits < 1 || splits > 64) return -1;
  if (!f32 && B >= 8 && R % 16 == 0 && R <= 512) {
    const size_t tc = 2 * (size_t)(64 + 2 * VB) * (R + 8);
    if (int rc = raise_smem(mla_value_up_tc_kernel, tc)) return rc;
    mla_value_up_tc_kernel<<<dim3(H, (vd + 63) / 64, (B + VB - 1) / VB), 256, tc, st>>>(part, ml, (const bf16*)w, B, H, nope, vd, R, splits, (bf16*)out);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  const size_t smem = sizeof(float) * AB_BT * (size_t)((R + 3) & ~3);
  const dim3 grid(H, (B + AB_BT - 1) / AB_BT, (vd + 63) / 64);
#define GO(T, AL) { if (int rc = raise_smem(mla_value_up_kernel<T, AL>, smem)) return rc; \
    mla_value_up_kernel<T, AL><<<grid, 256, smem, st>>>(part, ml, (const T*)w, B, H, nope, vd, R, splits, (T*)out); }
  if (f32) { if (R % 8 == 0) GO(float, true) else GO(float, false) }
  else { if (R % 8 == 0) GO(bf16, true) else GO(bf16, false) }
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
