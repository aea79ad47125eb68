// Prompts through the recurrent layers in chunks of 64 tokens (bf16 models, head widths that are multiples of 16 up to 128). The recurrences are
// those of recurrent_sm100.cu. Two kernels per layer:
//
//  * prepare, parallel over (chunk, head, sequence): everything that does not depend on the incoming state.
//      gated delta: with G_i the log-decay summed from the chunk's start, r the inverse norms of q and k,
//        L_ij = beta_i rk_i rk_j (k_i . k_j) e^(G_i - G_j)  (j < i),   T = (I + L)^-1,   P_ij = rq_i rk_j (q_i . k_j) e^(G_i - G_j)  (j <= i)
//      gated linear attention: G per key channel;  A_ij = sum_d q_id k_jd e^(G_id - G_jd)  (j <= i),  q e^G,  k e^(G_end - G).
//        Exponents are split at the token before each block row of 16, so that no factor below the diagonal exceeds one; a diagonal block uses the
//        same split while its decay is at most 2^60, and otherwise sums its terms with their own exponents.
//      retention: G_i = (i + 1) log d per head, q and k rotated in fp32; the same tiles as gated linear attention, and its carry.
//      channel-wise gated delta: G per key channel, unit q and k;  L_ij = beta_i sum_d k_id k_jd e^(G_id - G_jd),  P_ij likewise with q_i, exponents
//        split as above;  T = (I + L)^-1,  k e^G,  q e^G,  k e^(G_end - G).
//  * carry, one CTA per (16 state columns, head, sequence), chunk after chunk with the state in fp32 registers and the next chunk's tiles in flight:
//      gated delta:  X = K S, Y = Q S;  R = beta (V - rk e^G X);  U = T R;  O = rq e^G Y + P U;  S <- e^G_end S + K^T (rk e^(G_end - G) U)
//      linear:       O = (q e^G) S + A V;  S <- diag(e^G_end) S + (k e^(G_end - G))^T V
//      channel-wise: R = beta (V - (k e^G) S);  U = T R;  O = (q e^G) S + P U;  S <- diag(e^G_end) S + (k e^(G_end - G))^T U
//
// Products run on mma.sync m16n8k16. q, k, v are exact bf16 operands; every fp32 operand (S, T, P, A, R, U, the decayed q and k) enters as a
// (high, low) bf16 pair, so no factor loses more than its last 8 bits of 24. The tiles are 64 x 16 with a strict chain from chunk to chunk: the
// round trip of an accumulator through tensor memory would cost more than the products themselves.
#include "serving_common.cuh"
#include "warp_mma.cuh"

namespace mt {

typedef __nv_bfloat16 bf16;

constexpr int CH = 64;           // tokens per chunk
constexpr int CN = 16;           // state columns per carry CTA
constexpr int CLD = CH + 8;      // padded row of a 64-wide tile
constexpr int NLD = CN + 8;      // padded row of a 16-wide tile

struct ChunkArgs {
  int H, r, dk, dv, S;           // value heads, value heads per key head, widths, tokens per row of the batch
  int t_lo, t_hi, chunks;        // this launch covers tokens [t_lo, t_hi) of every row in `chunks` chunks
  const int64_t* slots;
  const int64_t* lengths;
  const int64_t* new_lens;       // or null
  float* rec;                    // [slots, H, dk, dv]
};

__device__ __forceinline__ int real_tokens(const ChunkArgs& a, int b) { return min(a.t_hi, a.new_lens ? (int)a.new_lens[b] : a.S); }
__device__ __forceinline__ long chunk_id(const ChunkArgs& a, int b, int c, int h) { return ((long)b * a.chunks + c) * a.H + h; }

// rows [0, CH) of a [CH, dk] bf16 tile to shared memory (row length ld), zeros past row m; dk is a multiple of 8
template <int cols>
__device__ __forceinline__ void tile_async(bf16* dst, int ld, const bf16* src, long stride, int m, int tid, int nt) {
  constexpr int v = cols / 8;
  for (int i = tid; i < CH * v; i += nt) {
    const int r = i / v, c = (i % v) * 8;
    la_cp_async16(dst + r * ld + c, src + (long)(r < m ? r : 0) * stride + c, r < m ? 16 : 0);
  }
}

// T = (I + L)^-1 for the strictly lower triangular L [64][68], as (high, low) bf16 tiles at out and out + 64 * 64. In blocks of 32: the diagonal
// blocks by forward substitution (a warp each, a lane per column), T21 = -T22 (L21 T11) by 128 threads. Called by every thread of the CTA.
__device__ __forceinline__ void unit_lower_inverse(const float* L, float (*Ts)[36], float (*Ms)[36], bf16* out, int tid) {
  const int warp = tid >> 5, lane = tid & 31;
  auto put = [&](int i, int j, float t) {
    const bf16 hi = __float2bfloat16_rn(t);
    out[i * CH + j] = hi;
    out[CH * CH + i * CH + j] = __float2bfloat16_rn(t - __bfloat162float(hi));
  };
  if (warp < 2) {
    const float* l0 = L + warp * 32 * 68 + warp * 32;
    float t[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < i; k += 4) {                   // entries at and right of the diagonal are zero
        const float4 l = *reinterpret_cast<const float4*>(l0 + i * 68 + k);
        s[0] += l.x * t[k];
        if (k + 1 < i) s[1] += l.y * t[k + 1];
        if (k + 2 < i) s[2] += l.z * t[k + 2];
        if (k + 3 < i) s[3] += l.w * t[k + 3];
      }
      t[i] = (i == lane ? 1.f : 0.f) - ((s[0] + s[1]) + (s[2] + s[3]));
      Ts[warp * 32 + i][lane] = t[i];
    }
#pragma unroll 8
    for (int i = 0; i < 32; ++i) put(warp * 32 + i, warp * 32 + lane, Ts[warp * 32 + i][lane]);
  }
  __syncthreads();
  const int row = (tid & 127) >> 2, c8 = (tid & 3) * 8;
  const bool mine = tid < 128;
  float acc[8];
  auto product = [&](const float* x, const float (*y)[36]) {         // acc = x[0 .. 31] . y[0 .. 31][c8 .. c8 + 7]
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll 4
    for (int k = 0; k < 32; ++k) {
      const float f = x[k];
      const float4 u = *reinterpret_cast<const float4*>(&y[k][c8]), v = *reinterpret_cast<const float4*>(&y[k][c8 + 4]);
      acc[0] += f * u.x; acc[1] += f * u.y; acc[2] += f * u.z; acc[3] += f * u.w;
      acc[4] += f * v.x; acc[5] += f * v.y; acc[6] += f * v.z; acc[7] += f * v.w;
    }
  };
  if (mine) {
    product(L + (32 + row) * 68, Ts);
    store_vec<8>(&Ms[row][c8], acc);
  }
  __syncthreads();
  if (mine) {
    product(&Ts[32 + row][0], Ms);
    float neg[8], low[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      neg[e] = -acc[e];
      low[e] = neg[e] - __bfloat162float(__float2bfloat16_rn(neg[e]));
    }
    store_vec<8>(out + (32 + row) * CH + c8, neg);
    store_vec<8>(out + CH * CH + (32 + row) * CH + c8, low);
  }
}

// ------------------------------------------------------------------------------------------------ gated delta: prepare
// grid (chunks, H, B), 128 threads. tp: per chunk and head four [64][64] bf16 tiles: T high, T low, P high, P low;
// gates: per chunk and head [4][64] floats: rk e^G, beta, rq e^G, rk e^(G_end - G), and e^G_end in gate_end.
template <int DK>
__global__ void __launch_bounds__(128) delta_chunk_prepare_kernel(ChunkArgs a, const bf16* __restrict__ mixed, long ldx, const bf16* __restrict__ ba, long ldb,
                                                                  const bf16* __restrict__ A_log, const bf16* __restrict__ dt_bias, bf16* __restrict__ tp,
                                                                  float* __restrict__ gates, float* __restrict__ gate_end) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int dk = DK, LD = DK + 8;
  const int r = a.r, kh = h / r, t0 = a.t_lo + c * CH;
  const int m = min(CH, real_tokens(a, b) - t0);
  if (m <= 0) return;
  bf16* ks = reinterpret_cast<bf16*>(raw);               // [64][LD]
  bf16* qs = ks + CH * LD;
  float* L = reinterpret_cast<float*>(qs + CH * LD);     // [64][68]
  __shared__ float G[CH], beta[CH], rk[CH], rq[CH], half_sum;
  const bf16* row0 = mixed + ((long)b * a.S + t0) * ldx;
  tile_async<dk>(qs, LD, row0 + (long)kh * dk, ldx, m, tid, 128);
  tile_async<dk>(ks, LD, row0 + (long)(a.H / r + kh) * dk, ldx, m, tid, 128);
  la_commit();
  float lg = 0.f;
  if (tid < CH) {
    float be = 0.f;
    if (tid < m) {
      const bf16* bb = ba + ((long)b * a.S + t0 + tid) * ldb + (long)kh * 2 * r + (h - kh * r);
      lg = -expf(to_f(A_log[h])) * softplus_f(to_f(bb[r]) + to_f(dt_bias[h]));
      be = sigmoid_f(to_f(bb[0]));
    }
    beta[tid] = be;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, lg, o);
      if (lane >= o) lg += x;
    }
    if (tid == 31) half_sum = lg;
  }
  la_wait<0>();
  __syncthreads();
  if (tid < CH) G[tid] = lg + (tid >= 32 ? half_sum : 0.f);
  // inverse norms: eight lanes per row, 16 rows of q and k per warp
  for (int i = 0; i < 16; i += 4) {
    const int row = warp * 16 + i + (lane >> 3);
    float sk = 0.f, sq = 0.f;
    for (int d = (lane & 7) * 2; d < dk; d += 16) {
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(ks + row * LD + d));
      const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(qs + row * LD + d));
      sk += x.x * x.x + x.y * x.y;
      sq += y.x * y.x + y.y * y.y;
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) {
      sk += __shfl_xor_sync(0xffffffffu, sk, o);
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
    }
    if ((lane & 7) == 0) {
      rk[row] = rsqrtf(sk + 1e-6f);
      rq[row] = rsqrtf(sq + 1e-6f) * rsqrtf((float)dk);
    }
  }
  __syncthreads();
  // rows 16 warp .. 16 warp + 15 of K K^T and Q K^T, columns up to the diagonal block
  float kk[8][4], qk[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) kk[n][e] = qk[n][e] = 0.f;
  for (int k = 0; k < dk; k += 16) {
    unsigned fk[4], fq[4];
    la_ldm4(fk, ks + (warp * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    la_ldm4(fq, qs + (warp * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      if (n <= 2 * warp) {
        unsigned fb[4];                                  // columns 8 n .. 8 n + 15
        la_ldm4(fb, ks + (n * 8 + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8);
        la_mma(kk[n], fk, fb[0], fb[1]);
        la_mma(kk[n + 1], fk, fb[2], fb[3]);
        la_mma(qk[n], fq, fb[0], fb[1]);
        la_mma(qk[n + 1], fq, fb[2], fb[3]);
      }
    }
  }
  bf16* out = tp + chunk_id(a, b, c, h) * 4 * CH * CH;
#pragma unroll
  for (int n = 0; n < 8; ++n) {
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int i = warp * 16 + (lane >> 2) + (e ? 8 : 0), j = n * 8 + (lane & 3) * 2;
      float l[2] = {0.f, 0.f}, p[2] = {0.f, 0.f};
      if (n <= 2 * warp + 1) {
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          if (j + x <= i) {
            const float f = expf(G[i] - G[j + x]) * rk[j + x];
            p[x] = qk[n][e + x] * f * rq[i];
            if (j + x < i) l[x] = kk[n][e + x] * f * rk[i] * beta[i];
          }
        }
        __nv_bfloat162 hi, lo;
        la_split2(p[0], p[1], hi, lo);
        *reinterpret_cast<__nv_bfloat162*>(out + 2 * CH * CH + i * CH + j) = hi;
        *reinterpret_cast<__nv_bfloat162*>(out + 3 * CH * CH + i * CH + j) = lo;
      }
      *reinterpret_cast<float2*>(L + i * 68 + j) = make_float2(l[0], l[1]);
    }
  }
  __syncthreads();
  if (warp >= 2) {
    const int i = tid - CH;
    float* g = gates + chunk_id(a, b, c, h) * 4 * CH;
    const float end = G[CH - 1];
    g[i] = rk[i] * expf(G[i]);
    g[CH + i] = beta[i];
    g[2 * CH + i] = rq[i] * expf(G[i]);
    g[3 * CH + i] = rk[i] * expf(end - G[i]);
    if (i == 0) gate_end[chunk_id(a, b, c, h)] = expf(end);
  }
  __shared__ __align__(16) float Ts[CH][36], Ms[32][36];
  unit_lower_inverse(L, Ts, Ms, out, tid);
}

// ------------------------------------------------------------------------------------------------ gated linear attention: prepare
// grid (chunks, H, B), 256 threads. aa: per chunk and head A high, A low [64][64]; qkg: per chunk and head four [64][dk] tiles: q e^G high, low,
// k e^(G_end - G) high, low; end: e^G_end [dk].
template <int DK>
__global__ void __launch_bounds__(256) gla_chunk_prepare_kernel(ChunkArgs a, const bf16* __restrict__ x, long ldx, const float* __restrict__ log_alpha,
                                                                bf16* __restrict__ aa, bf16* __restrict__ qkg, float* __restrict__ end) {
  extern __shared__ __align__(16) float sm[];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  constexpr int dk = DK, LD = DK + 4;
  const int H = a.H, t0 = a.t_lo + c * CH;
  const int m = min(CH, real_tokens(a, b) - t0);
  if (m <= 0) return;
  float* G = sm;                                         // [64][LD]
  float* ksc = G + CH * LD;                              // [64][LD] scaled keys up to the diagonal block
  float* qsc = ksc + CH * LD;                            // [16][LD]
  bf16* q = reinterpret_cast<bf16*>(qsc + 16 * LD);      // [64][dk + 8]
  bf16* k = q + CH * (dk + 8);
  constexpr int QLD = dk + 8;
  const bf16* row0 = x + ((long)b * a.S + t0) * ldx;
  tile_async<dk>(q, QLD, row0 + (long)h * dk, ldx, m, tid, 256);
  tile_async<dk>(k, QLD, row0 + (long)(H + h) * dk, ldx, m, tid, 256);
  const float* la = log_alpha + ((long)b * a.S + t0) * H * dk + (long)h * dk;
  for (int i = tid; i < CH * dk / 4; i += 256) {
    const int t = i / (dk / 4), d = (i % (dk / 4)) * 4;
    la_cp_async16(G + t * LD + d, la + (long)(t < m ? t : 0) * H * dk + d, t < m ? 16 : 0);
  }
  la_commit();
  la_wait<0>();
  __syncthreads();
  // running sums down the 64 tokens, in base 2: four segments of 16 tokens per channel, then the segments' offsets
  for (int w = tid; w < 4 * dk; w += 256) {
    float* g = G + (w / dk) * 16 * LD + w % dk;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) { s += g[i * LD] * 1.4426950408889634f; g[i * LD] = s; }
  }
  __syncthreads();
  float off[2] = {0.f, 0.f};                             // 4 dk <= 512 segments over 256 threads
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int w = tid + x * 256;
    if (w < 4 * dk)
      for (int s = 0; s < w / dk; ++s) off[x] += G[(s * 16 + 15) * LD + w % dk];
  }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int w = tid + x * 256;
    if (w < 4 * dk && w >= dk) {
      float* g = G + (w / dk) * 16 * LD + w % dk;
#pragma unroll
      for (int i = 0; i < 16; ++i) g[i * LD] += off[x];
    }
  }
  __syncthreads();
  const float scale = rsqrtf((float)dk);
  const long id = chunk_id(a, b, c, h);
  bf16* qg = qkg + id * 4 * CH * dk;
  for (int i = tid; i < CH * dk / 2; i += 256) {
    const int t = i / (dk / 2), d = (i % (dk / 2)) * 2;
    const float2 qv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + t * QLD + d));
    const float2 kv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + t * QLD + d));
    const float g0 = G[t * LD + d], g1 = G[t * LD + d + 1], e0 = G[(CH - 1) * LD + d], e1 = G[(CH - 1) * LD + d + 1];
    __nv_bfloat162 hi, lo;
    la_split2(qv.x * scale * exp2f(g0), qv.y * scale * exp2f(g1), hi, lo);
    *reinterpret_cast<__nv_bfloat162*>(qg + t * dk + d) = hi;
    *reinterpret_cast<__nv_bfloat162*>(qg + CH * dk + t * dk + d) = lo;
    la_split2(kv.x * exp2f(e0 - g0), kv.y * exp2f(e1 - g1), hi, lo);
    *reinterpret_cast<__nv_bfloat162*>(qg + 2 * CH * dk + t * dk + d) = hi;
    *reinterpret_cast<__nv_bfloat162*>(qg + 3 * CH * dk + t * dk + d) = lo;
  }
  if (tid < dk) end[id * dk + tid] = exp2f(G[(CH - 1) * LD + tid]);
  bf16* ah = aa + id * 2 * CH * CH;
  auto put = [&](int i, int j, float v) {
    const bf16 hi = __float2bfloat16_rn(v);
    ah[i * CH + j] = hi;
    ah[CH * CH + i * CH + j] = __float2bfloat16_rn(v - __bfloat162float(hi));
  };
  // block row by block row: exponents split at the last token before the block row, where no factor can overflow below the diagonal. The diagonal
  // block joins in when its own decay is at most 2^60 in every channel; otherwise its terms are summed with their own exponents.
  const int i0 = tid >> 4, j0 = tid & 15;
  for (int I = 0; I < 4; ++I) {
    const float* ref = G + (I * 16 - 1) * LD;            // not read for I = 0: nothing has decayed there
    bool mild = true;
    if (tid < dk) mild = (I ? ref[tid] : 0.f) - G[(I * 16 + 15) * LD + tid] <= 60.f;
    mild = __syncthreads_and(mild);
    for (int i = tid; i < 16 * dk; i += 256) {
      const int t = i / dk, d = i % dk;
      qsc[t * LD + d] = to_f(q[(I * 16 + t) * QLD + d]) * scale * exp2f(G[(I * 16 + t) * LD + d] - (I ? ref[d] : 0.f));
    }
    const int krows = mild ? I * 16 + 16 : I * 16;
    for (int i = tid; i < krows * dk; i += 256) {
      const int t = i / dk, d = i % dk;
      ksc[t * LD + d] = to_f(k[t * QLD + d]) * exp2f((I ? ref[d] : 0.f) - G[t * LD + d]);
    }
    __syncthreads();
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int d = 0; d < dk; d += 4) {
      const float4 u = *reinterpret_cast<const float4*>(qsc + i0 * LD + d);
#pragma unroll
      for (int J = 0; J < 4; ++J) {
        if (J * 16 < krows) {
          const float4 w = *reinterpret_cast<const float4*>(ksc + (J * 16 + j0) * LD + d);
          s[J] += u.x * w.x + u.y * w.y + u.z * w.z + u.w * w.w;
        }
      }
    }
    if (!mild) {
      const int i = I * 16 + i0, j = I * 16 + j0;
      float t = 0.f;
      if (j <= i)
        for (int d = 0; d < dk; ++d) t += to_f(q[i * QLD + d]) * to_f(k[j * QLD + d]) * exp2f(G[i * LD + d] - G[j * LD + d]);
#pragma unroll
      for (int J = 0; J < 4; ++J)
        if (J == I) s[J] = t * scale;
    }
#pragma unroll
    for (int J = 0; J < 4; ++J)
      if (J <= I) put(I * 16 + i0, J * 16 + j0, J == I && j0 > i0 ? 0.f : s[J]);
  }
}

// ------------------------------------------------------------------------------------------------ retention: prepare
// grid (chunks, H, B), 256 threads. x: q H*dk | k H*dk | .. raw; the outputs are those of gla_chunk_prepare_kernel.
template <int DK>
__global__ void __launch_bounds__(256) retention_chunk_prepare_kernel(ChunkArgs a, const bf16* __restrict__ x, long ldx, const float* __restrict__ log_decay,
                                                                      const float* __restrict__ inv_ts, int rot, bf16* __restrict__ aa, bf16* __restrict__ qkg,
                                                                      float* __restrict__ end) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int dk = DK, LD = DK + 8;
  const int t0 = a.t_lo + c * CH, m = min(CH, real_tokens(a, b) - t0);
  if (m <= 0) return;
  bf16* rq = reinterpret_cast<bf16*>(raw);               // raw tiles [64][LD]
  bf16* rk = rq + CH * LD;
  bf16 *qh = rk + CH * LD, *ql = qh + CH * LD, *kh = ql + CH * LD, *kl = kh + CH * LD;         // rotated, as pairs
  const bf16* row0 = x + ((long)b * a.S + t0) * ldx;
  tile_async<dk>(rq, LD, row0 + (long)h * dk, ldx, m, tid, 256);
  tile_async<dk>(rk, LD, row0 + (long)(a.H + h) * dk, ldx, m, tid, 256);
  la_commit();
  const float l2 = log_decay[h] * 1.4426950408889634f, scale = rsqrtf((float)dk);
  const long pos0 = a.lengths[b] + t0;
  la_wait<0>();
  __syncthreads();
  auto put = [&](bf16* hi, bf16* lo, int at, float v) {
    const bf16 t = __float2bfloat16_rn(v);
    hi[at] = t;
    lo[at] = __float2bfloat16_rn(v - __bfloat162float(t));
  };
  const int half = rot / 2;
  for (int i = tid; i < CH * half; i += 256) {
    const int t = i / half, d = i % half, at = t * LD + d;
    float sn, cs;
    sincosf((float)(pos0 + t) * inv_ts[d], &sn, &cs);
    const float q0 = to_f(rq[at]) * scale, q1 = to_f(rq[at + half]) * scale, k0 = to_f(rk[at]), k1 = to_f(rk[at + half]);
    put(qh, ql, at, q0 * cs - q1 * sn);
    put(qh, ql, at + half, q1 * cs + q0 * sn);
    put(kh, kl, at, k0 * cs - k1 * sn);
    put(kh, kl, at + half, k1 * cs + k0 * sn);
  }
  const int rest = dk - rot;
  for (int i = tid; i < CH * rest; i += 256) {
    const int at = (i / rest) * LD + rot + i % rest;
    put(qh, ql, at, to_f(rq[at]) * scale);
    put(kh, kl, at, to_f(rk[at]));
  }
  __syncthreads();
  const long id = chunk_id(a, b, c, h);
  bf16* qg = qkg + id * 4 * CH * dk;
  for (int i = tid; i < CH * dk / 8; i += 256) {
    const int t = i / (dk / 8), d = (i % (dk / 8)) * 8;
    const float fq = exp2f(l2 * (float)(t + 1)), fk = t < m ? exp2f(l2 * (float)(m - 1 - t)) : 0.f;
    float u[8], v[8];
    load_vec<8>(qh + t * LD + d, u);
    load_vec<8>(ql + t * LD + d, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) { u[e] = (u[e] + v[e]) * fq; v[e] = u[e] - __bfloat162float(__float2bfloat16_rn(u[e])); }
    store_vec<8>(qg + t * dk + d, u);
    store_vec<8>(qg + CH * dk + t * dk + d, v);
    load_vec<8>(kh + t * LD + d, u);
    load_vec<8>(kl + t * LD + d, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) { u[e] = (u[e] + v[e]) * fk; v[e] = u[e] - __bfloat162float(__float2bfloat16_rn(u[e])); }
    store_vec<8>(qg + 2 * CH * dk + t * dk + d, u);
    store_vec<8>(qg + 3 * CH * dk + t * dk + d, v);
  }
  for (int d = tid; d < dk; d += 256) end[id * dk + d] = exp2f(l2 * (float)m);
  // rows 16 rg .., columns 32 half ..
  const int rg = warp & 3, ch = warp >> 2;
  float s[4][4], s1[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[n][e] = s1[n][e] = 0.f;
  for (int k = 0; k < dk; k += 16) {
    unsigned fh[4], fl[4];
    la_ldm4(fh, qh + (rg * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
    la_ldm4(fl, ql + (rg * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
#pragma unroll
    for (int n = 0; n < 4; n += 2) {
      const int col = ch * 32 + n * 8;
      if (col <= rg * 16) {
        unsigned bh[4], bl[4];
        const int off = (col + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8;
        la_ldm4(bh, kh + off);
        la_ldm4(bl, kl + off);
        la_mma(s1[n], fl, bh[0], bh[1]);
        la_mma(s1[n], fh, bl[0], bl[1]);
        la_mma(s[n], fh, bh[0], bh[1]);
        la_mma(s1[n + 1], fl, bh[2], bh[3]);
        la_mma(s1[n + 1], fh, bl[2], bl[3]);
        la_mma(s[n + 1], fh, bh[2], bh[3]);
      }
    }
  }
  bf16* ah = aa + id * 2 * CH * CH;
#pragma unroll
  for (int n = 0; n < 4; ++n) {
    const int j = ch * 32 + n * 8 + (lane & 3) * 2;
    if (ch * 32 + (n & ~1) * 8 > rg * 16) continue;      // blocks above the diagonal are not read
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int i = rg * 16 + (lane >> 2) + (e ? 8 : 0);
      const float p0 = j <= i ? (s[n][e] + s1[n][e]) * exp2f(l2 * (float)(i - j)) : 0.f;
      const float p1 = j + 1 <= i ? (s[n][e + 1] + s1[n][e + 1]) * exp2f(l2 * (float)(i - j - 1)) : 0.f;
      la_split2(p0, p1, *reinterpret_cast<__nv_bfloat162*>(ah + i * CH + j), *reinterpret_cast<__nv_bfloat162*>(ah + CH * CH + i * CH + j));
    }
  }
}

// ------------------------------------------------------------------------------------------------ channel-wise gated delta: prepare
// grid (chunks, H, B), 256 threads. mixed: q | k | v after the convolution; da fp32 [B*S, H*dk]: product of the decay projection. tp: T high, T low,
// P high, P low as for the gated delta rule; qkg: six [64][dk] tiles: k e^G, q e^G, k e^(G_end - G), each high, low; betas [64]; end: e^G_end [dk].
//
// Warp (I, which) owns the 16 rows of block I of P (which 0, rows of q) or of L (1, rows of k). Its rows, scaled by e^(G - r_I) with r_I the sum at
// the last token before the block, stay in registers as fragments; the keys of block J sit in shared memory scaled by e^(G_end(J) - G), so that
// blocks I and J meet through the factor e^(r_I - G_end(J)), which is one for neighbours. No factor exceeds one.
template <int DK>
__global__ void __launch_bounds__(256, 2) channel_chunk_prepare_kernel(ChunkArgs a, const bf16* __restrict__ mixed, long ldx, const bf16* __restrict__ bl,
                                                                       long ldb, const float* __restrict__ da, const bf16* __restrict__ A_log,
                                                                       const bf16* __restrict__ dt_bias, bf16* __restrict__ tp, bf16* __restrict__ qkg,
                                                                       float* __restrict__ betas, float* __restrict__ end) {
  extern __shared__ __align__(16) float sm[];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  constexpr int dk = DK, LD = DK + 4, QLD = DK + 8, NT = 256;
  const int H = a.H, r = a.r, kh = h / r, t0 = a.t_lo + c * CH;
  const int m = min(CH, real_tokens(a, b) - t0);
  if (m <= 0) return;
  constexpr int QK = CH * QLD > CH * 68 ? CH * QLD : CH * 68;            // floats: a pair of bf16 tiles, or L
  float* G = sm;                                         // [64][LD]
  bf16* q = reinterpret_cast<bf16*>(G + CH * LD);        // [64][QLD]
  bf16* k = q + CH * QLD;
  float* L = G + CH * LD;                                // [64][68], over q and k once they are in registers
  bf16* ksh = reinterpret_cast<bf16*>(G + CH * LD + QK); // scaled keys [64][QLD], high and low; later the inverse's tiles
  bf16* ksl = ksh + CH * QLD;
  __shared__ float rk[CH], rq[CH], beta[CH];
  __shared__ int steep;                                  // blocks whose own decay is too strong for one split of the exponents
  const bf16* row0 = mixed + ((long)b * a.S + t0) * ldx;
  tile_async<dk>(q, QLD, row0 + (long)kh * dk, ldx, m, tid, NT);
  tile_async<dk>(k, QLD, row0 + (long)(H / r + kh) * dk, ldx, m, tid, NT);
  const float* dp = da + ((long)b * a.S + t0) * H * dk + (long)h * dk;
  for (int i = tid; i < CH * dk / 4; i += NT) {
    const int t = i / (dk / 4), d = (i % (dk / 4)) * 4;
    la_cp_async16(G + t * LD + d, dp + (long)(t < m ? t : 0) * H * dk + d, t < m ? 16 : 0);
  }
  la_commit();
  const long id = chunk_id(a, b, c, h);
  if (tid < CH) {
    const float be = tid < m ? sigmoid_f(to_f(bl[((long)b * a.S + t0 + tid) * ldb + h])) : 0.f;
    beta[tid] = be;
    betas[id * CH + tid] = be;
  }
  if (tid == 0) steep = 0;
  const float rate = -expf(to_f(A_log[h])) * 1.4426950408889634f, scale = rsqrtf((float)dk);
  la_wait<0>();
  __syncthreads();
  for (int i = 0; i < 8; i += 4) {                       // inverse norms: eight lanes per row, eight rows of q and k per warp
    const int row = warp * 8 + i + (lane >> 3);
    float sk = 0.f, sq = 0.f;
    for (int d = (lane & 7) * 2; d < dk; d += 16) {
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + row * QLD + d));
      const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(q + row * QLD + d));
      sk += x.x * x.x + x.y * x.y;
      sq += y.x * y.x + y.y * y.y;
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1) {
      sk += __shfl_xor_sync(0xffffffffu, sk, o);
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
    }
    if ((lane & 7) == 0) {
      rk[row] = rsqrtf(sk + 1e-6f);
      rq[row] = rsqrtf(sq + 1e-6f) * scale;
    }
  }
  // log decays in base 2, summed down the 64 tokens: segments of 16 tokens, then the segments' offsets
#pragma unroll
  for (int x = 0; x < 2; ++x) {                          // 4 dk <= 512 segments over 256 threads
    const int w = tid + x * NT, seg = w / dk, d = w % dk;
    if (seg < 4) {
      const float dt = to_f(dt_bias[(long)h * dk + d]);
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float* g = G + (seg * 16 + i) * LD + d;
        if (seg * 16 + i < m) s += rate * softplus_f(*g + dt);
        *g = s;
      }
      if (s < -60.f) atomicOr(&steep, 1 << seg);
    }
  }
  __syncthreads();
  float off[2] = {0.f, 0.f};
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int w = tid + x * NT;
    if (w < 4 * dk)
      for (int s = 0; s < w / dk; ++s) off[x] += G[(s * 16 + 15) * LD + w % dk];
  }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int w = tid + x * NT;
    if (w < 4 * dk && w >= dk) {
      float* g = G + (w / dk) * 16 * LD + w % dk;
#pragma unroll
      for (int i = 0; i < 16; ++i) g[i * LD] += off[x];
    }
  }
  __syncthreads();
  bf16* qg = qkg + id * 6 * CH * dk;
  for (int i = tid; i < CH * dk / 8; i += NT) {
    const int t = i / (dk / 8), d = (i % (dk / 8)) * 8;
    float qv[8], kv[8], g[8], x[8], y[8];
    load_vec<8>(q + t * QLD + d, qv);
    load_vec<8>(k + t * QLD + d, kv);
    load_vec<8>(G + t * LD + d, g);
    auto pair = [&](bf16* hi, bf16* lo) {                // x as a (high, low) pair
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = x[e] - __bfloat162float(__float2bfloat16_rn(x[e]));
      store_vec<8>(hi, x);
      store_vec<8>(lo, y);
    };
    bf16* at = qg + t * dk + d;
    float eg[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) { kv[e] *= rk[t]; eg[e] = exp2f(g[e]); x[e] = kv[e] * eg[e]; }
    pair(at, at + CH * dk);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = qv[e] * rq[t] * eg[e];
    pair(at + 2 * CH * dk, at + 3 * CH * dk);
    load_vec<8>(G + (CH - 1) * LD + d, eg);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = kv[e] * exp2f(eg[e] - g[e]);
    pair(at + 4 * CH * dk, at + 5 * CH * dk);
    load_vec<8>(G + (t | 15) * LD + d, eg);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = kv[e] * exp2f(eg[e] - g[e]);
    pair(ksh + t * QLD + d, ksl + t * QLD + d);
  }
  for (int d = tid; d < dk; d += NT) end[id * dk + d] = exp2f(G[(CH - 1) * LD + d]);
  const int I = warp >> 1, which = warp & 1, ra = I * 16 + (lane >> 2), rb = ra + 8, c2 = (lane & 3) * 2;
  const bf16* X = which ? k : q;
  const float fa = which ? rk[ra] : rq[ra], fb = which ? rk[rb] : rq[rb], ka = rk[ra], kb = rk[rb];
  const bool mild = !(steep >> I & 1);
  unsigned ah[DK / 16][4], al[DK / 16][4];
  float d0[4] = {}, d1[4] = {};                          // the diagonal block: columns 0 .. 7 and 8 .. 15
  auto split = [](float u, float v, unsigned& hi, unsigned& lo) {
    __nv_bfloat162 x, y;
    la_split2(u, v, x, y);
    hi = *reinterpret_cast<unsigned*>(&x);
    lo = *reinterpret_cast<unsigned*>(&y);
  };
  auto two = [](const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); };
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
    unsigned bh[4], bo[4];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int col = kk * 16 + e * 8 + c2;
      const float2 ref = I ? *reinterpret_cast<const float2*>(G + (I * 16 - 1) * LD + col) : make_float2(0.f, 0.f);
      const float2 ga = *reinterpret_cast<const float2*>(G + ra * LD + col), gb = *reinterpret_cast<const float2*>(G + rb * LD + col);
      const float2 xa = two(X + ra * QLD + col), xb = two(X + rb * QLD + col);
      split(xa.x * fa * exp2f(ga.x - ref.x), xa.y * fa * exp2f(ga.y - ref.y), ah[kk][2 * e], al[kk][2 * e]);
      split(xb.x * fb * exp2f(gb.x - ref.x), xb.y * fb * exp2f(gb.y - ref.y), ah[kk][2 * e + 1], al[kk][2 * e + 1]);
      if (mild) {
        const float2 ya = two(k + ra * QLD + col), yb = two(k + rb * QLD + col);
        split(ya.x * ka * exp2f(ref.x - ga.x), ya.y * ka * exp2f(ref.y - ga.y), bh[e], bo[e]);
        split(yb.x * kb * exp2f(ref.x - gb.x), yb.y * kb * exp2f(ref.y - gb.y), bh[2 + e], bo[2 + e]);
      }
    }
    if (mild) {
      la_mma(d0, al[kk], bh[0], bh[1]);
      la_mma(d1, al[kk], bh[2], bh[3]);
      la_mma(d0, ah[kk], bo[0], bo[1]);
      la_mma(d1, ah[kk], bo[2], bo[3]);
      la_mma(d0, ah[kk], bh[0], bh[1]);
      la_mma(d1, ah[kk], bh[2], bh[3]);
    }
  }
  if (!mild) {                                           // every term with its own exponents; entries above the diagonal are dropped later
    const int j0 = I * 16 + c2;
    float s00[2] = {}, s10[2] = {}, s11[2] = {};         // rows ra and rb on columns 0 .. 7, row rb on columns 8 .. 15
    for (int d = 0; d < dk; d += 2) {
      const float2 xa = two(X + ra * QLD + d), xb = two(X + rb * QLD + d);
      const float2 ga = *reinterpret_cast<const float2*>(G + ra * LD + d), gb = *reinterpret_cast<const float2*>(G + rb * LD + d);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float2 k0 = two(k + (j0 + e) * QLD + d), k1 = two(k + (j0 + 8 + e) * QLD + d);
        const float2 g0 = *reinterpret_cast<const float2*>(G + (j0 + e) * LD + d), g1 = *reinterpret_cast<const float2*>(G + (j0 + 8 + e) * LD + d);
        s00[e] += xa.x * k0.x * exp2f(ga.x - g0.x) + xa.y * k0.y * exp2f(ga.y - g0.y);
        s10[e] += xb.x * k0.x * exp2f(gb.x - g0.x) + xb.y * k0.y * exp2f(gb.y - g0.y);
        s11[e] += xb.x * k1.x * exp2f(gb.x - g1.x) + xb.y * k1.y * exp2f(gb.y - g1.y);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      d0[e] = s00[e] * fa * rk[j0 + e];
      d0[2 + e] = s10[e] * fb * rk[j0 + e];
      d1[2 + e] = s11[e] * fb * rk[j0 + 8 + e];
    }
  }
  __syncthreads();                                       // L takes the place of q and k; the scaled keys are visible
  bf16* out = tp + id * 4 * CH * CH;
  const float ba = beta[ra], bb = beta[rb];
  auto put = [&](int j, const float* s) {                // columns j, j + 1 of rows ra and rb
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int i = e ? rb : ra;
      if (which) {
        const float be = e ? bb : ba;
        *reinterpret_cast<float2*>(L + i * 68 + j) = make_float2(j < i ? be * s[e] : 0.f, j + 1 < i ? be * s[e + 1] : 0.f);
      } else {
        la_split2(j <= i ? s[e] : 0.f, j + 1 <= i ? s[e + 1] : 0.f, *reinterpret_cast<__nv_bfloat162*>(out + 2 * CH * CH + i * CH + j),
                  *reinterpret_cast<__nv_bfloat162*>(out + 3 * CH * CH + i * CH + j));
      }
    }
  };
  put(I * 16 + c2, d0);
  put(I * 16 + 8 + c2, d1);
  if (which) {
    const float zero[4] = {};
    for (int j = (I + 1) * 16 + c2; j < CH; j += 8) put(j, zero);
  }
  for (int J = 0; J < I; ++J) {
    float s0[4] = {}, s1[4] = {};
    const int off2 = (J * 16 + (lane & 7) + ((lane >> 4) << 3)) * QLD + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      unsigned th[4], tl[4], bh[4], bo[4];
      la_ldm4(bh, ksh + off2 + kk * 16);
      la_ldm4(bo, ksl + off2 + kk * 16);
      if (J + 1 == I) {
#pragma unroll
        for (int e = 0; e < 4; ++e) { th[e] = ah[kk][e]; tl[e] = al[kk][e]; }
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = kk * 16 + e * 8 + c2;
          const float2 ref = *reinterpret_cast<const float2*>(G + (I * 16 - 1) * LD + col), ge = *reinterpret_cast<const float2*>(G + (J * 16 + 15) * LD + col);
          const float f0 = exp2f(ref.x - ge.x), f1 = exp2f(ref.y - ge.y);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ah[kk][2 * e + x]));
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&al[kk][2 * e + x]));
            split((u.x + v.x) * f0, (u.y + v.y) * f1, th[2 * e + x], tl[2 * e + x]);
          }
        }
      }
      la_mma(s0, tl, bh[0], bh[1]);
      la_mma(s1, tl, bh[2], bh[3]);
      la_mma(s0, th, bo[0], bo[1]);
      la_mma(s1, th, bo[2], bo[3]);
      la_mma(s0, th, bh[0], bh[1]);
      la_mma(s1, th, bh[2], bh[3]);
    }
    put(J * 16 + c2, s0);
    put(J * 16 + 8 + c2, s1);
  }
  __syncthreads();
  float (*Ts)[36] = reinterpret_cast<float (*)[36]>(ksh);
  unit_lower_inverse(L, Ts, Ts + CH, out, tid);
}

// ------------------------------------------------------------------------------------------------ channel-wise gated delta: carry
// grid (dv / 16, H, B), 256 threads; the roles are those of chunk_carry_kernel. The six tiles of a chunk leave no room for a second stage, so
// they come in two groups: what R needs is fetched while the chunk before finishes, the rest while R is formed.
template <int DK>
__global__ void __launch_bounds__(256) channel_carry_kernel(ChunkArgs a, const bf16* __restrict__ x, long ldx, long voff, const bf16* __restrict__ tiles,
                                                            const bf16* __restrict__ qkg, const float* __restrict__ betas, const float* __restrict__ ends,
                                                            bf16* __restrict__ o) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = warp & 3, half = warp >> 2;
  constexpr int dk = DK, LD = DK + 8;
  const int dv = a.dv, H = a.H, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * CN;
  const int n = real_tokens(a, b), chunks = (n - a.t_lo + CH - 1) / CH;
  bf16* qk = reinterpret_cast<bf16*>(raw);               // six [64][LD]: k e^G, q e^G, k e^(G_end - G), high and low
  bf16* tpt = qk + 6 * CH * LD;                          // four [64][CLD]: T, P, high and low
  bf16* v = tpt + 4 * CH * CLD;                          // [64][NLD]
  bf16* Sh = v + CH * NLD;                               // [dk][NLD] high, low
  bf16* Sl = Sh + dk * NLD;
  bf16* W = Sl + dk * NLD;                               // R high, low, U high, low: [64][NLD] each
  float* be = reinterpret_cast<float*>(W + 4 * CH * NLD);          // [64]
  float* en = be + CH;                                   // [dk]
  auto first = [&](int c) {
    const int t0 = a.t_lo + c * CH, m = min(CH, n - t0);
    const long id = chunk_id(a, b, c, h);
    for (int i = 0; i < 4; ++i) tile_async<dk>(qk + i * CH * LD, LD, qkg + (id * 6 + i) * CH * dk, dk, CH, tid, 256);
    tile_async<CN>(v, NLD, x + ((long)b * a.S + t0) * ldx + voff + (long)h * dv + c0, ldx, m, tid, 256);
    for (int i = tid; i < CH / 4; i += 256) la_cp_async16(be + i * 4, betas + id * CH + i * 4, 16);
    la_commit();
  };
  auto second = [&](int c) {
    const long id = chunk_id(a, b, c, h);
    for (int i = 0; i < 4; ++i) tile_async<CH>(tpt + i * CH * CLD, CLD, tiles + (id * 4 + i) * CH * CH, CH, CH, tid, 256);
    for (int i = 4; i < 6; ++i) tile_async<dk>(qk + i * CH * LD, LD, qkg + (id * 6 + i) * CH * dk, dk, CH, tid, 256);
    for (int i = tid; i < dk / 4; i += 256) la_cp_async16(en + i * 4, ends + id * dk + i * 4, 16);
    la_commit();
  };
  const long slot = a.slots[b];
  const bool fresh = a.lengths[b] == 0 && a.t_lo == 0;
  float* sp = a.rec + (slot * H + h) * (long)dk * dv + c0;
  const bool owns = warp * 16 < dk;                      // warps past the key width hold no state rows
  float S[2][4];
  const int gr = lane >> 2, kc = (lane & 3) * 2;
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      S[nt][e] = (!fresh && owns) ? sp[(long)(warp * 16 + gr + (e >> 1) * 8) * dv + nt * 8 + kc + (e & 1)] : 0.f;
  auto publish = [&]() {
    if (!owns) return;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int at = (warp * 16 + gr + (e >> 1) * 8) * NLD + nt * 8 + kc;
        la_split2(S[nt][e], S[nt][e + 1], *reinterpret_cast<__nv_bfloat162*>(Sh + at), *reinterpret_cast<__nv_bfloat162*>(Sl + at));
      }
  };
  publish();
  if (chunks > 0) first(0);
  const int arow = rg * 16 + (lane & 15), acol = (lane >> 4) * 8, brow = lane & 15, i0 = rg * 16 + gr;
  for (int c = 0; c < chunks; ++c) {
    const int t0 = a.t_lo + c * CH;
    la_wait<0>();
    __syncthreads();                                     // the first group and S are visible, the second group's tiles are free
    second(c);
    float xx[4] = {}, x1[4] = {}, x2[4] = {}, y[4] = {}, y1[4] = {}, y2[4] = {};
#pragma unroll
    for (int k = 0; k < dk; k += 16) {
      unsigned kh[4], kl[4], qh[4], ql[4], sh[2], sl[2];
      la_ldm4(kh, qk + arow * LD + k + acol);
      la_ldm4(kl, qk + CH * LD + arow * LD + k + acol);
      la_ldm4(qh, qk + 2 * CH * LD + arow * LD + k + acol);
      la_ldm4(ql, qk + 3 * CH * LD + arow * LD + k + acol);
      la_ldm2t(sh, Sh + (k + brow) * NLD + half * 8);
      la_ldm2t(sl, Sl + (k + brow) * NLD + half * 8);
      la_mma(x1, kl, sh[0], sh[1]);
      la_mma(x2, kh, sl[0], sl[1]);
      la_mma(y1, ql, sh[0], sh[1]);
      la_mma(y2, qh, sl[0], sl[1]);
      la_mma(xx, kh, sh[0], sh[1]);
      la_mma(y, qh, sh[0], sh[1]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) { xx[e] += x1[e] + x2[e]; y[e] += y1[e] + y2[e]; }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = i0 + e * 8, at = i * NLD + half * 8 + kc;
      const float2 vv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + at));
      la_split2(be[i] * (vv.x - xx[2 * e]), be[i] * (vv.y - xx[2 * e + 1]), *reinterpret_cast<__nv_bfloat162*>(W + at),
                *reinterpret_cast<__nv_bfloat162*>(W + CH * NLD + at));
    }
    la_wait<0>();
    __syncthreads();                                     // R and the second group are visible, the first group's tiles are free
    if (c + 1 < chunks) first(c + 1);
    float u[4] = {}, u1[4] = {}, u2[4] = {};
#pragma unroll
    for (int k = 0; k < CH; k += 16) {
      if (k > rg * 16) break;                            // T is lower triangular
      unsigned th[4], tl[4], rh[2], rl[2];
      la_ldm4(th, tpt + arow * CLD + k + acol);
      la_ldm4(tl, tpt + CH * CLD + arow * CLD + k + acol);
      la_ldm2t(rh, W + (k + brow) * NLD + half * 8);
      la_ldm2t(rl, W + CH * NLD + (k + brow) * NLD + half * 8);
      la_mma(u1, tl, rh[0], rh[1]);
      la_mma(u2, th, rl[0], rl[1]);
      la_mma(u, th, rh[0], rh[1]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int at = (i0 + e * 8) * NLD + half * 8 + kc;
      la_split2(u[2 * e] + u1[2 * e] + u2[2 * e], u[2 * e + 1] + u1[2 * e + 1] + u2[2 * e + 1], *reinterpret_cast<__nv_bfloat162*>(W + 2 * CH * NLD + at),
                *reinterpret_cast<__nv_bfloat162*>(W + 3 * CH * NLD + at));
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 4; ++e) y1[e] = y2[e] = 0.f;
#pragma unroll
    for (int k = 0; k < CH; k += 16) {
      if (k > rg * 16) break;
      unsigned ph[4], pl[4], uh[2], ul[2];
      la_ldm4(ph, tpt + 2 * CH * CLD + arow * CLD + k + acol);
      la_ldm4(pl, tpt + 3 * CH * CLD + arow * CLD + k + acol);
      la_ldm2t(uh, W + 2 * CH * NLD + (k + brow) * NLD + half * 8);
      la_ldm2t(ul, W + 3 * CH * NLD + (k + brow) * NLD + half * 8);
      la_mma(y1, pl, uh[0], uh[1]);
      la_mma(y2, ph, ul[0], ul[1]);
      la_mma(y, ph, uh[0], uh[1]);
    }
    if (owns) {
      const float e0 = en[warp * 16 + gr], e1 = en[warp * 16 + gr + 8];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) { S[nt][0] *= e0; S[nt][1] *= e0; S[nt][2] *= e1; S[nt][3] *= e1; }
#pragma unroll
      for (int k = 0; k < CH; k += 16) {
        unsigned kh[4], kl[4], uh[4], ul[4];
        la_ldm4t(kh, qk + 4 * CH * LD + (k + la_at_row(lane)) * LD + warp * 16 + la_at_col(lane));
        la_ldm4t(kl, qk + 5 * CH * LD + (k + la_at_row(lane)) * LD + warp * 16 + la_at_col(lane));
        la_ldm4t(uh, W + 2 * CH * NLD + (k + brow) * NLD + (lane >> 4) * 8);
        la_ldm4t(ul, W + 3 * CH * NLD + (k + brow) * NLD + (lane >> 4) * 8);
        la_mma(S[0], kl, uh[0], uh[1]);
        la_mma(S[1], kl, uh[2], uh[3]);
        la_mma(S[0], kh, ul[0], ul[1]);
        la_mma(S[1], kh, ul[2], ul[3]);
        la_mma(S[0], kh, uh[0], uh[1]);
        la_mma(S[1], kh, uh[2], uh[3]);
      }
    }
    publish();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + i0 + e * 8;
      if (t < n)
        *reinterpret_cast<__nv_bfloat162*>(o + (((long)b * a.S + t) * H + h) * dv + c0 + half * 8 + kc) =
            __floats2bfloat162_rn(y[2 * e] + y1[2 * e] + y2[2 * e], y[2 * e + 1] + y1[2 * e + 1] + y2[2 * e + 1]);
    }
  }
  if (owns) {
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) sp[(long)(warp * 16 + gr + (e >> 1) * 8) * dv + nt * 8 + kc + (e & 1)] = S[nt][e];
  }
  for (int i = tid; i < (a.t_hi - max(n, a.t_lo)) * CN; i += 256)         // padding positions are read by the norm kernel: give them a value
    o[(((long)b * a.S + max(n, a.t_lo) + i / CN) * H + h) * dv + c0 + i % CN] = __float2bfloat16_rn(0.f);
}

template <int DK>
int launch_channel(const ChunkArgs& a, const bf16* mixed, long ldx, long voff, const bf16* beta, long ldb, const float* da, const bf16* A_log, const bf16* dt,
                   bf16* tp, bf16* qkg, float* betas, float* ends, bf16* o, int B, cudaStream_t st) {
  constexpr int two = CH * (DK + 8), QK = two > CH * 68 ? two : CH * 68, KS = two > 96 * 36 ? two : 96 * 36;       // floats: a pair of bf16 tiles each
  constexpr int s1 = 4 * (CH * (DK + 4) + QK + KS);
  constexpr int s2 = 2 * (6 * CH * (DK + 8) + 4 * CH * CLD + CH * NLD + 2 * DK * NLD + 4 * CH * NLD) + 4 * (CH + DK);
  if (cudaFuncSetAttribute(channel_chunk_prepare_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, s1) != cudaSuccess) return -2;
  if (cudaFuncSetAttribute(channel_carry_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, s2) != cudaSuccess) return -2;
  channel_chunk_prepare_kernel<DK><<<dim3(a.chunks, a.H, B), 256, s1, st>>>(a, mixed, ldx, beta, ldb, da, A_log, dt, tp, qkg, betas, ends);
  channel_carry_kernel<DK><<<dim3(a.dv / CN, a.H, B), 256, s2, st>>>(a, mixed, ldx, voff, tp, qkg, betas, ends, o);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

// ------------------------------------------------------------------------------------------------ carry
// grid (dv / 16, H, B), 256 threads: warp (rg, half) = (w & 3, w >> 2) forms rows 16 rg .. of the token-by-column tiles, columns 8 half ..;
// warp w holds state rows 16 w .. 16 w + 15.
template <bool DELTA, int DK>
__global__ void __launch_bounds__(256) chunk_carry_kernel(ChunkArgs a, const bf16* __restrict__ x, long ldx, long koff, long voff,
                                                          const bf16* __restrict__ tiles, const bf16* __restrict__ qkg, const float* __restrict__ gates,
                                                          const float* __restrict__ ends, bf16* __restrict__ o) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = warp & 3, half = warp >> 2;
  constexpr int dk = DK, LD = DK + 8;
  const int dv = a.dv, H = a.H, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * CN, kh = h / a.r;
  const int n = real_tokens(a, b), chunks = (n - a.t_lo + CH - 1) / CH;
  constexpr int NQK = DELTA ? 2 : 4, NTP = DELTA ? 4 : 2;
  // one stage: q / k tiles, v tile, 64 x 64 tiles, gates
  constexpr size_t st_qk = (size_t)CH * LD, st_v = (size_t)CH * NLD, st_tp = (size_t)CH * CLD;
  constexpr size_t stage = (NQK * st_qk + st_v + NTP * st_tp) * 2 + 4 * CH * 4;
  auto qkt = [&](int buf, int i) { return reinterpret_cast<bf16*>(raw + buf * stage) + i * st_qk; };
  auto vt = [&](int buf) { return reinterpret_cast<bf16*>(raw + buf * stage) + NQK * st_qk; };
  auto tpt = [&](int buf, int i) { return reinterpret_cast<bf16*>(raw + buf * stage) + NQK * st_qk + st_v + i * st_tp; };
  auto gt = [&](int buf) { return reinterpret_cast<float*>(raw + buf * stage + (NQK * st_qk + st_v + NTP * st_tp) * 2); };
  bf16* Sh = reinterpret_cast<bf16*>(raw + 2 * stage);   // [dk][NLD] high, low
  bf16* Sl = Sh + dk * NLD;
  bf16* W = Sl + dk * NLD;                               // gated delta: R high, low, U high, low, decayed U high, low: [64][NLD] each

  auto issue = [&](int c, int buf) {
    const int t0 = a.t_lo + c * CH, m = min(CH, n - t0);
    const long id = chunk_id(a, b, c, h);
    const bf16* row0 = x + ((long)b * a.S + t0) * ldx;
    if constexpr (DELTA) {
      tile_async<dk>(qkt(buf, 0), LD, row0 + (long)kh * dk, ldx, m, tid, 256);
      tile_async<dk>(qkt(buf, 1), LD, row0 + koff + (long)kh * dk, ldx, m, tid, 256);
    } else {
      for (int i = 0; i < 4; ++i) tile_async<dk>(qkt(buf, i), LD, qkg + (id * 4 + i) * CH * dk, dk, CH, tid, 256);
    }
    tile_async<CN>(vt(buf), NLD, row0 + voff + (long)h * dv + c0, ldx, m, tid, 256);
    for (int i = 0; i < NTP; ++i) tile_async<CH>(tpt(buf, i), CLD, tiles + (id * NTP + i) * CH * CH, CH, CH, tid, 256);
    const float* g = DELTA ? gates + id * 4 * CH : ends + id * dk;
    for (int i = tid; i < (DELTA ? CH : dk / 4); i += 256) la_cp_async16(gt(buf) + i * 4, g + i * 4, 16);
    la_commit();
  };

  const long slot = a.slots[b];
  const bool fresh = a.lengths[b] == 0 && a.t_lo == 0;
  float* sp = a.rec + (slot * H + h) * (long)dk * dv + c0;
  const bool owns = warp * 16 < dk;                      // warps past the key width hold no state rows
  float S[2][4];
  const int gr = lane >> 2, kc = (lane & 3) * 2;
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      S[nt][e] = (!fresh && owns) ? sp[(long)(warp * 16 + gr + (e >> 1) * 8) * dv + nt * 8 + kc + (e & 1)] : 0.f;
  auto publish = [&]() {
    if (!owns) return;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int at = (warp * 16 + gr + (e >> 1) * 8) * NLD + nt * 8 + kc;
        la_split2(S[nt][e], S[nt][e + 1], *reinterpret_cast<__nv_bfloat162*>(Sh + at), *reinterpret_cast<__nv_bfloat162*>(Sl + at));
      }
  };
  publish();
  if (chunks > 0) issue(0, 0);
  for (int c = 0; c < chunks; ++c) {
    const int buf = c & 1, t0 = a.t_lo + c * CH;
    la_wait<0>();
    __syncthreads();                                     // this chunk's tiles and S are visible; the other stage is free
    if (c + 1 < chunks) issue(c + 1, buf ^ 1);
    const float* g = gt(buf);
    const int arow = rg * 16 + (lane & 15), acol = (lane >> 4) * 8, brow = lane & 15;
    const int i0 = rg * 16 + gr;                         // this thread's rows of a token tile: i0, i0 + 8
    float y[4] = {0.f, 0.f, 0.f, 0.f};
    if constexpr (DELTA) {
      float xx[4] = {0.f, 0.f, 0.f, 0.f}, xl[4] = {0.f, 0.f, 0.f, 0.f}, yl[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < dk; k += 16) {
        unsigned fq[4], fk[4], sh[2], sl[2];
        la_ldm4(fq, qkt(buf, 0) + arow * LD + k + acol);
        la_ldm4(fk, qkt(buf, 1) + arow * LD + k + acol);
        la_ldm2t(sh, Sh + (k + brow) * NLD + half * 8);
        la_ldm2t(sl, Sl + (k + brow) * NLD + half * 8);
        la_mma(xl, fk, sl[0], sl[1]);
        la_mma(yl, fq, sl[0], sl[1]);
        la_mma(xx, fk, sh[0], sh[1]);
        la_mma(y, fq, sh[0], sh[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) { xx[e] += xl[e]; y[e] += yl[e]; }
      const bf16* v = vt(buf);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = i0 + e * 8, at = i * NLD + half * 8 + kc;
        const float2 vv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + at));
        const float be = g[CH + i], ek = g[i];
        la_split2(be * (vv.x - ek * xx[2 * e]), be * (vv.y - ek * xx[2 * e + 1]), *reinterpret_cast<__nv_bfloat162*>(W + at),
                  *reinterpret_cast<__nv_bfloat162*>(W + CH * NLD + at));
      }
      __syncthreads();
      float u[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f}, u2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < CH; k += 16) {
        if (k > rg * 16) break;                          // T is lower triangular
        unsigned th[4], tl[4], rh[2], rl[2];
        la_ldm4(th, tpt(buf, 0) + arow * CLD + k + acol);
        la_ldm4(tl, tpt(buf, 1) + arow * CLD + k + acol);
        la_ldm2t(rh, W + (k + brow) * NLD + half * 8);
        la_ldm2t(rl, W + CH * NLD + (k + brow) * NLD + half * 8);
        la_mma(u1, tl, rh[0], rh[1]);
        la_mma(u2, th, rl[0], rl[1]);
        la_mma(u, th, rh[0], rh[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) u[e] += u1[e] + u2[e];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = i0 + e * 8, at = i * NLD + half * 8 + kc;
        const float kd = g[3 * CH + i];
        la_split2(u[2 * e], u[2 * e + 1], *reinterpret_cast<__nv_bfloat162*>(W + 2 * CH * NLD + at),
                  *reinterpret_cast<__nv_bfloat162*>(W + 3 * CH * NLD + at));
        la_split2(kd * u[2 * e], kd * u[2 * e + 1], *reinterpret_cast<__nv_bfloat162*>(W + 4 * CH * NLD + at),
                  *reinterpret_cast<__nv_bfloat162*>(W + 5 * CH * NLD + at));
      }
      __syncthreads();
      y[0] *= g[2 * CH + i0]; y[1] *= g[2 * CH + i0]; y[2] *= g[2 * CH + i0 + 8]; y[3] *= g[2 * CH + i0 + 8];
      float y1[4] = {0.f, 0.f, 0.f, 0.f}, y2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < CH; k += 16) {
        if (k > rg * 16) break;
        unsigned ph[4], pl[4], uh[2], ul[2];
        la_ldm4(ph, tpt(buf, 2) + arow * CLD + k + acol);
        la_ldm4(pl, tpt(buf, 3) + arow * CLD + k + acol);
        la_ldm2t(uh, W + 2 * CH * NLD + (k + brow) * NLD + half * 8);
        la_ldm2t(ul, W + 3 * CH * NLD + (k + brow) * NLD + half * 8);
        la_mma(y1, pl, uh[0], uh[1]);
        la_mma(y2, ph, ul[0], ul[1]);
        la_mma(y, ph, uh[0], uh[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] += y1[e] + y2[e];
      if (owns) {
        const float ge = ends[chunk_id(a, b, c, h)];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[nt][e] *= ge;
#pragma unroll
        for (int k = 0; k < CH; k += 16) {
          unsigned fk[4], uh[4], ul[4];
          la_ldm4t(fk, qkt(buf, 1) + (k + la_at_row(lane)) * LD + warp * 16 + la_at_col(lane));
          la_ldm4t(uh, W + 4 * CH * NLD + (k + brow) * NLD + (lane >> 4) * 8);
          la_ldm4t(ul, W + 5 * CH * NLD + (k + brow) * NLD + (lane >> 4) * 8);
          la_mma(S[0], fk, ul[0], ul[1]);
          la_mma(S[1], fk, ul[2], ul[3]);
          la_mma(S[0], fk, uh[0], uh[1]);
          la_mma(S[1], fk, uh[2], uh[3]);
        }
      }
    } else {
      float y1[4] = {0.f, 0.f, 0.f, 0.f}, y2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < dk; k += 16) {
        unsigned qh[4], ql[4], sh[2], sl[2];
        la_ldm4(qh, qkt(buf, 0) + arow * LD + k + acol);
        la_ldm4(ql, qkt(buf, 1) + arow * LD + k + acol);
        la_ldm2t(sh, Sh + (k + brow) * NLD + half * 8);
        la_ldm2t(sl, Sl + (k + brow) * NLD + half * 8);
        la_mma(y1, ql, sh[0], sh[1]);
        la_mma(y2, qh, sl[0], sl[1]);
        la_mma(y, qh, sh[0], sh[1]);
      }
#pragma unroll
      for (int k = 0; k < CH; k += 16) {
        if (k > rg * 16) break;                          // A is lower triangular
        unsigned fh[4], fl[4], fv[2];
        la_ldm4(fh, tpt(buf, 0) + arow * CLD + k + acol);
        la_ldm4(fl, tpt(buf, 1) + arow * CLD + k + acol);
        la_ldm2t(fv, vt(buf) + (k + brow) * NLD + half * 8);
        la_mma(y1, fl, fv[0], fv[1]);
        la_mma(y2, fh, fv[0], fv[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] += y1[e] + y2[e];
      if (owns) {
        const float e0 = g[warp * 16 + gr], e1 = g[warp * 16 + gr + 8];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) { S[nt][0] *= e0; S[nt][1] *= e0; S[nt][2] *= e1; S[nt][3] *= e1; }
#pragma unroll
        for (int k = 0; k < CH; k += 16) {
          unsigned kh_[4], kl[4], fv[4];
          la_ldm4t(kh_, qkt(buf, 2) + (k + la_at_row(lane)) * LD + warp * 16 + la_at_col(lane));
          la_ldm4t(kl, qkt(buf, 3) + (k + la_at_row(lane)) * LD + warp * 16 + la_at_col(lane));
          la_ldm4t(fv, vt(buf) + (k + brow) * NLD + (lane >> 4) * 8);
          la_mma(S[0], kl, fv[0], fv[1]);
          la_mma(S[1], kl, fv[2], fv[3]);
          la_mma(S[0], kh_, fv[0], fv[1]);
          la_mma(S[1], kh_, fv[2], fv[3]);
        }
      }
      __syncthreads();                                   // every warp has read S
    }
    publish();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + i0 + e * 8;
      if (t < n)
        *reinterpret_cast<__nv_bfloat162*>(o + (((long)b * a.S + t) * H + h) * dv + c0 + half * 8 + kc) = __floats2bfloat162_rn(y[2 * e], y[2 * e + 1]);
    }
  }
  if (owns) {
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) sp[(long)(warp * 16 + gr + (e >> 1) * 8) * dv + nt * 8 + kc + (e & 1)] = S[nt][e];
  }
  for (int i = tid; i < (a.t_hi - max(n, a.t_lo)) * CN; i += 256)         // padding positions are read by the norm kernel: give them a value
    o[(((long)b * a.S + max(n, a.t_lo) + i / CN) * H + h) * dv + c0 + i % CN] = __float2bfloat16_rn(0.f);
}

size_t carry_smem(int delta, int dk) {
  const size_t nqk = delta ? 2 : 4, ntp = delta ? 4 : 2;
  const size_t stage = (nqk * CH * (dk + 8) + (size_t)CH * NLD + ntp * CH * CLD) * 2 + 4 * CH * 4;
  return 2 * stage + 2 * (2 * (size_t)dk * NLD + (delta ? 6 * CH * NLD : 0));
}

template <bool DELTA, int DK>
int launch_carry_dk(const ChunkArgs& a, const bf16* x, long ldx, long koff, long voff, const bf16* tiles, const bf16* qkg, const float* gates,
                    const float* ends, bf16* o, int B, cudaStream_t st) {
  const size_t smem = carry_smem(DELTA, DK);
  auto k = chunk_carry_kernel<DELTA, DK>;
  if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
  k<<<dim3(a.dv / CN, a.H, B), 256, smem, st>>>(a, x, ldx, koff, voff, tiles, qkg, gates, ends, o);
  return 0;
}
template <bool DELTA>
int launch_carry(const ChunkArgs& a, const bf16* x, long ldx, long koff, long voff, const bf16* tiles, const bf16* qkg, const float* gates,
                 const float* ends, bf16* o, int B, cudaStream_t st) {
  switch (a.dk) {
#define GO(DK) case DK: return launch_carry_dk<DELTA, DK>(a, x, ldx, koff, voff, tiles, qkg, gates, ends, o, B, st);
    GO(16) GO(32) GO(48) GO(64) GO(80) GO(96) GO(112) GO(128)
#undef GO
    default: return -1;
  }
}

}  // namespace mt

using namespace mt;

// both halves of the layer fit the chunked kernels
extern "C" int mt_chunk_supported(int dk, int dv) { return dk % 16 == 0 && dk >= 16 && dk <= 128 && dv % 16 == 0 && dv >= 16; }

extern "C" int mt_delta_chunks(const void* mixed, long ldx, const void* ba, long ldb, const void* A_log, const void* dt_bias, int hk, int hv, int dk, int dv,
                               int S, int t_lo, int t_hi, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* tp,
                               float* gates, float* ends, void* o, int B, cudaStream_t st) {
  if (!mt_chunk_supported(dk, dv) || ldx % 8) return -1;
  const ChunkArgs a{hv, hv / hk, dk, dv, S, t_lo, t_hi, (t_hi - t_lo + CH - 1) / CH, slots, lengths, new_lens, rec};
  const size_t s1 = 2 * 2 * (size_t)CH * (dk + 8) + 4 * CH * 68;
  switch (dk) {
#define GO(DK) case DK: \
    if (cudaFuncSetAttribute(delta_chunk_prepare_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1) != cudaSuccess) return -2; \
    delta_chunk_prepare_kernel<DK><<<dim3(a.chunks, hv, B), 128, s1, st>>>(a, (const bf16*)mixed, ldx, (const bf16*)ba, ldb, (const bf16*)A_log, \
                                                                          (const bf16*)dt_bias, (bf16*)tp, gates, ends); break;
    GO(16) GO(32) GO(48) GO(64) GO(80) GO(96) GO(112) GO(128)
#undef GO
  }
  if (int rc = launch_carry<true>(a, (const bf16*)mixed, ldx, (long)hk * dk, 2L * hk * dk, (const bf16*)tp, nullptr, gates, ends, (bf16*)o, B, st)) return rc;
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_gla_chunks(const void* x, long ldx, const float* log_alpha, int H, int dk, int dv, int S, int t_lo, int t_hi, float* rec,
                             const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* aa, void* qkg, float* ends, void* o, int B,
                             cudaStream_t st) {
  if (!mt_chunk_supported(dk, dv) || ldx % 8) return -1;
  const ChunkArgs a{H, 1, dk, dv, S, t_lo, t_hi, (t_hi - t_lo + CH - 1) / CH, slots, lengths, new_lens, rec};
  const size_t s1 = 4 * (size_t)(2 * CH + 16) * (dk + 4) + 2 * 2 * (size_t)CH * (dk + 8);
  switch (dk) {
#define GO(DK) case DK: \
    if (cudaFuncSetAttribute(gla_chunk_prepare_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1) != cudaSuccess) return -2; \
    gla_chunk_prepare_kernel<DK><<<dim3(a.chunks, H, B), 256, s1, st>>>(a, (const bf16*)x, ldx, log_alpha, (bf16*)aa, (bf16*)qkg, ends); break;
    GO(16) GO(32) GO(48) GO(64) GO(80) GO(96) GO(112) GO(128)
#undef GO
  }
  if (int rc = launch_carry<false>(a, (const bf16*)x, ldx, 0, 2L * H * dk, (const bf16*)aa, (const bf16*)qkg, nullptr, ends, (bf16*)o, B, st)) return rc;
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_retention_chunks(const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, int H, int dk, int dv, int S, int t_lo,
                                   int t_hi, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* aa, void* qkg, float* ends,
                                   void* o, int B, cudaStream_t st) {
  if (!mt_chunk_supported(dk, dv) || ldx % 8) return -1;
  const ChunkArgs a{H, 1, dk, dv, S, t_lo, t_hi, (t_hi - t_lo + CH - 1) / CH, slots, lengths, new_lens, rec};
  const size_t s1 = 6 * 2 * (size_t)CH * (dk + 8);
  switch (dk) {
#define GO(DK) case DK: \
    if (cudaFuncSetAttribute(retention_chunk_prepare_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1) != cudaSuccess) return -2; \
    retention_chunk_prepare_kernel<DK><<<dim3(a.chunks, H, B), 256, s1, st>>>(a, (const bf16*)x, ldx, log_decay, inv_ts, rot, (bf16*)aa, (bf16*)qkg, ends); \
    break;
    GO(16) GO(32) GO(48) GO(64) GO(80) GO(96) GO(112) GO(128)
#undef GO
  }
  if (int rc = launch_carry<false>(a, (const bf16*)x, ldx, 0, 2L * H * dk, (const bf16*)aa, (const bf16*)qkg, nullptr, ends, (bf16*)o, B, st)) return rc;
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_channel_delta_chunks(const void* mixed, long ldx, const void* beta, long ldb, const float* da, const void* A_log, const void* dt_bias, int hk,
                                       int hv, int dk, int dv, int S, int t_lo, int t_hi, float* rec, const int64_t* slots, const int64_t* lengths,
                                       const int64_t* new_lens, void* tp, void* qkg, float* betas, float* ends, void* o, int B, cudaStream_t st) {
  if (!mt_chunk_supported(dk, dv) || ldx % 8) return -1;
  const ChunkArgs a{hv, hv / hk, dk, dv, S, t_lo, t_hi, (t_hi - t_lo + CH - 1) / CH, slots, lengths, new_lens, rec};
  switch (dk) {
#define GO(DK) case DK: return launch_channel<DK>(a, (const bf16*)mixed, ldx, 2L * hk * dk, (const bf16*)beta, ldb, da, (const bf16*)A_log, \
                                                  (const bf16*)dt_bias, (bf16*)tp, (bf16*)qkg, betas, ends, (bf16*)o, B, st);
    GO(16) GO(32) GO(48) GO(64) GO(80) GO(96) GO(112) GO(128)
#undef GO
    default: return -1;
  }
}
