// Routed experts at inference when few rows reach each expert (decoding), or when widths do not fit the padded tcgen05 path: the weights of
// every chosen expert are streamed once per 32 of its rows. The score of a choice multiplies the expert's input; it is applied to both
// up-projections in fp32, in front of the clamps:
//   up:    h[pair] = act(s (Wg x), s (Wu x)),  act(g, u) = min(g, L) sigmoid(1.702 min(g, L)) (clamp(u, -L, L) + 1)
//   down:  y[pair] = Wd h[pair]
// A CTA owns 16 * MW weight rows of one expert. Its four warps sit MW along the rows and 4 / MW along the contraction, operands pass through
// a three-stage cp.async ring, mma.sync m16n8k16 takes the weights in the M position (a step is bound by reading weights: with a handful of
// tokens per expert the 128-row tiles of tcgen05 would be empty). Also here: the activation of the padded path, and plain kernels for fp32
// and for widths that are not multiples of 8.
#include "serving_common.cuh"
#include "warp_mma.cuh"

namespace mt {
namespace expert {

__device__ __forceinline__ float clamped_act(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.f);
}

struct Args {
  const void* x;              // up: [T, K]; down: [n, K]
  const void *w0, *w1;        // [E, M, K]
  const float* wts;           // [n] scores (up)
  const int *idx, *sizes, *offs, *row_pair;
  int n, k, M, K;
  float limit;
  void* out;                  // [n, M]
};

constexpr int NT = 32;        // rows per pass
constexpr int STAGES = 3;

template <bool UP, int MW>
__global__ void __launch_bounds__(128)
stream_kernel(const Args a) {
  constexpr int KW = 4 / MW, BM = 16 * MW, BK = MW == 4 ? 64 : (MW == 2 ? 128 : 256), LD = BK + 8, NWT = UP ? 2 : 1;
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sw = sm;                                             // [STAGES][NWT][BM][LD]
  __nv_bfloat16* sx = sm + STAGES * NWT * BM * LD;                    // [STAGES][NT][LD]
  __shared__ int rows[NT], pairs[NT];
  __shared__ float score[NT];
  const int e = blockIdx.y, m0 = blockIdx.x * BM;
  const int size = a.sizes[e], off = a.offs[e];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wm = warp % MW, wk = warp / MW;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x);
  const __nv_bfloat16* w[2] = {reinterpret_cast<const __nv_bfloat16*>(a.w0) + (long)e * a.M * a.K,
                               UP ? reinterpret_cast<const __nv_bfloat16*>(a.w1) + (long)e * a.M * a.K : nullptr};
  const int steps = (a.K + BK - 1) / BK;
  for (int r0 = 0; r0 < size; r0 += NT) {
    __syncthreads();
    if (tid < NT) {
      const int p = r0 + tid < size ? a.row_pair[off + r0 + tid] : -1;
      pairs[tid] = p;
      rows[tid] = p < 0 ? -1 : (UP ? p / a.k : p);
      if (UP) score[tid] = p < 0 ? 0.f : a.wts[p];
    }
    __syncthreads();
    auto load = [&](int step) {
      const int st = step % STAGES, k0 = step * BK;
      constexpr int V = BK / 8;
#pragma unroll
      for (int wt = 0; wt < NWT; ++wt)
        for (int i = tid; i < BM * V; i += 128) {
          const int r = i / V, c = (i % V) * 8;
          const bool ok = m0 + r < a.M && k0 + c < a.K;
          la_cp_async16(sw + ((st * NWT + wt) * BM + r) * LD + c, ok ? w[wt] + (long)(m0 + r) * a.K + k0 + c : w[wt], ok ? 16 : 0);
        }
      for (int i = tid; i < NT * V; i += 128) {
        const int r = i / V, c = (i % V) * 8;
        const bool ok = rows[r] >= 0 && k0 + c < a.K;
        la_cp_async16(sx + (st * NT + r) * LD + c, ok ? x + (long)rows[r] * a.K + k0 + c : x, ok ? 16 : 0);
      }
    };
    float acc[NWT][4][4];
#pragma unroll
    for (int wt = 0; wt < NWT; ++wt)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[wt][j][q] = 0.f;
    for (int s = 0; s < STAGES - 1; ++s) {
      if (s < steps) load(s);
      la_commit();
    }
    for (int s = 0; s < steps; ++s) {
      la_wait<STAGES - 2>();
      __syncthreads();
      if (s + STAGES - 1 < steps) load(s + STAGES - 1);
      la_commit();
      const int st = s % STAGES;
      const __nv_bfloat16* xs = sx + st * NT * LD;
#pragma unroll
      for (int kk = 0; kk < BK / 16 / KW; ++kk) {
        const int kc = (kk * KW + wk) * 16;
        unsigned bx[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
          la_ldm4(bx[j], xs + (j * 16 + (lane & 7) + ((lane >> 4) << 3)) * LD + kc + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int wt = 0; wt < NWT; ++wt) {
          unsigned aw[4];
          la_ldm4(aw, sw + ((st * NWT + wt) * BM + wm * 16 + (lane & 15)) * LD + kc + (lane >> 4) * 8);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            la_mma(acc[wt][2 * j], aw, bx[j][0], bx[j][1]);
            la_mma(acc[wt][2 * j + 1], aw, bx[j][2], bx[j][3]);
          }
        }
      }
    }
    la_wait<0>();
    __syncthreads();
    // partial products of the KW warps through shared memory: part [KW][NWT][NT][BM + 1]
    float* part = reinterpret_cast<float*>(sm);
    constexpr int PL = BM + 1;
#pragma unroll
    for (int wt = 0; wt < NWT; ++wt)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q)
          part[((wk * NWT + wt) * NT + j * 8 + (lane & 3) * 2 + (q & 1)) * PL + wm * 16 + (lane >> 2) + (q >> 1) * 8] = acc[wt][j][q];
    __syncthreads();
    for (int i = tid; i < NT * BM; i += 128) {
      const int t = i / BM, r = i % BM;
      if (pairs[t] < 0 || m0 + r >= a.M) continue;
      float v[NWT];
#pragma unroll
      for (int wt = 0; wt < NWT; ++wt) {
        v[wt] = 0.f;
#pragma unroll
        for (int q = 0; q < KW; ++q) v[wt] += part[((q * NWT + wt) * NT + t) * PL + r];
      }
      float o = v[0];
      if constexpr (UP) o = clamped_act(score[t] * v[0], score[t] * v[NWT - 1], a.limit);
      reinterpret_cast<__nv_bfloat16*>(a.out)[(long)pairs[t] * a.M + m0 + r] = __float2bfloat16_rn(o);
    }
  }
}

// one warp per output row, one pair at a time
template <typename T, bool UP>
__global__ void __launch_bounds__(256)
plain_kernel(const Args a) {
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= a.M) return;
  for (int p = blockIdx.y; p < a.n; p += gridDim.y) {
    const long wrow = ((long)a.idx[p] * a.M + m) * a.K;
    const T* x = reinterpret_cast<const T*>(a.x) + (long)(UP ? p / a.k : p) * a.K;
    float g = 0.f, u = 0.f;
    for (int c = lane; c < a.K; c += 32) {
      const float v = to_f(x[c]);
      g += to_f(reinterpret_cast<const T*>(a.w0)[wrow + c]) * v;
      if (UP) u += to_f(reinterpret_cast<const T*>(a.w1)[wrow + c]) * v;
    }
    g = warp_add(g);
    if (UP) g = clamped_act(a.wts[p] * g, a.wts[p] * warp_add(u), a.limit);
    if (lane == 0) reinterpret_cast<T*>(a.out)[(long)p * a.M + m] = from_f<T>(g);
  }
}

// gu [rows, 2F] of the padded layout -> h [rows, F]; padding rows become zero
__global__ void __launch_bounds__(256)
act_kernel(const __nv_bfloat16* __restrict__ gu, const float* __restrict__ wts, const int* __restrict__ row_pair, const int* __restrict__ offs, int E, int F,
           float limit, __nv_bfloat16* __restrict__ h) {
  const long used = offs[E], per = F / 8;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < used * per; i += gridDim.x * 256l) {
    const long r = i / per;
    const int c = (int)(i % per) * 8;
    const int p = row_pair[r];
    const float s = p < 0 ? 0.f : wts[p];
    float g[8], u[8];
    load_vec<8>(gu + r * 2 * F + c, g);
    load_vec<8>(gu + r * 2 * F + F + c, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float gg = fminf(s * g[e], limit), uu = fminf(fmaxf(s * u[e], -limit), limit);
      g[e] = __fdividef(gg, 1.f + __expf(-1.702f * gg)) * (uu + 1.f);
    }
    store_vec<8>(h + r * F + c, g);
  }
}

template <bool UP, int MW>
int stream(const Args& a, int E, cudaStream_t st) {
  constexpr int BM = 16 * MW, BK = MW == 4 ? 64 : (MW == 2 ? 128 : 256), LD = BK + 8, NWT = UP ? 2 : 1, KW = 4 / MW;
  constexpr int ring = STAGES * (NWT * BM + NT) * LD * 2, part = KW * NWT * NT * (BM + 1) * 4;
  constexpr int smem = ring > part ? ring : part;
  auto k = stream_kernel<UP, MW>;
  if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  k<<<dim3((a.M + BM - 1) / BM, E), 128, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <bool UP>
int run(int f32, const Args& a, int E, int sms, cudaStream_t st) {
  if (a.n <= 0) return 0;
  if (!f32 && a.K % 8 == 0) {
    // CTAs that will find rows: at most one expert per pair
    const long hit = a.n < E ? a.n : E;
    if (hit * ((a.M + 63) / 64) >= 2l * sms) return stream<UP, 4>(a, E, st);
    if (hit * ((a.M + 31) / 32) >= 2l * sms) return stream<UP, 2>(a, E, st);
    return stream<UP, 1>(a, E, st);
  }
  const dim3 grid((a.M + 7) / 8, a.n < 65535 ? a.n : 65535);
  if (f32) plain_kernel<float, UP><<<grid, 256, 0, st>>>(a);
  else plain_kernel<__nv_bfloat16, UP><<<grid, 256, 0, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace expert
}  // namespace mt

using namespace mt::expert;

// x [T, D], w0 / w1 [E, F, D], wts / idx [n] (pair t * k + c), sizes / offs / row_pair of mt_moe_sort -> h [n, F]
extern "C" int mt_expert_up(int f32, const void* x, const void* w0, const void* w1, const float* wts, const int* idx, const int* sizes, const int* offs,
                            const int* row_pair, int n, int k, int E, int F, int D, float limit, void* h, int sms, cudaStream_t st) {
  return run<true>(f32, Args{x, w0, w1, wts, idx, sizes, offs, row_pair, n, k, F, D, limit, h}, E, sms, st);
}

// h [n, F], w [E, D, F] -> y [n, D]
extern "C" int mt_expert_down(int f32, const void* h, const void* w, const int* idx, const int* sizes, const int* offs, const int* row_pair, int n, int E,
                              int D, int F, void* y, int sms, cudaStream_t st) {
  return run<false>(f32, Args{h, w, nullptr, nullptr, idx, sizes, offs, row_pair, n, 1, D, F, 0.f, y}, E, sms, st);
}

extern "C" int mt_expert_act(const void* gu, const float* wts, const int* row_pair, const int* offs, int E, int F, float limit, void* h, int rows_max, int sms,
                             cudaStream_t st) {
  if (F % 8) return -1;
  const long blocks = ((long)rows_max * (F / 8) + 255) / 256;
  act_kernel<<<(unsigned)(blocks < sms * 16l ? blocks : sms * 16l), 256, 0, st>>>(reinterpret_cast<const __nv_bfloat16*>(gu), wts, row_pair, offs, E, F, limit,
                                                                                 reinterpret_cast<__nv_bfloat16*>(h));
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
