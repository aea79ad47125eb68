// Routed experts at inference when few rows reach each expert (decoding), or when widths do not fit the padded tcgen05 path: the weights of
// every chosen expert are streamed once per 32 of its rows. The score of a choice multiplies the expert's input; it is applied to both
// up-projections in fp32, in front of the clamps:
//   up:    h[pair] = act(s (Wg x), s (Wu x)),  act(g, u) = min(g, L) sigmoid(1.702 min(g, L)) (clamp(u, -L, L) + 1)
//   down:  y[pair] = Wd h[pair]
// Ungated experts have one up-projection, whose activation the score multiplies:  h[pair] = s relu(W x)^2.
// A persistent CTA works through items of 16 * MW weight rows of one expert. Its four warps sit MW along the rows and 4 / MW along the
// contraction, operands pass through a cp.async ring of three or four stages, mma.sync m16n8k16 takes the weights in the M position (a step is bound by
// reading weights: with a handful of tokens per expert the 128-row tiles of tcgen05 would be empty). Also here: the activation of the padded path, and plain kernels for fp32
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

enum { DOWN = 0, GATED = 1, RELU2 = 2 };
__device__ __forceinline__ float relu2(float s, float v) { return v > 0.f ? s * v * v : 0.f; }

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
// per warp layout: contraction of a stage, and stages, so that at least two CTAs fit an SM
constexpr int depth(int mw) { return mw == 4 ? 64 : 128; }
constexpr int stages(int mw) { return mw == 2 ? 3 : 4; }

// One work item: BM weight rows of one expert against up to NT of its rows. Items are numbered expert by expert (experts without rows have
// none), and a CTA takes every gridDim.x-th one.
struct Item {
  int e, r0, m0;              // expert, first of its rows, first weight row
  int base;                   // number of the expert's first item
};

template <int BM>
__device__ __forceinline__ bool find(const Args& a, int E, int number, Item& it) {
  const int tiles = (a.M + BM - 1) / BM;
  while (it.e < E) {
    const int count = (a.sizes[it.e] + NT - 1) / NT * tiles;
    if (number < it.base + count) {
      it.r0 = (number - it.base) / tiles * NT;
      it.m0 = (number - it.base) % tiles * BM;
      return true;
    }
    it.base += count;
    ++it.e;
  }
  return false;
}

// The ring runs on over item borders: while an item's sums are finished the loads of the next one are in flight.
template <int MODE, int MW>
__global__ void __launch_bounds__(128)
stream_kernel(const Args a, int E) {
  constexpr int KW = 4 / MW, BM = 16 * MW, BK = depth(MW), STAGES = stages(MW), LD = BK + 8, NWT = MODE == GATED ? 2 : 1, PL = BM + 1;
  constexpr bool UP = MODE != DOWN;
  constexpr int V = BK / 8, XR = NT * V / 128;                        // 16-byte pieces of a row; pieces of x per thread
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* sw = sm;                                             // [STAGES][NWT][BM][LD]
  __nv_bfloat16* sx = sm + STAGES * NWT * BM * LD;                    // [STAGES][NT][LD]
  float* part = reinterpret_cast<float*>(sx + STAGES * NT * LD);      // [KW][NWT][NT][PL]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wm = warp % MW, wk = warp / MW;
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x);
  const int steps = (a.K + BK - 1) / BK;

  // ---- loader: item, step, and what this thread copies of it
  Item ld{0, 0, 0, 0};
  int ld_number = blockIdx.x, ld_step = 0, ld_stage = 0;
  bool ld_more = find<BM>(a, E, ld_number, ld);
  const __nv_bfloat16* xrow[XR];
  const __nv_bfloat16 *w0 = nullptr, *w1 = nullptr;
  auto enter = [&]() {
    if (!ld_more) return;
    w0 = reinterpret_cast<const __nv_bfloat16*>(a.w0) + ((long)ld.e * a.M + ld.m0) * a.K;
    if (MODE == GATED) w1 = reinterpret_cast<const __nv_bfloat16*>(a.w1) + ((long)ld.e * a.M + ld.m0) * a.K;
    const int size = a.sizes[ld.e], off = a.offs[ld.e];
#pragma unroll
    for (int j = 0; j < XR; ++j) {
      const int r = ld.r0 + (tid + j * 128) / V;
      const int p = r < size ? a.row_pair[off + r] : -1;
      xrow[j] = p < 0 ? nullptr : x + (long)(UP ? p / a.k : p) * a.K;
    }
  };
  enter();
  auto load = [&]() {
    if (ld_more) {
      const int k0 = ld_step * BK;
      for (int i = tid; i < BM * V; i += 128) {
        const int r = i / V, c = (i % V) * 8;
        const bool ok = ld.m0 + r < a.M && k0 + c < a.K;
        const long at = ok ? (long)r * a.K + k0 + c : 0;
        la_cp_async16(sw + ((ld_stage * NWT) * BM + r) * LD + c, w0 + at, ok ? 16 : 0);
        if (MODE == GATED) la_cp_async16(sw + ((ld_stage * NWT + NWT - 1) * BM + r) * LD + c, w1 + at, ok ? 16 : 0);
      }
#pragma unroll
      for (int j = 0; j < XR; ++j) {
        const int i = tid + j * 128, r = i / V, c = (i % V) * 8;
        const bool ok = xrow[j] != nullptr && k0 + c < a.K;
        la_cp_async16(sx + (ld_stage * NT + r) * LD + c, ok ? xrow[j] + k0 + c : x, ok ? 16 : 0);
      }
      if (++ld_step == steps) {
        ld_step = 0;
        ld_number += gridDim.x;
        ld_more = find<BM>(a, E, ld_number, ld);
        enter();
      }
    }
    ld_stage = ld_stage + 1 == STAGES ? 0 : ld_stage + 1;
    la_commit();
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) load();

  Item it{0, 0, 0, 0};
  int stage = 0;
  for (int number = blockIdx.x; find<BM>(a, E, number, it); number += gridDim.x) {
    float acc[NWT][4][4];
#pragma unroll
    for (int wt = 0; wt < NWT; ++wt)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[wt][j][q] = 0.f;
    for (int s = 0; s < steps; ++s) {
      la_wait<STAGES - 2>();
      __syncthreads();
      load();
      const __nv_bfloat16* xs = sx + stage * NT * LD;
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
          la_ldm4(aw, sw + ((stage * NWT + wt) * BM + wm * 16 + (lane & 15)) * LD + kc + (lane >> 4) * 8);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            la_mma(acc[wt][2 * j], aw, bx[j][0], bx[j][1]);
            la_mma(acc[wt][2 * j + 1], aw, bx[j][2], bx[j][3]);
          }
        }
      }
      stage = stage + 1 == STAGES ? 0 : stage + 1;
    }
    // the KW partial products meet in shared memory (the previous item's were read before this item's first barrier)
#pragma unroll
    for (int wt = 0; wt < NWT; ++wt)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q)
          part[((wk * NWT + wt) * NT + j * 8 + (lane & 3) * 2 + (q & 1)) * PL + wm * 16 + (lane >> 2) + (q >> 1) * 8] = acc[wt][j][q];
    __syncthreads();
    const int left = a.sizes[it.e] - it.r0, off = a.offs[it.e] + it.r0;
    for (int i = tid; i < NT * BM; i += 128) {
      const int t = i / BM, r = i % BM;
      if (t >= left || it.m0 + r >= a.M) continue;
      const int p = a.row_pair[off + t];
      float v[NWT];
#pragma unroll
      for (int wt = 0; wt < NWT; ++wt) {
        v[wt] = 0.f;
#pragma unroll
        for (int q = 0; q < KW; ++q) v[wt] += part[((q * NWT + wt) * NT + t) * PL + r];
      }
      float o = v[0];
      if constexpr (MODE == GATED) o = clamped_act(a.wts[p] * v[0], a.wts[p] * v[NWT - 1], a.limit);
      if constexpr (MODE == RELU2) o = relu2(a.wts[p], v[0]);
      reinterpret_cast<__nv_bfloat16*>(a.out)[(long)p * a.M + it.m0 + r] = __float2bfloat16_rn(o);
    }
  }
  la_wait<0>();
}

// one warp per output row, one pair at a time
template <typename T, int MODE>
__global__ void __launch_bounds__(256)
plain_kernel(const Args a) {
  constexpr bool UP = MODE != DOWN;
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= a.M) return;
  for (int p = blockIdx.y; p < a.n; p += gridDim.y) {
    const long wrow = ((long)a.idx[p] * a.M + m) * a.K;
    const T* x = reinterpret_cast<const T*>(a.x) + (long)(UP ? p / a.k : p) * a.K;
    float g = 0.f, u = 0.f;
    for (int c = lane; c < a.K; c += 32) {
      const float v = to_f(x[c]);
      g += to_f(reinterpret_cast<const T*>(a.w0)[wrow + c]) * v;
      if (MODE == GATED) u += to_f(reinterpret_cast<const T*>(a.w1)[wrow + c]) * v;
    }
    g = warp_add(g);
    if (MODE == GATED) g = clamped_act(a.wts[p] * g, a.wts[p] * warp_add(u), a.limit);
    if (MODE == RELU2) g = relu2(a.wts[p], g);
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

// the same for ungated experts: u [rows, F] -> h [rows, F]
__global__ void __launch_bounds__(256)
relu2_kernel(const __nv_bfloat16* __restrict__ u, const float* __restrict__ wts, const int* __restrict__ row_pair, const int* __restrict__ offs, int E, int F,
             __nv_bfloat16* __restrict__ h) {
  const long used = offs[E], per = F / 8;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < used * per; i += gridDim.x * 256l) {
    const long r = i / per;
    const int c = (int)(i % per) * 8, p = row_pair[r];
    const float s = p < 0 ? 0.f : wts[p];
    float v[8];
    load_vec<8>(u + r * F + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = relu2(s, v[e]);
    store_vec<8>(h + r * F + c, v);
  }
}

template <int MODE, int MW>
int stream(const Args& a, int E, int sms, cudaStream_t st) {
  constexpr int BM = 16 * MW, STAGES = stages(MW), LD = depth(MW) + 8, NWT = MODE == GATED ? 2 : 1, KW = 4 / MW;
  constexpr int smem = STAGES * (NWT * BM + NT) * LD * 2 + KW * NWT * NT * (BM + 1) * 4;
  auto k = stream_kernel<MODE, MW>;
  if (cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  const long items = ((long)(a.n < E ? a.n : E) + a.n / NT) * ((a.M + BM - 1) / BM);       // at most
  const long slots = (long)sms * (227 * 1024 / (smem + 1024));
  k<<<(unsigned)(items < slots ? items : slots), 128, smem, st>>>(a, E);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <int MODE>
int run(int f32, const Args& a, int E, int sms, cudaStream_t st) {
  if (a.n <= 0) return 0;
  if (!f32 && a.K % 8 == 0) {
    const long hit = a.n < E ? a.n : E;                     // experts that will find rows, at most
    if (hit * ((a.M + 63) / 64) >= 2l * sms) return stream<MODE, 4>(a, E, sms, st);
    if (hit * ((a.M + 31) / 32) >= 2l * sms) return stream<MODE, 2>(a, E, sms, st);
    return stream<MODE, 1>(a, E, sms, st);
  }
  const dim3 grid((a.M + 7) / 8, a.n < 65535 ? a.n : 65535);
  if (f32) plain_kernel<float, MODE><<<grid, 256, 0, st>>>(a);
  else plain_kernel<__nv_bfloat16, MODE><<<grid, 256, 0, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace expert
}  // namespace mt

using namespace mt::expert;

// w1 null: ungated experts. x [T, D], w0 / w1 [E, F, D], wts / idx [n] (pair t * k + c), sizes / offs / row_pair of mt_moe_sort -> h [n, F]
extern "C" int mt_expert_up(int f32, const void* x, const void* w0, const void* w1, const float* wts, const int* idx, const int* sizes, const int* offs,
                            const int* row_pair, int n, int k, int E, int F, int D, float limit, void* h, int sms, cudaStream_t st) {
  const Args a{x, w0, w1, wts, idx, sizes, offs, row_pair, n, k, F, D, limit, h};
  return w1 ? run<GATED>(f32, a, E, sms, st) : run<RELU2>(f32, a, E, sms, st);
}

// h [n, F], w [E, D, F] -> y [n, D]
extern "C" int mt_expert_down(int f32, const void* h, const void* w, const int* idx, const int* sizes, const int* offs, const int* row_pair, int n, int E,
                              int D, int F, void* y, int sms, cudaStream_t st) {
  return run<DOWN>(f32, Args{h, w, nullptr, nullptr, idx, sizes, offs, row_pair, n, 1, D, F, 0.f, y}, E, sms, st);
}

// gated: gu [rows, 2F] holds both up-projections; otherwise [rows, F]
extern "C" int mt_expert_act(const void* gu, int gated, const float* wts, const int* row_pair, const int* offs, int E, int F, float limit, void* h, int rows_max,
                             int sms, cudaStream_t st) {
  if (F % 8) return -1;
  const long blocks = ((long)rows_max * (F / 8) + 255) / 256;
  if (!gated) {
    relu2_kernel<<<(unsigned)(blocks < sms * 16l ? blocks : sms * 16l), 256, 0, st>>>(reinterpret_cast<const __nv_bfloat16*>(gu), wts, row_pair, offs, E, F,
                                                                                     reinterpret_cast<__nv_bfloat16*>(h));
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  act_kernel<<<(unsigned)(blocks < sms * 16l ? blocks : sms * 16l), 256, 0, st>>>(reinterpret_cast<const __nv_bfloat16*>(gu), wts, row_pair, offs, E, F, limit,
                                                                                 reinterpret_cast<__nv_bfloat16*>(h));
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
