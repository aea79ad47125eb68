// The border between two sublayers of a model with an fp32 residual stream and sandwich norms, in one pass per row:
//   x += mult * rms(branch) * (offset + w_post);    y = rms(x) * (offset + w_next)
// The branch comes in the compute type (a GEMM output), x stays fp32, y is rounded once for the next GEMM. Without a branch it is the
// plain norm of the stream. residual_join is the same for pre-norm layers: one or two branches, each with a factor, a bias and a norm of its own
// or without, one factor per lane on their sum, and the stream handed on normalised or as it is. residual_gate is the same for sandwich-normed layers
// whose branch is gated lane by lane, with layer or RMS norms; the branch may be a sum of rows that an index picks. Also here: the ungated
// activations between the two products of a feed-forward, and the gate of a per-layer token embedding. Bandwidth-bound.
#include "serving_common.cuh"
#include "residual_gate.h"

namespace mt {

template <typename T, int VEC>
__global__ void residual_norm_kernel(float* __restrict__ x, const T* __restrict__ branch, const T* __restrict__ w_post, float mult,
                                     const T* __restrict__ w_next, T* __restrict__ y, int D, float eps_post, float eps_next, float offset) {
  extern __shared__ __align__(16) float row[];           // D floats
  __shared__ float red[32];
  const long r = blockIdx.x;
  float* xr = x + r * D;
  float scale = 0.f;
  if (branch) {
    const T* br = branch + r * D;
    float ss = 0.f;
    for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
      float v[VEC];
      load_vec<VEC>(br + c, v);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
      store_vec<VEC>(row + c, v);
    }
    scale = rsqrtf(block_add(ss, red) / (float)D + eps_post) * mult;
  }
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(xr + c, v);
    if (branch) {
      float b[VEC], w[VEC];
      load_vec<VEC>(row + c, b);
      load_vec<VEC>(w_post + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] += b[e] * scale * (offset + w[e]);
      store_vec<VEC>(xr + c, v);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
    store_vec<VEC>(row + c, v);
  }
  if (!y) return;
  const float rstd = rsqrtf(block_add(ss, red) / (float)D + eps_next);
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    float v[VEC], w[VEC];
    load_vec<VEC>(row + c, v);
    load_vec<VEC>(w_next + c, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * rstd * (offset + w[e]);
    store_vec<VEC>(y + r * D + c, v);
  }
}

struct JoinBranch {
  const void *out, *bias, *norm;       // [rows, D]; bias [D] or null; norm weight [D] or null: not normalised
  float factor;
};

// x += lanes * (a + b);   y = rms(x) * w_next, or x. One CTA per row, a thread holds VEC neighbouring lanes ITER times.
template <typename T, int VEC, int ITER>
__global__ void __launch_bounds__(256)
residual_join_kernel(float* __restrict__ x, const JoinBranch a, const JoinBranch b, const T* __restrict__ lanes, const T* __restrict__ w_next,
                     T* __restrict__ y, int D, float eps) {
  __shared__ float red[2][8];
  const long r = blockIdx.x;
  const int nt = blockDim.x;
  float* xr = x + r * D;
  float add[ITER][VEC], xv[ITER][VEC], t[ITER][VEC];
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * nt + threadIdx.x) * VEC;
    if (c < D) load_vec<VEC>(xr + c, xv[i]);
  }
  auto load = [&](const JoinBranch& j, float (&v)[ITER][VEC]) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * nt + threadIdx.x) * VEC;
      if (c < D) {
        load_vec<VEC>(static_cast<const T*>(j.out) + r * D + c, v[i]);
        if (j.bias) {
          float w[VEC];
          load_vec<VEC>(static_cast<const T*>(j.bias) + c, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i][e] += w[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += v[i][e] * v[i][e];
      }
    }
    return ss;
  };
  auto scale = [&](const JoinBranch& j, float (&v)[ITER][VEC], float rstd) {
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * nt + threadIdx.x) * VEC;
      if (c < D) {
        float w[VEC];
        if (j.norm) load_vec<VEC>(static_cast<const T*>(j.norm) + c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i][e] *= j.norm ? j.factor * rstd * w[e] : j.factor;
      }
    }
  };
  float sa = load(a, add), sb = 0.f;
  if (b.out) sb = load(b, t);
  if (a.norm || b.norm) {
    sa = warp_add(sa);
    sb = warp_add(sb);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sa; red[1][threadIdx.x >> 5] = sb; }
    __syncthreads();
    sa = sb = 0.f;
    for (int i = 0; i < (nt + 31) / 32; ++i) { sa += red[0][i]; sb += red[1][i]; }
  }
  scale(a, add, rsqrtf(sa / (float)D + eps));
  if (b.out) {
    scale(b, t, rsqrtf(sb / (float)D + eps));
#pragma unroll
    for (int i = 0; i < ITER; ++i)
#pragma unroll
      for (int e = 0; e < VEC; ++e) add[i][e] += t[i][e];
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * nt + threadIdx.x) * VEC;
    if (c < D) {
      float w[VEC];
      if (lanes) load_vec<VEC>(lanes + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        xv[i][e] += lanes ? w[e] * add[i][e] : add[i][e];
        ss += xv[i][e] * xv[i][e];
      }
      store_vec<VEC>(xr + c, xv[i]);
    }
  }
  if (!y) return;
  float rstd = 1.f;
  if (w_next) {
    __syncthreads();                                     // the sums of the branches have been read
    rstd = rsqrtf(block_add(ss, red[0]) / (float)D + eps);
  }
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * nt + threadIdx.x) * VEC;
    if (c < D) {
      float w[VEC];
      if (w_next) load_vec<VEC>(w_next + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv[i][e] *= w_next ? rstd * w[e] : 1.f;
      store_vec<VEC>(y + r * D + c, xv[i]);
    }
  }
}

// Mean and sum of squared deviations of the row that a block holds in registers, `n` of its elements in this warp: the deviations are taken
// from the warp's own mean, and the warps are joined by the shift of their means, so that one barrier is enough. `sh` holds one entry per warp.
template <int VEC, int ITER>
__device__ __forceinline__ float2 row_moments(const float (&v)[ITER][VEC], int D, bool centred, float3* sh) {
  const int nt = blockDim.x, w0 = threadIdx.x & ~31;
  int n = 0;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    n += min(max(D - (i * nt + w0) * VEC, 0), 32 * VEC);
    if ((i * nt + (int)threadIdx.x) * VEC < D) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) s += v[i][e];
    }
  }
  const float mean = centred && n > 0 ? warp_add(s) / (float)n : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ITER; ++i)
    if ((i * nt + (int)threadIdx.x) * VEC < D) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += (v[i][e] - mean) * (v[i][e] - mean);
    }
  ss = warp_add(ss);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = make_float3(mean, ss, (float)n);
  __syncthreads();
  const int warps = (nt + 31) / 32;
  float all = 0.f;
  for (int i = 0; i < warps; ++i) all += sh[i].x * sh[i].z;
  all /= (float)D;
  float m2 = 0.f;
  for (int i = 0; i < warps; ++i) m2 += sh[i].y + sh[i].z * (sh[i].x - all) * (sh[i].x - all);
  return make_float2(all, m2);
}

// x += norm(b * sigmoid(g + bias)) * w_post;   y = norm(x) * w_next, or x, where b is the sum of `per_token` rows (dest: their numbers) and
// `extra`, and norm subtracts the mean (centred) or not. Without a gate the factor is one; without rows x is only read; `fresh`: x is written
// without being read. One CTA per row, a thread holds VEC neighbouring lanes ITER times.
template <typename T, int VEC, int ITER>
__global__ void __launch_bounds__(256)
residual_gate_kernel(const ResidualGate a, int D) {
  __shared__ float3 red[2][8];
  const long r = blockIdx.x;
  const int nt = blockDim.x;
  float* xr = a.x + r * D;
  float xv[ITER][VEC];
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * nt + threadIdx.x) * VEC;
    if (c < D && !a.fresh) load_vec<VEC>(xr + c, xv[i]);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv[i][e] = 0.f;
    }
  }
  if (a.rows) {
    float b[ITER][VEC];
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * nt + threadIdx.x) * VEC;
      if (c >= D) continue;
      float t[VEC];
      if (a.extra) load_vec<VEC>(static_cast<const T*>(a.extra) + r * D + c, b[i]);
      else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) b[i][e] = 0.f;
      }
      for (int j = 0; j < a.per_token; ++j) {
        const long at = a.dest ? min(max((long)a.dest[r * a.per_token + j], 0l), a.n_rows - 1) : r * a.per_token + j;
        load_vec<VEC>(static_cast<const T*>(a.rows) + at * D + c, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) b[i][e] += t[e];
      }
      if (a.gate) {
        float g[VEC];
        load_vec<VEC>(static_cast<const T*>(a.gate) + r * a.ldg + c, g);
        load_vec<VEC>(static_cast<const T*>(a.bias) + c, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) b[i][e] *= sigmoid_t<T>(g[e] + t[e]);
      }
    }
    const float2 m = row_moments<VEC, ITER>(b, D, a.centred, red[0]);
    const float rstd = rsqrtf(m.y / (float)D + a.eps);
#pragma unroll
    for (int i = 0; i < ITER; ++i) {
      const int c = (i * nt + threadIdx.x) * VEC;
      if (c >= D) continue;
      float w[VEC];
      load_vec<VEC>(static_cast<const T*>(a.w_post) + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv[i][e] += (b[i][e] - m.x) * rstd * w[e];
      store_vec<VEC>(xr + c, xv[i]);
    }
  }
  if (!a.y) return;
  float2 m = make_float2(0.f, 0.f);
  float rstd = 1.f;
  if (a.w_next) {
    m = row_moments<VEC, ITER>(xv, D, a.centred, red[1]);
    rstd = rsqrtf(m.y / (float)D + a.eps);
  }
#pragma unroll
  for (int i = 0; i < ITER; ++i) {
    const int c = (i * nt + threadIdx.x) * VEC;
    if (c >= D) continue;
    if (a.w_next) {
      float w[VEC];
      load_vec<VEC>(static_cast<const T*>(a.w_next) + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) xv[i][e] = (xv[i][e] - m.x) * rstd * w[e];
    }
    store_vec<VEC>(static_cast<T*>(a.y) + r * a.ldy + c, xv[i]);
  }
}

__device__ __forceinline__ float act_value(float x, int code) {
  switch (code) {
    case 0: return silu_f(x);
    case 1: return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    case 2: return fmaxf(x, 0.f);
    case 5: return x > 0.f ? x * x : 0.f;
    default: return 0.5f * x * (1.f + erff(x * 0.7071067811865476f));
  }
}

// Gelu for a bf16 result: Abramowitz and Stegun 7.1.26, erfc(z) = t (a1 + t (a2 + t (a3 + t (a4 + t a5)))) e^(-z^2) with t = 1 / (1 + p z), absolute
// error below 1.5e-7; 1 + erf is formed without cancellation for negative arguments.
__device__ __forceinline__ float gelu_erf_bf16(float x) {
  const float z = fabsf(x) * 0.7071067811865476f, t = __fdividef(1.f, 1.f + 0.3275911f * z);
  const float c = t * (0.254829592f + t * (-0.284496736f + t * (1.421413741f + t * (-1.453152027f + t * 1.061405429f)))) * __expf(-z * z);
  return 0.5f * x * (x < 0.f ? c : 2.f - c);
}
template <typename T> __device__ __forceinline__ float act_typed(float x, int code) { return act_value(x, code); }
template <> __device__ __forceinline__ float act_typed<__nv_bfloat16>(float x, int code) {
  return code == 4 ? gelu_erf_bf16(x) : (code == 0 ? silu_t<__nv_bfloat16>(x) : act_value(x, code));
}

template <typename T>
__global__ void act_kernel(const T* __restrict__ x, T* __restrict__ y, long n, int code) {
  const long nv = n / 8;
  for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < nv; i += (long)gridDim.x * blockDim.x) {
    float v[8];
    load_vec<8>(x + i * 8, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = act_typed<T>(v[e], code);
    store_vec<8>(y + i * 8, v);
  }
  if (blockIdx.x == 0 && threadIdx.x < n - nv * 8) y[nv * 8 + threadIdx.x] = from_f<T>(act_typed<T>(to_f(x[nv * 8 + threadIdx.x]), code));
}

// The same over rows that lie in a wider matrix, x [rows, ldx] -> y [rows, F]. Code 6 is xIELU with its two numbers in `par`:
// a z^2 + z / 2 for positive z, b (e^z - 1 - z) + z / 2 for the others, a = softplus(par 0), b = 1/2 + softplus(par 1).
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
act_rows_kernel(const T* __restrict__ x, long ldx, T* __restrict__ y, long rows, int F, int code, const T* __restrict__ par) {
  const long per = F / VEC;
  const float a = code == 6 ? softplus_f(to_f(par[0])) : 0.f, b = code == 6 ? 0.5f + softplus_f(to_f(par[1])) : 0.f;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < rows * per; i += gridDim.x * 256l) {
    const long r = i / per;
    const int c = (int)(i % per) * VEC;
    float v[VEC];
    load_vec<VEC>(x + r * ldx + c, v);
    if (code == 6) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float z = v[e], neg = fminf(z, 0.f);
        float t;                                         // e^z - 1 - z of a negative z; for a bf16 result two terms are enough near zero
        if constexpr (sizeof(T) == 2) t = neg > -0.015625f ? neg * neg * (0.5f + neg * (1.f / 6.f)) : __expf(neg) - 1.f - neg;
        else t = expm1f(neg) - neg;
        v[e] = (z > 0.f ? a * z * z : b * t) + 0.5f * z;
      }
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = act_typed<T>(v[e], code);
    }
    store_vec<VEC>(y + r * F + c, v);
  }
}

// out[n, c] = gelu_tanh(g[n, c]) * table[token[n], c]
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
token_gate_kernel(const T* __restrict__ g, const T* __restrict__ table, const int64_t* __restrict__ tokens, long N, int dim, long vocab, T* __restrict__ out) {
  const long per = dim / VEC;
  for (long i = blockIdx.x * 256l + threadIdx.x; i < N * per; i += gridDim.x * 256l) {
    const long n = i / per;
    const int c = (int)(i % per) * VEC;
    const long tok = min(max((long)tokens[n], 0l), vocab - 1);
    float v[VEC], e[VEC];
    load_vec<VEC>(g + n * dim + c, v);
    load_vec<VEC>(table + tok * dim + c, e);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = act_value(v[k], 1) * e[k];
    store_vec<VEC>(out + n * dim + c, v);
  }
}

template <typename T>
int residual_join_t(float* x, const JoinBranch& a, const JoinBranch& b, const void* lanes, const void* w_next, void* y, long rows, int D, float eps,
                    cudaStream_t st) {
  auto go = [&](auto kernel, int vec, int iter) {
    int threads = (((D + vec * iter - 1) / (vec * iter)) + 31) / 32 * 32;
    if (threads > 256) return -1;
    kernel<<<(unsigned)rows, threads, 0, st>>>(x, a, b, (const T*)lanes, (const T*)w_next, (T*)y, D, eps);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  uintptr_t bits = 0;
  for (const void* p : {a.out, a.bias, a.norm, b.out, b.bias, b.norm, lanes, w_next, (const void*)x, (const void*)y}) bits |= reinterpret_cast<uintptr_t>(p);
  if (D % 8 == 0 && bits % 16 == 0) {
    if (D <= 2048) return go(residual_join_kernel<T, 8, 1>, 8, 1);
    if (D <= 4096) return go(residual_join_kernel<T, 8, 2>, 8, 2);
  }
  if (D % 4 == 0 && bits % 16 == 0) {
    if (D <= 1024) return go(residual_join_kernel<T, 4, 1>, 4, 1);
    if (D <= 2048) return go(residual_join_kernel<T, 4, 2>, 4, 2);
    if (D <= 4096) return go(residual_join_kernel<T, 4, 4>, 4, 4);
    return go(residual_join_kernel<T, 4, 16>, 4, 16);
  }
  return D <= 1024 ? go(residual_join_kernel<T, 1, 4>, 1, 4) : go(residual_join_kernel<T, 1, 32>, 1, 32);
}

template <typename T>
int residual_gate_t(const ResidualGate& a, long rows, int D, cudaStream_t st) {
  auto go = [&](auto kernel, int vec, int iter) {
    const int threads = (((D + vec * iter - 1) / (vec * iter)) + 31) / 32 * 32;
    if (threads > 256) return -1;
    kernel<<<(unsigned)rows, threads, 0, st>>>(a, D);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  uintptr_t bits = 0;
  for (const void* p : {a.rows, a.extra, a.gate, a.bias, a.w_post, a.w_next, (const void*)a.x, (const void*)a.y}) bits |= reinterpret_cast<uintptr_t>(p);
  const bool al = bits % 16 == 0;
  if (D % 8 == 0 && al && (!a.gate || a.ldg % 8 == 0) && a.ldy % 8 == 0) {
    if (D <= 2048) return go(residual_gate_kernel<T, 8, 1>, 8, 1);
    if (D <= 4096) return go(residual_gate_kernel<T, 8, 2>, 8, 2);
    if (D <= 8192) return go(residual_gate_kernel<T, 8, 4>, 8, 4);
  }
  return D <= 1024 ? go(residual_gate_kernel<T, 1, 4>, 1, 4) : go(residual_gate_kernel<T, 1, 32>, 1, 32);
}

template <typename T>
int residual_norm_t(float* x, const void* b, const void* wp, float mult, const void* wn, void* y, long rows, int D, float e1, float e2, float off,
                    cudaStream_t st) {
  const size_t smem = (size_t)D * 4;
  if (smem > 200 * 1024) return -1;
  const int threads = D >= 2048 ? 256 : (D >= 512 ? 128 : 64);
  auto k4 = residual_norm_kernel<T, 4>;
  auto k1 = residual_norm_kernel<T, 1>;
  auto k = D % 4 == 0 ? k4 : k1;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
  k<<<(unsigned)rows, threads, smem, st>>>(x, (const T*)b, (const T*)wp, mult, (const T*)wn, (T*)y, D, e1, e2, off);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace mt

using namespace mt;

extern "C" int mt_residual_norm(float* x, const void* branch, const void* w_post, float mult, const void* w_next, void* y, int f32, long rows, int D,
                                float eps_post, float eps_next, float offset, cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? residual_norm_t<float>(x, branch, w_post, mult, w_next, y, rows, D, eps_post, eps_next, offset, st)
             : residual_norm_t<__nv_bfloat16>(x, branch, w_post, mult, w_next, y, rows, D, eps_post, eps_next, offset, st);
}

extern "C" int mt_act_fwd(const void* x, void* y, int f32, long n, int code, int sms, cudaStream_t st) {
  if (n <= 0) return 0;
  long blocks = (n / 8 + 255) / 256;
  const int grid = (int)(blocks < 1 ? 1 : (blocks < (long)sms * 8 ? blocks : (long)sms * 8));
  if (f32) act_kernel<float><<<grid, 256, 0, st>>>((const float*)x, (float*)y, n, code);
  else act_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)y, n, code);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_residual_join(float* x, const void* a, const void* a_bias, const void* a_norm, float a_factor, const void* b, const void* b_bias,
                                const void* b_norm, float b_factor, const void* lanes, const void* w_next, void* y, int f32, long rows, int D, float eps,
                                cudaStream_t st) {
  if (rows <= 0) return 0;
  const JoinBranch ja{a, a_bias, a_norm, a_factor}, jb{b, b_bias, b_norm, b_factor};
  return f32 ? residual_join_t<float>(x, ja, jb, lanes, w_next, y, rows, D, eps, st) : residual_join_t<__nv_bfloat16>(x, ja, jb, lanes, w_next, y, rows, D, eps, st);
}

extern "C" int mt_token_gate(const void* g, const void* table, const int64_t* tokens, void* out, int f32, long N, int dim, long vocab, int sms,
                             cudaStream_t st) {
  if (N <= 0 || dim <= 0) return 0;
  const bool v8 = dim % 8 == 0 && (reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  const long blocks = (N * (dim / (v8 ? 8 : 1)) + 255) / 256;
  const unsigned grid = (unsigned)(blocks < sms * 8l ? blocks : sms * 8l);
#define GO(T, V) token_gate_kernel<T, V><<<grid, 256, 0, st>>>((const T*)g, (const T*)table, tokens, N, dim, vocab, (T*)out)
  if (f32) { if (v8) GO(float, 8); else GO(float, 1); }
  else { if (v8) GO(__nv_bfloat16, 8); else GO(__nv_bfloat16, 1); }
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_residual_gate(const ResidualGate* a, int f32, long rows, int D, cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? residual_gate_t<float>(*a, rows, D, st) : residual_gate_t<__nv_bfloat16>(*a, rows, D, st);
}

extern "C" int mt_act_rows(const void* x, long ldx, void* y, int f32, long rows, int F, int code, const void* par, int sms, cudaStream_t st) {
  if (rows <= 0 || F <= 0) return 0;
  if (code == 6 && !par) return -1;
  const bool v8 = F % 8 == 0 && ldx % 8 == 0 && (reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y)) % 16 == 0;
  const long blocks = (rows * (F / (v8 ? 8 : 1)) + 255) / 256;
  const unsigned grid = (unsigned)(blocks < sms * 16l ? blocks : sms * 16l);
#define GO(T, V) act_rows_kernel<T, V><<<grid, 256, 0, st>>>((const T*)x, ldx, (T*)y, rows, F, code, (const T*)par)
  if (f32) { if (v8) GO(float, 8); else GO(float, 1); }
  else { if (v8) GO(__nv_bfloat16, 8); else GO(__nv_bfloat16, 1); }
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
