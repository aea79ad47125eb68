// The border between two sublayers of a model with an fp32 residual stream and sandwich norms, in one pass per row:
//   x += mult * rms(branch) * (offset + w_post);    y = rms(x) * (offset + w_next)
// The branch comes in the compute type (a GEMM output), x stays fp32, y is rounded once for the next GEMM. Without a branch it is the
// plain norm of the stream. Also here: the ungated activation between the two products of a feed-forward. Bandwidth-bound.
#include "serving_common.cuh"

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

__device__ __forceinline__ float act_value(float x, int code) {
  switch (code) {
    case 0: return silu_f(x);
    case 1: return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
    case 2: return fmaxf(x, 0.f);
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
