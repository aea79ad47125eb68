// Small device helpers shared by the inference kernels of the recurrent and latent-attention layers: conversions between fp32 and the
// storage type, vector loads, warp sums and the elementary functions of the gates.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace mt {

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T> __device__ __forceinline__ T from_f(float x);
template <> __device__ __forceinline__ float from_f<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }

// N consecutive elements as fp32; the address is aligned to min(16, N * sizeof(T)) bytes
template <int N>
__device__ __forceinline__ void load_vec(const float* p, float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 t = *reinterpret_cast<const float4*>(p + i);
      f[i] = t.x; f[i + 1] = t.y; f[i + 2] = t.z; f[i + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = p[i];
  }
}
template <int N>
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&f)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 8) {
      const uint4 t = *reinterpret_cast<const uint4*>(p + i);
      const uint32_t w[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[j]));
        f[i + 2 * j] = v.x; f[i + 2 * j + 1] = v.y;
      }
    }
  } else if constexpr (N == 4) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int N>
__device__ __forceinline__ void store_vec(float* p, const float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = f[i];
  }
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}
template <int N>
__device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float (&f)[N]) {
  if constexpr (N % 8 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 8)
      *reinterpret_cast<uint4*>(p + i) = make_uint4(pack_bf16(f[i], f[i + 1]), pack_bf16(f[i + 2], f[i + 3]), pack_bf16(f[i + 4], f[i + 5]),
                                                    pack_bf16(f[i + 6], f[i + 7]));
  } else if constexpr (N == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]));
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = __float2bfloat16_rn(f[i]);
  }
}

__device__ __forceinline__ float warp_add(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the block; every thread gets it. `sh` holds one float per warp and may be reused after the next __syncthreads.
__device__ __forceinline__ float block_add(float v, float* sh) {
  v = warp_add(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  const int n = (blockDim.x + 31) >> 5;
  for (int i = 0; i < n; ++i) t += sh[i];
  return t;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// for results that are rounded to bf16 a hardware exponential and reciprocal are exact enough
template <typename T> __device__ __forceinline__ float silu_t(float x) { return silu_f(x); }
template <> __device__ __forceinline__ float silu_t<__nv_bfloat16>(float x) { return __fdividef(x, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) { return sigmoid_f(x); }
template <> __device__ __forceinline__ float sigmoid_t<__nv_bfloat16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

}  // namespace mt
