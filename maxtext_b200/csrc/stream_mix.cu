// The border between two sublayers of a model with several fp32 residual streams and static hyper-connections, in one pass per token:
//   X <- M^T X + w (sum of the branch's rows)^T,    y = scaled and shifted layer norm of r^T X
// where the rows of X [k, D] are the streams of a token.
// The branch comes in the compute type (a GEMM output, or the rows of the chosen experts of the token), the streams stay fp32, y is rounded
// once for the next GEMM. Without a branch it only reads the streams; without y it only mixes them. Bandwidth-bound.
#include "serving_common.cuh"

namespace mt {

constexpr int STREAMS_MAX = 16;

template <typename T, int K, int VEC>
__global__ void stream_mix_kernel(float* __restrict__ x, int k_, const T* __restrict__ branch, const int* __restrict__ dest, int per_token,
                                  const T* __restrict__ mix, const T* __restrict__ write, const T* __restrict__ read, const T* __restrict__ w,
                                  const T* __restrict__ b, T* __restrict__ y, int D, float eps) {
  extern __shared__ __align__(16) float row[];           // D floats: the weighted sum of the streams
  __shared__ float red[32];
  __shared__ float cm[STREAMS_MAX * STREAMS_MAX], cw[STREAMS_MAX], cr[STREAMS_MAX];
  constexpr int KM = K > 0 ? K : STREAMS_MAX;
  const int k = K > 0 ? K : k_;
  if (branch)
    for (int i = threadIdx.x; i < k * k; i += blockDim.x) cm[i] = to_f(mix[i]);
  for (int i = threadIdx.x; i < k; i += blockDim.x) {
    cw[i] = branch ? to_f(write[i]) : 0.f;
    cr[i] = read ? to_f(read[i]) : 1.f;
  }
  __syncthreads();
  const long r = blockIdx.x;
  float* xr = x + r * k * D;
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    float v[KM][VEC];
#pragma unroll
    for (int s = 0; s < KM; ++s)
      if (s < k) load_vec<VEC>(xr + (long)s * D + c, v[s]);
    float u[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = 0.f;
    if (branch) {
      float a[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[e] = 0.f;
      for (int j = 0; j < per_token; ++j) {
        const long br = dest ? dest[r * per_token + j] : r * per_token + j;
        float t[VEC];
        load_vec<VEC>(branch + br * D + c, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) a[e] += t[e];
      }
#pragma unroll
      for (int t = 0; t < KM; ++t) {
        if (t < k) {
          float n[VEC];
#pragma unroll
          for (int e = 0; e < VEC; ++e) n[e] = cw[t] * a[e];
#pragma unroll
          for (int s = 0; s < KM; ++s)
            if (s < k) {
              const float m = cm[s * k + t];
#pragma unroll
              for (int e = 0; e < VEC; ++e) n[e] += m * v[s][e];
            }
          store_vec<VEC>(xr + (long)t * D + c, n);
#pragma unroll
          for (int e = 0; e < VEC; ++e) u[e] += cr[t] * n[e];
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < KM; ++s)
        if (s < k) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) u[e] += cr[s] * v[s][e];
        }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum += u[e];
    store_vec<VEC>(row + c, u);
  }
  if (!y) return;
  const float mean = block_add(sum, red) / (float)D;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    float u[VEC];
    load_vec<VEC>(row + c, u);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += (u[e] - mean) * (u[e] - mean);
  }
  const float rstd = rsqrtf(block_add(ss, red) / (float)D + eps);
  for (int c = threadIdx.x * VEC; c < D; c += blockDim.x * VEC) {
    float u[VEC], g[VEC], h[VEC];
    load_vec<VEC>(row + c, u);
    load_vec<VEC>(w + c, g);
    load_vec<VEC>(b + c, h);
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = (u[e] - mean) * rstd * g[e] + h[e];
    store_vec<VEC>(y + r * D + c, u);
  }
}

template <typename T>
int stream_mix_t(float* x, int k, const void* branch, const int* dest, int per_token, const void* mix, const void* write, const void* read, const void* w,
                 const void* b, void* y, long rows, int D, float eps, cudaStream_t st) {
  const size_t smem = (size_t)D * 4;
  if (smem > 200 * 1024 || k < 1 || k > STREAMS_MAX) return -1;
  const int threads = D >= 2048 ? 256 : (D >= 512 ? 128 : 64);
  auto launch = [&](auto kernel) {
    if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
    kernel<<<(unsigned)rows, threads, smem, st>>>(x, k, (const T*)branch, dest, per_token, (const T*)mix, (const T*)write, (const T*)read, (const T*)w,
                                                  (const T*)b, (T*)y, D, eps);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  if (D % 4) return launch(stream_mix_kernel<T, 0, 1>);
  switch (k) {
    case 1: return launch(stream_mix_kernel<T, 1, 4>);
    case 2: return launch(stream_mix_kernel<T, 2, 4>);
    case 3: return launch(stream_mix_kernel<T, 3, 4>);
    case 4: return launch(stream_mix_kernel<T, 4, 4>);
    default: return launch(stream_mix_kernel<T, 0, 4>);
  }
}

}  // namespace mt

using namespace mt;

// x [rows, k, D]; branch rows of D elements in the compute type (dest null: rows t * per_token ..), or null; y null: no read
extern "C" int mt_stream_mix(float* x, int k, const void* branch, const int* dest, int per_token, const void* mix, const void* write, const void* read,
                             const void* w, const void* b, void* y, int f32, long rows, int D, float eps, cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? stream_mix_t<float>(x, k, branch, dest, per_token, mix, write, read, w, b, y, rows, D, eps, st)
             : stream_mix_t<__nv_bfloat16>(x, k, branch, dest, per_token, mix, write, read, w, b, y, rows, D, eps, st);
}
