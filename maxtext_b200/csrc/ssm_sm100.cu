// Selective scan (Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces") at inference:
//   x  = silu(causal depthwise convolution + bias)
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,   y_c = (sum_n S[c, n] C_n + D_c x_c) * silu(z_c)
// with dt = softplus(pre-activation + bias) and A = -exp(A_log). States, decays and step sizes are fp32.
//
// A channel's states are spread over P neighbouring lanes, NS per lane, and stay in registers over the whole prompt. Half of a CTA's warps
// run the recurrence; the other half load and prepare the next tile of tokens (softplus, dt * x, B and C as fp32) and finish the previous
// one (skip, gate, store), so the chain of steps never waits for memory. The read-out of four steps is reduced over the lanes in one
// transposed exchange. One token per sequence runs a streaming kernel of its own, bound by reading and writing the states.
#include "serving_common.cuh"

namespace mt {
namespace ssm {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ------------------------------------------------------------------------------------------------ convolution
// One thread: VEC channels of TT consecutive tokens. hist [slots, taps-1, C] holds the inputs before the first new token; only the threads
// of the first tile touch it, and they also write what the next call needs.
constexpr int CONV_TT = 16;

template <typename T, int TAPS, int VEC>
__global__ void __launch_bounds__(128)
conv_kernel(const T* __restrict__ x, long ldx, const T* __restrict__ w, const T* __restrict__ bias, int taps_, int C, int S, float* __restrict__ hist,
            const int64_t* __restrict__ slots, const int64_t* __restrict__ lengths, const int64_t* __restrict__ new_lens, T* __restrict__ y) {
  const int taps = TAPS > 0 ? TAPS : taps_;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= C) return;
  const int b = blockIdx.z, s0 = blockIdx.y * CONV_TT;
  const int s1 = min(S, s0 + CONV_TT);
  const bool cached = lengths[b] > 0;
  float* h = hist + slots[b] * (long)(taps - 1) * C + c;
  const T* xb = x + (long)b * S * ldx + c;
  T* yb = y + (long)b * S * C + c;
  float bv[VEC];
  load_vec<VEC>(bias + c, bv);
  // input at token s (negative: history)
  auto at = [&](int s, float (&v)[VEC]) {
    if (s >= 0) load_vec<VEC>(xb + (long)s * ldx, v);
    else if (cached) load_vec<VEC>(h + (long)(taps - 1 + s) * C, v);
    else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = 0.f;
    }
  };
  if constexpr (TAPS > 0) {
    float wv[TAPS][VEC], win[TAPS][VEC];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_vec<VEC>(w + (long)j * C + c, wv[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) at(s0 - (TAPS - 1) + j, win[j]);
    for (int s = s0; s < s1; ++s) {
      at(s, win[TAPS - 1]);
      float o[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        float a = bv[e];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a += wv[j][e] * win[j][e];
        o[e] = silu_t<T>(a);
      }
      store_vec<VEC>(yb + (long)s * C, o);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) win[j][e] = win[j + 1][e];
    }
  } else {
    for (int s = s0; s < s1; ++s) {
      float a[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[e] = bv[e];
      for (int j = 0; j < taps; ++j) {
        float v[VEC], t[VEC];
        at(s - (taps - 1) + j, v);
        load_vec<VEC>(w + (long)j * C + c, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) a[e] += t[e] * v[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[e] = silu_t<T>(a[e]);
      store_vec<VEC>(yb + (long)s * C, a);
    }
  }
  if (s0 == 0) {
    const int n = new_lens ? (int)new_lens[b] : S;
    if (n < 1) return;
    for (int j = 0; j < taps - 1; ++j) {                    // row n + j of [history | new tokens]; reads stay ahead of the writes
      float v[VEC];
      at(n + j - (taps - 1), v);
      store_vec<VEC>(h + (long)j * C, v);
    }
  }
}

// ------------------------------------------------------------------------------------------------ prompts
template <typename T> struct Decay {                        // S <- decay * S + add
  static __device__ __forceinline__ float arg(float a_log) { return -expf(a_log) * LOG2E; }
  static __device__ __forceinline__ float step(float S, float dt, float a, float add) { return fmaf(exp2_fast(dt * a), S, add); }
};
template <> struct Decay<float> {                           // through expm1, so that the rounding of slow decays does not add up
  static __device__ __forceinline__ float arg(float a_log) { return -expf(a_log); }
  static __device__ __forceinline__ float step(float S, float dt, float a, float add) { return fmaf(expm1f(dt * a), S, add) + S; }
};

// x [B*S, C] (contiguous), z [B*S, ldz] (already offset), q [B*S, ldq] with B at column off and C at off + N, dt [B*S, C] fp32 pre-activations
struct ScanArgs {
  const void* x; const void* z; long ldz; const void* q; long ldq; int off;
  const float* dt; const void* dt_bias; const void* A_log; const void* D;
  int C, N, S;
  float* rec; const int64_t* slots; const int64_t* lengths; const int64_t* new_lens;
  void* y;
};

constexpr int SCAN_THREADS = 128;                           // of each role

template <typename T, int P, int NS>
__global__ void __launch_bounds__(2 * SCAN_THREADS)
scan_kernel(const ScanArgs a) {
  constexpr int CH = SCAN_THREADS / P;                      // channels of the CTA
  constexpr int NP = P * NS;                                // states, padded
  constexpr int TT = NP <= 32 ? 64 : 32;                    // tokens of a tile
  extern __shared__ __align__(16) float smem[];
  float* sBC = smem;                                        // [2][TT][2][NP]
  float2* sdt = reinterpret_cast<float2*>(sBC + 2 * TT * 2 * NP);      // [2][TT][CH]: (dt, dt * x)
  float* sy = reinterpret_cast<float*>(sdt + 2 * TT * CH);             // [2][TT][CH]
  const int b = blockIdx.y, c0 = blockIdx.x * CH;
  const bool consumer = threadIdx.x < SCAN_THREADS;
  const int tid = consumer ? threadIdx.x : threadIdx.x - SCAN_THREADS;
  const int n_real = a.new_lens ? (int)a.new_lens[b] : a.S;
  const int tiles = (min(a.S, n_real) + TT - 1) / TT;
  const T* xb = reinterpret_cast<const T*>(a.x) + (long)b * a.S * a.C;
  const T* zb = reinterpret_cast<const T*>(a.z) + (long)b * a.S * a.ldz;
  const T* qb = reinterpret_cast<const T*>(a.q) + (long)b * a.S * a.ldq + a.off;
  const float* db = a.dt + (long)b * a.S * a.C;
  T* yb = reinterpret_cast<T*>(a.y) + (long)b * a.S * a.C;

  auto prepare = [&](int tile) {
    const int t0 = tile * TT;
    float* bc = sBC + (tile & 1) * TT * 2 * NP;
    float2* dd = sdt + (tile & 1) * TT * CH;
    for (int i = tid; i < TT * CH; i += SCAN_THREADS) {
      const int t = t0 + i / CH, c = c0 + i % CH;
      float2 v = make_float2(0.f, 0.f);                     // padding neither decays nor writes
      if (t < n_real && t < a.S && c < a.C) {
        v.x = softplus_f(db[(long)t * a.C + c] + to_f(reinterpret_cast<const T*>(a.dt_bias)[c]));
        v.y = v.x * to_f(xb[(long)t * a.C + c]);
      }
      dd[i] = v;
    }
    for (int i = tid; i < TT * 2 * NP; i += SCAN_THREADS) {
      const int t = t0 + i / (2 * NP), j = i % (2 * NP), which = j / NP, n = j % NP;
      bc[i] = (t < n_real && t < a.S && n < a.N) ? to_f(qb[(long)t * a.ldq + which * a.N + n]) : 0.f;
    }
  };
  auto finish = [&](int tile) {
    const int t0 = tile * TT;
    const float* yy = sy + (tile & 1) * TT * CH;
    for (int i = tid; i < TT * CH; i += SCAN_THREADS) {
      const int t = t0 + i / CH, c = c0 + i % CH;
      if (t < n_real && t < a.S && c < a.C) {
        const float x = to_f(xb[(long)t * a.C + c]), z = to_f(zb[(long)t * a.ldz + c]);
        yb[(long)t * a.C + c] = from_f<T>((yy[i] + to_f(reinterpret_cast<const T*>(a.D)[c]) * x) * silu_t<T>(z));
      }
    }
  };

  const int lc = tid / P, ln = tid % P, c = c0 + lc;
  float S[NS], A[NS];
  float* rec = a.rec + (a.slots[b] * (long)a.C + c) * a.N + ln * NS;
  if (consumer) {
    const bool cached = a.lengths[b] > 0;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const bool ok = c < a.C && ln * NS + i < a.N;
      S[i] = (ok && cached) ? rec[i] : 0.f;
      A[i] = ok ? Decay<T>::arg(to_f(reinterpret_cast<const T*>(a.A_log)[(long)c * a.N + ln * NS + i])) : 0.f;
    }
  } else if (tiles > 0) {
    prepare(0);
  }
  __syncthreads();
  for (int tile = 0; tile < tiles; ++tile) {
    if (consumer) {
      const float* bc = sBC + (tile & 1) * TT * 2 * NP + ln * NS;
      const float2* dd = sdt + (tile & 1) * TT * CH + lc;
      float* yy = sy + (tile & 1) * TT * CH + lc;
      for (int t = 0; t < TT; t += 4) {
        float r[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float2 d = dd[(t + u) * CH];
          float Bv[NS], Cv[NS];
          load_vec<NS>(bc + (t + u) * 2 * NP, Bv);
          load_vec<NS>(bc + (t + u) * 2 * NP + NP, Cv);
          float acc = 0.f;
#pragma unroll
          for (int i = 0; i < NS; ++i) {
            S[i] = Decay<T>::step(S[i], d.x, A[i], d.y * Bv[i]);
            acc = fmaf(S[i], Cv[i], acc);
          }
          r[u] = acc;
        }
        if constexpr (P == 1) {
#pragma unroll
          for (int u = 0; u < 4; ++u) yy[(t + u) * CH] = r[u];
        } else if constexpr (P == 2) {
          const bool odd = ln & 1;
          const float s0 = odd ? r[0] : r[2], s1 = odd ? r[1] : r[3];
          const float k0 = (odd ? r[2] : r[0]) + __shfl_xor_sync(0xffffffffu, s0, 1), k1 = (odd ? r[3] : r[1]) + __shfl_xor_sync(0xffffffffu, s1, 1);
          yy[(t + (odd ? 2 : 0)) * CH] = k0;
          yy[(t + (odd ? 3 : 1)) * CH] = k1;
        } else {
          // lane bit 0 picks steps {0,1} or {2,3}, lane bit 1 one of the two; the remaining bits add up
          const bool o1 = ln & 1, o2 = ln & 2;
          const float s0 = o1 ? r[0] : r[2], s1 = o1 ? r[1] : r[3];
          const float k0 = (o1 ? r[2] : r[0]) + __shfl_xor_sync(0xffffffffu, s0, 1), k1 = (o1 ? r[3] : r[1]) + __shfl_xor_sync(0xffffffffu, s1, 1);
          float v = (o2 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, o2 ? k0 : k1, 2);
#pragma unroll
          for (int o = 4; o < P; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (ln < 4) yy[(t + (o1 ? 2 : 0) + (o2 ? 1 : 0)) * CH] = v;
        }
      }
    } else {
      if (tile + 1 < tiles) prepare(tile + 1);
      if (tile > 0) finish(tile - 1);
    }
    __syncthreads();
  }
  if (consumer) {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (c < a.C && ln * NS + i < a.N) rec[i] = S[i];
  } else {
    if (tiles > 0) finish(tiles - 1);
    // right padding: nothing reads it as a value, but later products multiply it by zero
    for (int i = max(n_real, 0) * CH + tid; i < a.S * CH; i += SCAN_THREADS)
      if (c0 + i % CH < a.C) yb[(long)(i / CH) * a.C + c0 + i % CH] = from_f<T>(0.f);
  }
}

// ------------------------------------------------------------------------------------------------ one token per sequence
template <typename T, int P, int NS>
__global__ void __launch_bounds__(256)
step_kernel(const ScanArgs a) {
  const int b = blockIdx.y;
  const int i0 = blockIdx.x * 256 + threadIdx.x, c = i0 / P, ln = i0 % P;
  const bool live = c < a.C;
  const int cc = live ? c : 0;
  float* rec = a.rec + (a.slots[b] * (long)a.C + cc) * a.N + ln * NS;
  const bool vec = NS % 4 == 0 && a.N % 4 == 0, cached = a.lengths[b] > 0;
  const int left = a.N - ln * NS;                           // states of this lane that exist
  float S[NS], Bv[NS], Cv[NS], A[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) S[i] = 0.f;
  if (live && cached) {
    if (vec) {
#pragma unroll
      for (int i = 0; i < NS; i += 4)
        if (i < left) {
          const float4 t = *reinterpret_cast<const float4*>(rec + i);
          S[i] = t.x;
          if constexpr (NS >= 4) { S[i + 1] = t.y; S[i + 2] = t.z; S[i + 3] = t.w; }
        }
    } else {
#pragma unroll
      for (int i = 0; i < NS; ++i)
        if (i < left) S[i] = rec[i];
    }
  }
  const T* q = reinterpret_cast<const T*>(a.q) + (long)b * a.ldq + a.off + ln * NS;
  const T* al = reinterpret_cast<const T*>(a.A_log) + (long)cc * a.N + ln * NS;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool ok = live && i < left;
    Bv[i] = ok ? to_f(q[i]) : 0.f;
    Cv[i] = ok ? to_f(q[a.N + i]) : 0.f;
    A[i] = ok ? Decay<T>::arg(to_f(al[i])) : 0.f;
  }
  const float x = live ? to_f(reinterpret_cast<const T*>(a.x)[(long)b * a.C + cc]) : 0.f;
  const float dt = live ? softplus_f(a.dt[(long)b * a.C + cc] + to_f(reinterpret_cast<const T*>(a.dt_bias)[cc])) : 0.f;
  const float dx = dt * x;
  float acc = 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    S[i] = Decay<T>::step(S[i], dt, A[i], dx * Bv[i]);
    acc = fmaf(S[i], Cv[i], acc);
  }
#pragma unroll
  for (int o = 1; o < P; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  if (!live) return;
  if (vec) {
#pragma unroll
    for (int i = 0; i < NS; i += 4)
      if (i < left) {
        if constexpr (NS >= 4) *reinterpret_cast<float4*>(rec + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
      }
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (i < left) rec[i] = S[i];
  }
  if (ln == 0) {
    const float z = to_f(reinterpret_cast<const T*>(a.z)[(long)b * a.ldz + c]);
    reinterpret_cast<T*>(a.y)[(long)b * a.C + c] = from_f<T>((acc + to_f(reinterpret_cast<const T*>(a.D)[c]) * x) * silu_t<T>(z));
  }
}

template <typename T, int P, int NS>
int run(const ScanArgs& a, int B, cudaStream_t st) {
  if (a.S == 1) {
    step_kernel<T, P, NS><<<dim3((unsigned)(((long)a.C * P + 255) / 256), B), 256, 0, st>>>(a);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  constexpr int CH = SCAN_THREADS / P, NP = P * NS, TT = NP <= 32 ? 64 : 32;
  constexpr int smem = (2 * TT * 2 * NP + 2 * TT * CH * 2 + 2 * TT * CH) * 4;
  auto k = scan_kernel<T, P, NS>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  k<<<dim3((a.C + CH - 1) / CH, B), 2 * SCAN_THREADS, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
int run_t(const ScanArgs& a, int B, cudaStream_t st) {
  if (a.N <= 4) return run<T, 1, 4>(a, B, st);
  if (a.N <= 8) return run<T, 2, 4>(a, B, st);
  if (a.N <= 16) return run<T, 4, 4>(a, B, st);
  if (a.N <= 32) return run<T, 8, 4>(a, B, st);
  if (a.N <= 64) return run<T, 8, 8>(a, B, st);
  if (a.N <= 128) return run<T, 16, 8>(a, B, st);
  if (a.N <= 256) return run<T, 32, 8>(a, B, st);
  return -1;
}

template <typename T>
int conv_t(const void* x, long ldx, const void* w, const void* bias, int taps, int C, int S, float* hist, const int64_t* slots, const int64_t* lengths,
           const int64_t* new_lens, void* y, int B, cudaStream_t st) {
  const int vec = (C % 8 == 0 && ldx % 8 == 0) ? 8 : 1;
  const dim3 grid((C / vec + 127) / 128, (S + CONV_TT - 1) / CONV_TT, B);
  auto launch = [&](auto k) {
    k<<<grid, 128, 0, st>>>((const T*)x, ldx, (const T*)w, (const T*)bias, taps, C, S, hist, slots, lengths, new_lens, (T*)y);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  };
  // only the first tile of tokens may see the history
  if (taps < 1 || taps - 1 > CONV_TT) return -1;
  if (vec == 8) {
    switch (taps) {
      case 2: return launch(conv_kernel<T, 2, 8>);
      case 3: return launch(conv_kernel<T, 3, 8>);
      case 4: return launch(conv_kernel<T, 4, 8>);
      default: return launch(conv_kernel<T, 0, 8>);
    }
  }
  return launch(conv_kernel<T, 0, 1>);
}

}  // namespace ssm
}  // namespace mt

using namespace mt::ssm;

extern "C" int mt_ssm_conv(int f32, const void* x, long ldx, const void* w, const void* bias, int taps, int C, int S, float* hist, const int64_t* slots,
                           const int64_t* lengths, const int64_t* new_lens, void* y, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  return f32 ? conv_t<float>(x, ldx, w, bias, taps, C, S, hist, slots, lengths, new_lens, y, B, st)
             : conv_t<__nv_bfloat16>(x, ldx, w, bias, taps, C, S, hist, slots, lengths, new_lens, y, B, st);
}

extern "C" int mt_ssm_scan(int f32, const void* x, const void* z, long ldz, const void* q, long ldq, int off, const float* dt, const void* dt_bias,
                           const void* A_log, const void* D, int C, int N, int S, float* rec, const int64_t* slots, const int64_t* lengths,
                           const int64_t* new_lens, void* y, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const ScanArgs a{x, z, ldz, q, ldq, off, dt, dt_bias, A_log, D, C, N, S, rec, slots, lengths, new_lens, y};
  return f32 ? run_t<float>(a, B, st) : run_t<__nv_bfloat16>(a, B, st);
}
