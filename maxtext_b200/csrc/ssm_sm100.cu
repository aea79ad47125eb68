// Selective scan (Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces") at inference:
//   u = silu(causal depthwise convolution + bias)
//   s <- exp(d alpha) * s + (d u) b,    y = (<s, c> + skip u) silu(z)
// per channel, with d = softplus(pre-activation + bias) and alpha = -exp(A_log). States, decays and step sizes are fp32. In the code x is the
// channel's input u, dt its step size, B and C are b and c, A is alpha and D the skip factor.
//
// A channel's states are spread over P neighbouring lanes, NS per lane, and stay in registers over the whole prompt. Four of a CTA's twelve
// warps run the recurrence; the others load and prepare the next tile of tokens (softplus, dt * x, B and C as fp32) and finish the previous
// one (skip, gate, store), with all loads of a tile in flight together, so the chain of steps never waits for memory. The read-out of four
// steps is reduced over the lanes in one transposed exchange. One token per sequence runs a streaming kernel of its own, bound by reading
// and writing the states.
#include "serving_common.cuh"
#include <type_traits>

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
  if (bias) {
    load_vec<VEC>(bias + c, bv);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) bv[e] = 0.f;
  }
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

constexpr int SCAN_THREADS = 128;                           // that run the recurrence
constexpr int FEED_THREADS = 256;                           // that load, prepare and finish

// Step size for a bf16 model: hardware exponential and logarithm, the series of log(1 + y) where the logarithm would cancel (relative error
// below 1e-5 everywhere)
template <typename T> __device__ __forceinline__ float softplus_t(float x) { return softplus_f(x); }
template <> __device__ __forceinline__ float softplus_t<__nv_bfloat16>(float x) {
  const float y = __expf(-fabsf(x));
  const float series = y * (1.f + y * (-1.f / 2 + y * (1.f / 3 + y * (-1.f / 4 + y * (1.f / 5)))));
  return fmaxf(x, 0.f) + (y < 0.0625f ? series : __logf(1.f + y));
}

// both roles of the scan kernel, from their own code
__device__ __forceinline__ void tile_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(SCAN_THREADS + FEED_THREADS) : "memory"); }

// W values as they lie in memory: converting them where they are loaded would make one load wait for the other
template <typename T, int W> struct alignas(sizeof(T) * W) Raw { T e[W]; };
template <typename T, int W> __device__ __forceinline__ Raw<T, W> read_raw(const T* p) { return *reinterpret_cast<const Raw<T, W>*>(p); }
template <typename T, int W> __device__ __forceinline__ Raw<T, W> fill_raw(float v) {
  Raw<T, W> r;
#pragma unroll
  for (int i = 0; i < W; ++i) r.e[i] = from_f<T>(v);
  return r;
}

// What a feeding thread holds of tile `in` on its way to shared memory and of tile `out` on its way to y, W channels at a time, G pieces each.
// `issue` starts the global loads, `settle` uses them. Tiles outside 0 .. tiles - 1 are skipped.
template <typename T, int CH, int NP, int TT, int W, int G>
struct Feeder {
  static constexpr int CW = CH / W, STEP = FEED_THREADS / CW, ND = (TT + STEP - 1) / STEP;
  static constexpr int BW = W == 4 ? 16 / (int)sizeof(T) : 1, NB = (TT * 2 * NP / BW + FEED_THREADS - 1) / FEED_THREADS;
  static constexpr int PIECES = ND > NB ? ND : NB;
  Raw<float, W> d[G];
  Raw<T, W> x[G], xo[G], z[G];
  Raw<T, BW> v[G];
  float bias[W], skip[W];
  const T *xb, *zb, *qb;
  const float* db;
  T* yb;
  float *sBC, *sy;
  float2* sdt;
  long ldz, ldq;
  int C, N, tiles, t_end, tid, c, ft;
  bool live;

  __device__ __forceinline__ void issue(int g, int in, int out) {
    const bool has_in = in < tiles, has_out = out >= 0 && out < tiles;
#pragma unroll
    for (int j = 0; j < G; ++j) {
      const int r = ft + (g + j) * STEP, t = in * TT + r, to = out * TT + r;
      const bool row = g + j < ND && r < TT && live;
      d[j] = fill_raw<float, W>(-INFINITY);                 // padding: softplus 0, so it neither decays nor writes
      x[j] = fill_raw<T, W>(0.f);
      if (row && has_in && t < t_end) {
        d[j] = read_raw<float, W>(db + (long)t * C + c);
        x[j] = read_raw<T, W>(xb + (long)t * C + c);
      }
      if (row && has_out && to < t_end) {
        xo[j] = read_raw<T, W>(xb + (long)to * C + c);
        z[j] = read_raw<T, W>(zb + (long)to * ldz + c);
      }
      // B and C of a token are neighbours; wide loads are only taken when N fills the padded width
      const int i = (tid + (g + j) * FEED_THREADS) * BW, tb = in * TT + i / (2 * NP), k = i % (2 * NP), n = k % NP;
      v[j] = fill_raw<T, BW>(0.f);
      if (has_in && g + j < NB && i < TT * 2 * NP && tb < t_end && n < N) v[j] = read_raw<T, BW>(qb + (long)tb * ldq + (k / NP) * N + n);
    }
  }

  __device__ __forceinline__ void settle(int g, int in, int out) {
    const bool has_in = in < tiles, has_out = out >= 0 && out < tiles;
    const int lc = (tid % CW) * W;
    const float* yy = sy + (out & 1) * TT * CH + lc;
    float* bc = sBC + (in & 1) * TT * 2 * NP;
    float2* dd = sdt + (in & 1) * TT * CH + lc;
#pragma unroll
    for (int j = 0; j < G; ++j) {
      const int r = ft + (g + j) * STEP, to = out * TT + r, i = (tid + (g + j) * FEED_THREADS) * BW;
      const bool row = g + j < ND && r < TT;
      if (row && live && has_out && to < t_end) {
        float o[W];
        load_vec<W>(yy + r * CH, o);
#pragma unroll
        for (int e = 0; e < W; ++e) o[e] = (o[e] + skip[e] * to_f(xo[j].e[e])) * silu_t<T>(to_f(z[j].e[e]));
        store_vec<W>(yb + (long)to * C + c, o);
      }
      if (has_in && row) {
        float p[2 * W];
#pragma unroll
        for (int e = 0; e < W; ++e) {
          p[2 * e] = live && d[j].e[e] != -INFINITY ? softplus_t<T>(d[j].e[e] + bias[e]) : 0.f;
          p[2 * e + 1] = p[2 * e] * to_f(x[j].e[e]);
        }
        if constexpr (W == 4) store_vec<8>(reinterpret_cast<float*>(dd + r * CH), p);
        else dd[r * CH] = make_float2(p[0], p[1]);
      }
      if (has_in && g + j < NB && i < TT * 2 * NP) {
        float o[BW];
#pragma unroll
        for (int e = 0; e < BW; ++e) o[e] = to_f(v[j].e[e]);
        store_vec<BW>(bc + i, o);
      }
    }
  }
};

template <typename T, int P, int NS>
__global__ void __launch_bounds__(SCAN_THREADS + FEED_THREADS)
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

  const int t_end = min(n_real, a.S);
  // Turn n (-1 .. tiles) brings tile n + 1 in and takes tile n - 1 out. Where registers allow it the loads of turn n + 1 start at the end of
  // turn n and stay in flight across the barrier.
  auto feed = [&](auto width) {
    constexpr int W = decltype(width)::value;
    using Probe = Feeder<T, CH, NP, TT, W, 1>;
    constexpr bool AHEAD = W == 4 && Probe::PIECES <= 2;
    Feeder<T, CH, NP, TT, W, AHEAD ? Probe::PIECES : (W == 4 ? 2 : 4)> f;
    f.xb = xb; f.zb = zb; f.qb = qb; f.db = db; f.yb = yb; f.sBC = sBC; f.sy = sy; f.sdt = sdt; f.ldz = a.ldz; f.ldq = a.ldq;
    f.C = a.C; f.N = a.N; f.tiles = tiles; f.t_end = t_end; f.tid = tid; f.ft = tid / f.CW;
    f.c = c0 + (tid % f.CW) * W;
    f.live = f.c < a.C;
    if (f.live) {
      load_vec<W>(reinterpret_cast<const T*>(a.dt_bias) + f.c, f.bias);
      load_vec<W>(reinterpret_cast<const T*>(a.D) + f.c, f.skip);
    }
    if constexpr (AHEAD) f.issue(0, 0, -2);
    for (int n = -1; n <= tiles; ++n) {
      if constexpr (AHEAD) {
        f.settle(0, n + 1, n - 1);
        f.issue(0, n + 2, n);
      } else {
#pragma unroll 1
        for (int g = 0; g < f.PIECES; g += W == 4 ? 2 : 4) {
          f.issue(g, n + 1, n - 1);
          f.settle(g, n + 1, n - 1);
        }
      }
      if (n < tiles) tile_barrier();
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
  }
  // the two roles meet at the same barriers: one before the first tile and one after every tile
  if (consumer) {
    tile_barrier();
    for (int tile = 0; tile < tiles; ++tile) {
      const float* bc = sBC + (tile & 1) * TT * 2 * NP + ln * NS;
      const float2* dd = sdt + (tile & 1) * TT * CH + lc;
      float* yy = sy + (tile & 1) * TT * CH + lc;
      // Four steps at a time. Operands are read one group ahead and a group's read-outs are reduced while the next group computes, without
      // a branch in the loop, so that loads, exchanges and exponentials of neighbouring groups overlap in one warp.
      float2 d[4];
      float Bv[4][NS], Cv[4][NS], r[4];
      auto fetch = [&](int t) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          d[u] = dd[(t + u) * CH];
          load_vec<NS>(bc + (t + u) * 2 * NP, Bv[u]);
          load_vec<NS>(bc + (t + u) * 2 * NP + NP, Cv[u]);
        }
      };
      auto steps = [&]() {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          float acc = 0.f;
#pragma unroll
          for (int i = 0; i < NS; ++i) {
            S[i] = Decay<T>::step(S[i], d[u].x, A[i], d[u].y * Bv[u][i]);
            acc = fmaf(S[i], Cv[u][i], acc);
          }
          r[u] = acc;
        }
      };
      // sums of q[0..3] over the P lanes: lane bit 0 takes steps {0,1} or {2,3}, lane bit 1 one of the two, the remaining bits add up
      const bool b0 = ln & 1, b1 = ln & 2;
      float* mine = yy + (P == 1 ? 0 : (b0 ? 2 : 0) + (P > 2 && b1 ? 1 : 0)) * CH;
      auto reduce = [&](const float (&q)[4], float (&o)[4]) {
        if constexpr (P == 1) {
#pragma unroll
          for (int u = 0; u < 4; ++u) o[u] = q[u];
        } else {
          const float s0 = b0 ? q[0] : q[2], s1 = b0 ? q[1] : q[3];
          o[0] = (b0 ? q[2] : q[0]) + __shfl_xor_sync(0xffffffffu, s0, 1);
          o[1] = (b0 ? q[3] : q[1]) + __shfl_xor_sync(0xffffffffu, s1, 1);
          if constexpr (P > 2) {
            o[0] = (b1 ? o[1] : o[0]) + __shfl_xor_sync(0xffffffffu, b1 ? o[0] : o[1], 2);
#pragma unroll
            for (int x = 4; x < P; x <<= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], x);
          }
        }
      };
      auto put = [&](int t, const float (&o)[4]) {
        if constexpr (P == 1) {
#pragma unroll
          for (int u = 0; u < 4; ++u) mine[(t + u) * CH] = o[u];
        } else if constexpr (P == 2) {
          mine[t * CH] = o[0];
          mine[(t + 1) * CH] = o[1];
        } else {
          mine[t * CH] = o[0];                              // lanes above the fourth hold the same sum
        }
      };
      fetch(0);
      steps();
      fetch(4);
#pragma unroll 2
      for (int t = 4; t < TT; t += 4) {
        const float q[4] = {r[0], r[1], r[2], r[3]};
        float o[4];
        reduce(q, o);
        steps();
        fetch(min(t + 4, TT - 4));
        put(t - 4, o);
      }
      float o[4];
      reduce(r, o);
      put(TT - 4, o);
      tile_barrier();
    }
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (c < a.C && ln * NS + i < a.N) rec[i] = S[i];
  } else {
    const bool wide = CH % 4 == 0 && a.C % 4 == 0 && a.N == NP && a.ldz % 4 == 0 && a.ldq % 8 == 0 && a.off % 8 == 0;
    if (wide) feed(std::integral_constant<int, 4>{});
    else feed(std::integral_constant<int, 1>{});
    // right padding: nothing reads it as a value, but later products multiply it by zero
    for (int i = max(n_real, 0) * CH + tid; i < a.S * CH; i += FEED_THREADS)
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
  k<<<dim3((a.C + CH - 1) / CH, B), SCAN_THREADS + FEED_THREADS, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
int run_t(const ScanArgs& a, int B, cudaStream_t st) {
  if (a.N <= 4) return run<T, 1, 4>(a, B, st);
  if (a.N <= 8) return run<T, 2, 4>(a, B, st);
  if (a.N <= 16) return run<T, 4, 4>(a, B, st);
  if (a.N <= 32) return run<T, 8, 4>(a, B, st);
  if (a.N <= 64) return run<T, 16, 4>(a, B, st);
  if (a.N <= 128) return run<T, 32, 4>(a, B, st);
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
