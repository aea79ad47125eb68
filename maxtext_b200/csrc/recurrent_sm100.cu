// Inference kernels of the recurrent layers. Per head a matrix state S [dk, dv] in fp32, per token
//   gated delta:               S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q       (g, beta scalars per head)
//   gated linear attention:    S <- diag(alpha) S + k v^T;                        o = S^T q       (alpha per key channel)
//   retention:                 S <- d S + k v^T;                                  o = S^T q       (d fixed per head; q and k rotated)
//   channel-wise gated delta:  S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q  (g per key channel)
// Three families:
//  * decode (one token per sequence): one CTA per sequence and key head does everything between the input and the output projection:
//    short convolution, unit norms, gates, state update, read-out, head norm and output gate. Bound by reading and writing S once: it passes through
//    shared memory, and S^T k and S^T q come out of the same pass because S_new^T q = g S^T q + (k . q) u.
//  * scan (prompts): S stays in registers over the whole prompt. The columns of S never mix, so a CTA takes 16 of them and a warp 4;
//    eight lanes share a column and reduce with three shuffles.
//  * the elementwise parts of a prompt: convolution, per-channel decay, head norm with output gate.
// The decay multiplies as S + (g - 1) S with g - 1 from expm1: a slow decay is applied thousands of times, and the rounding of g itself would add up.
// Rows of a batch read the state of slot slot_ids[b] (zeros when lengths[b] == 0) and stop after new_lens[b] tokens.
#include "serving_common.cuh"
#include "warp_mma.cuh"

namespace mt {

constexpr int DEC_NT = 256;      // threads of a decode CTA
constexpr int SCAN_NT = 128;     // threads of a scan CTA
constexpr int SCAN_COLS = 16;    // state columns per scan CTA
constexpr int SCAN_TC = 16;      // tokens staged in shared memory at a time

struct RecArgs {
  int hk, r, dk, dv, S;          // key heads, value heads per key head, widths, tokens per row
  const int64_t* slot_ids;
  const int64_t* lengths;
  const int64_t* new_lens;       // or null: S everywhere
  float* rec;                    // [slots, hk * r, dk, dv]
};

template <typename T>
struct DeltaArgs {
  const T* x; long ldx;          // packed per key head: q dk | k dk | v r*dv | z r*dv
  const T* ba; long ldb;         // packed per key head: b r | a r
  const T* conv_w; int taps;     // [taps, conv_dim], channels q | k | v over all heads
  float* conv;                   // [slots, taps - 1, conv_dim]
  const T* A_log; const T* dt_bias;
};

template <typename T>
struct GlaArgs {
  const T* x; long ldx;          // q H*dk | k H*dk | v H*dv | gate H*dv | rank
  const T* w; const T* bias;     // decay projection [H*dk, rank], [H*dk]
  int rank; float inv_tau;
};

template <typename T>
struct RetArgs {
  const T* x; long ldx;          // q H*dk | k H*dk | v H*dv | gate H*dv
  const float* log_decay;        // [H]
  const float* inv_ts; int rot;  // rotated lanes, halves paired
};

template <typename T>
struct ChanArgs {
  const T* x; long ldx;          // decode: q hk*dk | k hk*dk | v hv*dv before the convolution
  const T* beta; long ldb;       // logits [N, >= hv]
  const T* conv_w; int taps;     // [taps, conv_dim]
  float* conv;                   // [slots, taps - 1, conv_dim]
  const float* da;               // product of the decay projection [N, hv*dk]
  const T* A_log; const T* dt_bias;        // [hv], [hv*dk]
  const T* z; long ldz;          // decode: gate logits [N, >= hv*dv]
};

enum { DELTA = 0, GLA = 1, RET = 2, CHAN = 3 };

__device__ __forceinline__ float beta_gate(float b) { return sigmoid_f(b); }
__device__ __forceinline__ float log_decay(float a, float A_log, float dt) { return -expf(A_log) * softplus_f(a + dt); }

// lane e of a head (at x) turned by pos * inv_ts; halves paired
template <typename T>
__device__ __forceinline__ float turned(const T* x, int e, int rot, float c, float sn) {
  const float v = to_f(x[e]);
  if (e >= rot) return v;
  const int half = rot / 2;
  return e < half ? v * c - to_f(x[e + half]) * sn : v * c + to_f(x[e - half]) * sn;
}

// ------------------------------------------------------------------------------------------------ decode
// grid (hk, B). TILE: the state of a head passes through shared memory (cp.async, several CTAs per SM hide each other's phases); otherwise it is read
// twice from global memory (states too wide for shared memory, or not a multiple of 16 bytes).
template <typename T, int KIND, bool TILE>
__global__ void __launch_bounds__(DEC_NT) recurrent_decode_kernel(RecArgs a, DeltaArgs<T> d, GlaArgs<T> gl, RetArgs<T> rt, ChanArgs<T> ch_,
                                                                 const T* __restrict__ norm_w, float eps, T* __restrict__ out, int dvp, int rows) {
  constexpr bool RULE = KIND == DELTA || KIND == CHAN;  // the write removes what the key retrieves
  constexpr bool VECDEC = KIND == GLA || KIND == CHAN;  // a decay per key channel
  extern __shared__ __align__(16) float sm[];
  const int kh = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int dk = a.dk, dv = a.dv, r = a.r, H = a.hk * r;
  const int nrg = DEC_NT / dvp;                         // row groups of `rows` rows each
  const int rg = tid / dvp, c = tid % dvp;
  float* tile = sm;                                     // [dk * dv]
  float* qs = tile + (TILE ? dk * dv : 0);              // [rows * nrg] each
  float* ks = qs + rows * nrg;
  float* al = ks + rows * nrg;                          // decay - 1 per key channel
  float* qa = al + (VECDEC ? rows * nrg : 0);           // decayed q and k (CHAN: they differ between the value heads of a key head)
  float* ka = qa + (KIND == CHAN ? rows * nrg : 0);
  float* redk = ka + (KIND == CHAN ? rows * nrg : 0);   // [DEC_NT]
  float* redq = redk + DEC_NT;
  float* wsum = redq + DEC_NT;                          // [DEC_NT / 32]
  float* vs = wsum + DEC_NT / 32;                       // [r * dv]
  const long slot = a.slot_ids[b];
  const bool fresh = a.lengths[b] == 0;
  const bool col = c < dv;
  const int row0 = rg * rows, nrows = min(rows, dk - row0);

  auto state_of = [&](int h) { return a.rec + ((slot * H + h) * dk) * (long)dv; };
  auto load_tile = [&](int h) {
    if constexpr (TILE) {
      const float* p = state_of(h);
      if (!fresh)
        for (int i = tid * 4; i < dk * dv; i += DEC_NT * 4) la_cp_async16(tile + i, p + i, 16);
      else
        for (int i = tid * 4; i < dk * dv; i += DEC_NT * 4) *reinterpret_cast<float4*>(tile + i) = make_float4(0.f, 0.f, 0.f, 0.f);
      la_commit();
    }
  };
  load_tile(kh * r);                                    // in flight while the convolution and the gates are computed

  const T* xr;
  if constexpr (RULE) {
    const int per = 2 * dk + 2 * r * dv, key_dim = a.hk * dk, conv_dim = 2 * key_dim + H * dv, K = KIND == DELTA ? d.taps : ch_.taps;
    xr = KIND == DELTA ? d.x + b * d.ldx + (long)kh * per : ch_.x + b * ch_.ldx;
    float* cs = (KIND == DELTA ? d.conv : ch_.conv) + slot * (long)(K - 1) * conv_dim;
    const T* conv_w = KIND == DELTA ? d.conv_w : ch_.conv_w;
    for (int i = tid; i < 2 * dk + r * dv; i += DEC_NT) {
      const int ch = i < dk ? kh * dk + i : (i < 2 * dk ? key_dim + kh * dk + (i - dk) : 2 * key_dim + kh * r * dv + (i - 2 * dk));
      const float xv = to_f(xr[KIND == DELTA ? i : ch]);
      float acc = to_f(conv_w[(long)(K - 1) * conv_dim + ch]) * xv;
      for (int j = 0; j < K - 1; ++j) {
        const float old = fresh ? 0.f : cs[(long)j * conv_dim + ch];
        acc += to_f(conv_w[(long)j * conv_dim + ch]) * old;
        if (j > 0) cs[(long)(j - 1) * conv_dim + ch] = old;
      }
      if (K > 1) cs[(long)(K - 2) * conv_dim + ch] = xv;
      const float y = to_f(from_f<T>(silu_t<T>(acc)));
      if (i < dk) qs[i] = y;
      else if (i < 2 * dk) ks[i - dk] = y;
      else vs[i - 2 * dk] = y;
    }
  } else if constexpr (KIND == RET) {
    xr = rt.x + b * rt.ldx;
    const float pos = (float)a.lengths[b];
    const T *xq = xr + (long)kh * dk, *xk = xr + (long)H * dk + (long)kh * dk;
    for (int i = tid; i < dk; i += DEC_NT) {
      float sn = 0.f, c = 1.f;
      if (i < rt.rot) sincosf(pos * rt.inv_ts[i % (rt.rot / 2)], &sn, &c);
      qs[i] = turned(xq, i, rt.rot, c, sn);
      ks[i] = turned(xk, i, rt.rot, c, sn);
    }
    for (int i = tid; i < dv; i += DEC_NT) vs[i] = to_f(xr[2L * H * dk + kh * dv + i]);
  } else {
    xr = gl.x + b * gl.ldx;
    for (int i = tid; i < dk; i += DEC_NT) {
      const T* w = gl.w + ((long)kh * dk + i) * gl.rank;
      const T* lo = xr + 2L * H * (dk + dv);
      float z = to_f(gl.bias[kh * dk + i]);
      for (int j = 0; j < gl.rank; j += 8) {
        float wv[8];
        load_vec<8>(w + j, wv);
#pragma unroll
        for (int e = 0; e < 8; ++e) z += wv[e] * to_f(lo[j + e]);
      }
      al[i] = expm1f(log_sigmoid_f(z) * gl.inv_tau);
      qs[i] = to_f(xr[(long)kh * dk + i]);
      ks[i] = to_f(xr[(long)H * dk + kh * dk + i]);
    }
    for (int i = tid; i < dv; i += DEC_NT) vs[i] = to_f(xr[2L * H * dk + kh * dv + i]);
  }
  __syncthreads();
  // per-token scalars, by every warp on its own
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int i = tid & 31; i < dk; i += 32) {
    qq += qs[i] * qs[i]; kk += ks[i] * ks[i]; qk += qs[i] * ks[i];
  }
  qk = warp_add(qk);
  float rq = rsqrtf((float)dk), rk = 1.f;
  if constexpr (RULE) {
    rq *= rsqrtf(warp_add(qq) + 1e-6f);
    rk = rsqrtf(warp_add(kk) + 1e-6f);
  }
  qk *= rq * rk;
  if (KIND == GLA) {                                         // S_new^T q = S^T (alpha q) + (k . q) v
    __syncthreads();
    for (int i = tid; i < dk; i += DEC_NT) qs[i] += al[i] * qs[i];
  }
  for (int j = 0; j < r; ++j) {
    const int h = kh * r + j;
    if (j > 0) load_tile(h);
    if constexpr (KIND == CHAN) {
      const float rate = -expf(to_f(ch_.A_log[h]));
      for (int i = tid; i < dk; i += DEC_NT) {
        const float g = expm1f(rate * softplus_f(ch_.da[((long)b * H + h) * dk + i] + to_f(ch_.dt_bias[(long)h * dk + i])));
        al[i] = g;
        qa[i] = qs[i] + g * qs[i];
        ka[i] = ks[i] + g * ks[i];
      }
    }
    la_wait<0>();
    __syncthreads();
    float* gp = state_of(h);
    const float* sp = (TILE ? tile : gp) + (long)row0 * dv + c;
    const bool read = col && (TILE || !fresh);
    float pk = 0.f, pq = 0.f;
    if (read) {
#pragma unroll 8
      for (int i = 0; i < nrows; ++i) {
        const float s = sp[(long)i * dv];
        if (RULE) pk += s * (KIND == CHAN ? ka : ks)[row0 + i];
        pq += s * (KIND == CHAN ? qa : qs)[row0 + i];
      }
    }
    if (RULE) redk[tid] = pk;
    redq[tid] = pq;
    __syncthreads();
    float sk = 0.f, sq = 0.f;
    for (int g = 0; g < nrg; ++g) {
      if (RULE) sk += redk[g * dvp + c];
      sq += redq[g * dvp + c];
    }
    float dm1 = 0.f, u = 0.f;
    const float v = col ? vs[j * dv + c] : 0.f;
    if constexpr (KIND == DELTA) {
      const T* bb = d.ba + b * d.ldb + (long)kh * 2 * r;
      dm1 = expm1f(log_decay(to_f(bb[r + j]), to_f(d.A_log[h]), to_f(d.dt_bias[h])));
      sk += dm1 * sk;
      sq += dm1 * sq;
      u = beta_gate(to_f(bb[j])) * (v - rk * sk);
    } else if constexpr (KIND == CHAN) {
      u = beta_gate(to_f(ch_.beta[b * ch_.ldb + h])) * (v - rk * sk);
    } else {
      if constexpr (KIND == RET) {
        dm1 = expm1f(rt.log_decay[h]);
        sq += dm1 * sq;
      }
      u = v;
    }
    const float o = col ? rq * sq + qk * u : 0.f;
    const float ku = rk * u;
    if (col) {
      float* wp = gp + (long)row0 * dv + c;
#pragma unroll 8
      for (int i = 0; i < nrows; ++i) {
        const float s = read ? sp[(long)i * dv] : 0.f;
        wp[(long)i * dv] = s + (VECDEC ? al[row0 + i] : dm1) * s + ks[row0 + i] * ku;
      }
    }
    // head norm over dv and output gate
    const float ws = warp_add(o * o);
    if ((tid & 31) == 0) wsum[tid >> 5] = ws;
    __syncthreads();
    float ss = 0.f;
    for (int g = 0; g < dvp / 32; ++g) ss += wsum[g];                 // row group 0 sees every column once
    if (rg == 0 && col) {
      const float rstd = rsqrtf(ss / (float)dv + eps);
      const T* zp = KIND == DELTA ? xr + 2 * dk + r * dv + j * dv : KIND == CHAN ? ch_.z + b * ch_.ldz + (long)h * dv
                                  : xr + 2L * H * dk + (long)H * dv + kh * dv;
      const float z = to_f(zp[c]);
      out[((long)b * H + h) * dv + c] = from_f<T>(o * rstd * (norm_w ? to_f(norm_w[c]) : 1.f) * (KIND == CHAN ? sigmoid_f(z) : silu_t<T>(z)));
    }
  }
}

// ------------------------------------------------------------------------------------------------ convolution of a prompt
// y[n, ch] = silu(sum_j w[j, ch] x[t - taps + 1 + j]) with inputs before the row's first new token taken from the state.
// grid (channel groups, token tiles, B); a thread owns VEC channels and walks CONV_TT tokens.
constexpr int CONV_TT = 16;

template <typename T, int VEC, int MAXK>
__global__ void delta_conv_kernel(RecArgs a, DeltaArgs<T> d, T* __restrict__ y) {
  const int dk = a.dk, dv = a.dv, r = a.r, key_dim = a.hk * dk, conv_dim = 2 * key_dim + a.hk * r * dv, K = d.taps;
  const int ch = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (ch >= conv_dim) return;
  const int b = blockIdx.z, t0 = blockIdx.y * CONV_TT;
  const int per = 2 * dk + 2 * r * dv;
  long src;                                              // column of the packed projection
  if (ch < key_dim) src = (long)(ch / dk) * per + ch % dk;
  else if (ch < 2 * key_dim) src = (long)((ch - key_dim) / dk) * per + dk + (ch - key_dim) % dk;
  else src = (long)((ch - 2 * key_dim) / (r * dv)) * per + 2 * dk + (ch - 2 * key_dim) % (r * dv);
  const T* __restrict__ xb = d.x + (long)b * a.S * d.ldx + src;
  const bool fresh = a.lengths[b] == 0;
  const float* cs = d.conv + a.slot_ids[b] * (long)(K - 1) * conv_dim + ch;
  float w[MAXK][VEC], hist[MAXK][VEC];                   // hist[j]: input of tap j; the last K entries are used
#pragma unroll
  for (int j = 0; j < MAXK; ++j) {
    const int tap = j - (MAXK - K), t = t0 + tap - (K - 1);
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[j][e] = hist[j][e] = 0.f;
    if (tap >= 0) {
      load_vec<VEC>(d.conv_w + (long)tap * conv_dim + ch, w[j]);
      if (j < MAXK - 1) {
        if (t >= 0) load_vec<VEC>(xb + (long)t * d.ldx, hist[j]);
        else if (!fresh) load_vec<VEC>(cs + (long)(K - 1 + t) * conv_dim, hist[j]);
      }
    }
  }
  const int t1 = min(t0 + CONV_TT, a.S);
  T* __restrict__ yb = y + (long)b * a.S * conv_dim + ch;
  for (int t = t0; t < t1; t += 4) {
    float in[4][VEC];                                    // four loads in flight
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (t + u < t1) load_vec<VEC>(xb + (long)(t + u) * d.ldx, in[u]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (t + u < t1) {
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          hist[MAXK - 1][e] = in[u][e];
          acc[e] = 0.f;
        }
#pragma unroll
        for (int j = 0; j < MAXK; ++j)
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[e] += w[j][e] * hist[j][e];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = silu_t<T>(acc[e]);
        store_vec<VEC>(yb + (long)(t + u) * conv_dim, acc);
#pragma unroll
        for (int j = 0; j < MAXK - 1; ++j)
#pragma unroll
          for (int e = 0; e < VEC; ++e) hist[j][e] = hist[j + 1][e];
      }
    }
  }
}

// the last taps - 1 inputs of every row become its state; runs after delta_conv_kernel has read the old one. grid (channels / 128, B)
template <typename T>
__global__ void conv_state_kernel(RecArgs a, DeltaArgs<T> d) {
  const int dk = a.dk, dv = a.dv, r = a.r, key_dim = a.hk * dk, conv_dim = 2 * key_dim + a.hk * r * dv, K = d.taps;
  const int ch = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (ch >= conv_dim) return;
  const int per = 2 * dk + 2 * r * dv;
  long src;
  if (ch < key_dim) src = (long)(ch / dk) * per + ch % dk;
  else if (ch < 2 * key_dim) src = (long)((ch - key_dim) / dk) * per + dk + (ch - key_dim) % dk;
  else src = (long)((ch - 2 * key_dim) / (r * dv)) * per + 2 * dk + (ch - 2 * key_dim) % (r * dv);
  const int n = a.new_lens ? (int)a.new_lens[b] : a.S;
  const bool fresh = a.lengths[b] == 0;
  float* cs = d.conv + a.slot_ids[b] * (long)(K - 1) * conv_dim + ch;
  for (int j = 0; j < K - 1; ++j) {
    const int t = n - (K - 1) + j;                       // an older input sits at row n + j > j: rows are read before they are replaced
    const float v = t >= 0 ? to_f(d.x[((long)b * a.S + t) * d.ldx + src]) : (fresh ? 0.f : cs[(long)(K - 1 + t) * conv_dim]);
    cs[(long)j * conv_dim] = v;
  }
}

// ------------------------------------------------------------------------------------------------ per-channel decay of a prompt
// log_alpha[n, c] = log_sigmoid(bias[c] + sum_j w[c, j] lo[n, j]) / tau. grid (channels / 128, tokens / 32); rank is a multiple of 8.
template <typename T>
__global__ void __launch_bounds__(128) gla_decay_kernel(const T* __restrict__ lo, long ldx, const T* __restrict__ w, const T* __restrict__ bias, int rank,
                                                        float inv_tau, float* __restrict__ out, long N, int C) {
  __shared__ __align__(16) float as[32][8];
  const int c = blockIdx.x * 128 + threadIdx.x;
  const long n0 = (long)blockIdx.y * 32;
  float acc[32];
  const float b0 = c < C ? to_f(bias[c]) : 0.f;
#pragma unroll
  for (int i = 0; i < 32; ++i) acc[i] = b0;
  for (int j0 = 0; j0 < rank; j0 += 8) {
    __syncthreads();
    for (int i = threadIdx.x; i < 256; i += 128) as[i >> 3][i & 7] = n0 + (i >> 3) < N ? to_f(lo[(n0 + (i >> 3)) * ldx + j0 + (i & 7)]) : 0.f;
    __syncthreads();
    if (c < C) {
      float wv[8];
      load_vec<8>(w + (long)c * rank + j0, wv);
#pragma unroll
      for (int i = 0; i < 32; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i] += wv[e] * as[i][e];
    }
  }
  if (c < C) {
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (n0 + i < N) out[(n0 + i) * C + c] = log_sigmoid_f(acc[i]) * inv_tau;
  }
}

// The same with the product on tensor cores (bf16): grid (ceil(C / 64), ceil(N / 64)), 128 threads; rows of lo and w start on 16 bytes.
__global__ void __launch_bounds__(128) gla_decay_tc_kernel(const __nv_bfloat16* __restrict__ lo, long ldx, const __nv_bfloat16* __restrict__ w,
                                                           const __nv_bfloat16* __restrict__ bias, int rank, float inv_tau, float* __restrict__ out, long N,
                                                           int C) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int kp = (rank + 15) & ~15, LD = kp + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c0 = blockIdx.x * 64;
  const long n0 = (long)blockIdx.y * 64;
  __nv_bfloat16* as = reinterpret_cast<__nv_bfloat16*>(raw);       // [64][LD]
  __nv_bfloat16* ws = as + 64 * LD;
  for (int i = tid; i < 64 * (kp / 8); i += 128) {
    const int r = i / (kp / 8), k = (i % (kp / 8)) * 8;
    const bool ka = k < rank, na = n0 + r < N, ca = c0 + r < C;
    la_cp_async16(as + r * LD + k, lo + (na ? n0 + r : 0) * ldx + (ka ? k : 0), ka && na ? 16 : 0);
    la_cp_async16(ws + r * LD + k, w + (long)(ca ? c0 + r : 0) * rank + (ka ? k : 0), ka && ca ? 16 : 0);
  }
  la_commit();
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = c0 + n * 8 + (lane & 3) * 2 + (e & 1);
      acc[n][e] = c < C ? to_f(bias[c]) : 0.f;
    }
  la_wait<0>();
  __syncthreads();
  for (int k = 0; k < kp; k += 16) {
    unsigned fa[4];
    la_ldm4(fa, as + (warp * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8);
#pragma unroll
    for (int n = 0; n < 8; n += 2) {
      unsigned fb[4];
      la_ldm4(fb, ws + (n * 8 + (lane & 7) + ((lane >> 4) << 3)) * LD + k + ((lane >> 3) & 1) * 8);
      la_mma(acc[n], fa, fb[0], fb[1]);
      la_mma(acc[n + 1], fa, fb[2], fb[3]);
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const long n = n0 + warp * 16 + (lane >> 2) + e * 8;
    if (n >= N) continue;
#pragma unroll
    for (int x = 0; x < 8; ++x) {
      const int c = c0 + x * 8 + (lane & 3) * 2;           // C is even
      if (c < C) *reinterpret_cast<float2*>(out + n * C + c) = make_float2(log_sigmoid_f(acc[x][2 * e]) * inv_tau, log_sigmoid_f(acc[x][2 * e + 1]) * inv_tau);
    }
  }
}

// ------------------------------------------------------------------------------------------------ scan over a prompt
// grid (ceil(dv / 16), heads, B). q / k of token n sit at q[n * ldq + (h / r) * dk]; likewise v and, for GLA, log_alpha (fp32).
template <typename T, int KIND, int RPT>
__global__ void __launch_bounds__(SCAN_NT) recurrent_scan_kernel(RecArgs a, const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                                                long ldx, const float* __restrict__ log_alpha, const T* __restrict__ ba, long ldb,
                                                                const T* __restrict__ A_log, const T* __restrict__ dt_bias, RetArgs<T> rt, ChanArgs<T> ch,
                                                                T* __restrict__ o) {
  constexpr bool RULE = KIND == DELTA || KIND == CHAN, VECDEC = KIND == GLA || KIND == CHAN;
  constexpr int GS = RPT + 4;                            // floats per row group: the eight groups start in different banks
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dk = a.dk, dv = a.dv, r = a.r, H = a.hk * r, kh = h / r;
  float* qs = sm;                                        // [TC][8 * GS]
  float* ks = qs + SCAN_TC * 8 * GS;
  float* as = ks + SCAN_TC * 8 * GS;                     // decay - 1 per key channel
  float* vs = as + (VECDEC ? SCAN_TC * 8 * GS : 0);      // [TC][16]
  float* sc = vs + SCAN_TC * SCAN_COLS;                  // [TC][4]: decay - 1, beta, rq, k.q (normalised); rk is folded into ks
  const int c0 = blockIdx.x * SCAN_COLS, cl = warp * 4 + (lane & 3), c = c0 + cl, rg = lane >> 2;
  const bool col = c < dv;
  const long slot = a.slot_ids[b];
  const bool fresh = a.lengths[b] == 0;
  const int n = a.new_lens ? (int)a.new_lens[b] : a.S;
  float* sp = a.rec + ((slot * H + h) * dk) * (long)dv + c;
  float S[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) S[i] = (!fresh && col && rg * RPT + i < dk) ? sp[(long)(rg * RPT + i) * dv] : 0.f;
  const float qscale = rsqrtf((float)dk);
  for (int i = tid; i < SCAN_TC * 8 * GS; i += SCAN_NT) {      // padding rows stay zero
    qs[i] = 0.f; ks[i] = 0.f;
    if (VECDEC) as[i] = 0.f;
  }
  const float rate = KIND == CHAN ? -expf(to_f(ch.A_log[h])) : 0.f;
  for (int t0 = 0; t0 < n; t0 += SCAN_TC) {
    const int m = min(SCAN_TC, n - t0);
    __syncthreads();
    for (int i = tid; i < m * dk; i += SCAN_NT) {
      const int t = i / dk, e = i % dk;
      const long row = (long)b * a.S + t0 + t;
      const int at = t * 8 * GS + (e / RPT) * GS + e % RPT;
      if constexpr (KIND == RET) {
        float sn = 0.f, c_ = 1.f;
        if (e < rt.rot) sincosf((float)(a.lengths[b] + t0 + t) * rt.inv_ts[e % (rt.rot / 2)], &sn, &c_);
        qs[at] = turned(q + row * ldx + (long)kh * dk, e, rt.rot, c_, sn);
        ks[at] = turned(k + row * ldx + (long)kh * dk, e, rt.rot, c_, sn);
      } else {
        qs[at] = to_f(q[row * ldx + (long)kh * dk + e]);
        ks[at] = to_f(k[row * ldx + (long)kh * dk + e]);
      }
      if (KIND == GLA) as[at] = expm1f(log_alpha[row * (long)H * dk + (long)h * dk + e]);
      if (KIND == CHAN) as[at] = expm1f(rate * softplus_f(ch.da[row * (long)H * dk + (long)h * dk + e] + to_f(ch.dt_bias[(long)h * dk + e])));
    }
    for (int i = tid; i < m * SCAN_COLS; i += SCAN_NT) {
      const int t = i / SCAN_COLS, e = c0 + i % SCAN_COLS;
      vs[i] = e < dv ? to_f(v[((long)b * a.S + t0 + t) * ldx + (long)h * dv + e]) : 0.f;
    }
    __syncthreads();
    for (int t = warp; t < m; t += SCAN_NT / 32) {
      float qq = 0.f, kk = 0.f, qk = 0.f;
      for (int e = lane; e < dk; e += 32) {
        const int at = t * 8 * GS + (e / RPT) * GS + e % RPT;
        qq += qs[at] * qs[at]; kk += ks[at] * ks[at]; qk += qs[at] * ks[at];
      }
      qk = warp_add(qk);
      float rq = qscale, rk = 1.f;
      if (KIND == RET && lane == 0) sc[t * 4] = expm1f(rt.log_decay[h]);
      if (KIND == CHAN && lane == 0) sc[t * 4 + 1] = beta_gate(to_f(ch.beta[((long)b * a.S + t0 + t) * ch.ldb + h]));
      if constexpr (RULE) {
        rq *= rsqrtf(warp_add(qq) + 1e-6f);
        rk = rsqrtf(warp_add(kk) + 1e-6f);
        for (int e = lane; e < dk; e += 32) ks[t * 8 * GS + (e / RPT) * GS + e % RPT] *= rk;
        if (KIND == DELTA && lane == 0) {
          const T* bb = ba + ((long)b * a.S + t0 + t) * ldb + (long)kh * 2 * r + (h - kh * r);
          sc[t * 4] = expm1f(log_decay(to_f(bb[r]), to_f(A_log[h]), to_f(dt_bias[h])));
          sc[t * 4 + 1] = beta_gate(to_f(bb[0]));
        }
      }
      if (lane == 0) { sc[t * 4 + 2] = rq; sc[t * 4 + 3] = qk * rq * rk; }
    }
    __syncthreads();
    for (int t = 0; t < m; ++t) {
      const float* qt = qs + t * 8 * GS + rg * GS;
      const float* kt = ks + t * 8 * GS + rg * GS;
      const float* at = as + t * 8 * GS + rg * GS;
      float sk = 0.f, sq = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        if constexpr (VECDEC) S[i] += at[i] * S[i];
        if constexpr (RULE) sk += S[i] * kt[i];
        sq += S[i] * qt[i];
      }
#pragma unroll
      for (int w = 4; w <= 16; w <<= 1) {
        if (RULE) sk += __shfl_xor_sync(0xffffffffu, sk, w);
        sq += __shfl_xor_sync(0xffffffffu, sq, w);
      }
      const float rq = sc[t * 4 + 2], kq = sc[t * 4 + 3];
      float u = vs[t * SCAN_COLS + cl];
      if constexpr (KIND == CHAN) u = sc[t * 4 + 1] * (u - sk);
      if constexpr (!VECDEC) {
        const float dm1 = sc[t * 4];
        sk += dm1 * sk;
        sq += dm1 * sq;
        if (KIND == DELTA) u = sc[t * 4 + 1] * (u - sk);
#pragma unroll
        for (int i = 0; i < RPT; ++i) S[i] += dm1 * S[i];
      }
#pragma unroll
      for (int i = 0; i < RPT; ++i) S[i] += kt[i] * u;
      if (rg == 0 && col) o[((long)b * a.S + t0 + t) * (long)H * dv + (long)h * dv + c] = from_f<T>(rq * sq + kq * u);
    }
  }
  // padding positions of the output are read by the norm kernel: give them a value
  for (int t = n + tid / SCAN_COLS; t < a.S; t += SCAN_NT / SCAN_COLS) {
    const int e = c0 + tid % SCAN_COLS;
    if (e < dv) o[((long)b * a.S + t) * (long)H * dv + (long)h * dv + e] = from_f<T>(0.f);
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i)
    if (col && rg * RPT + i < dk) sp[(long)(rg * RPT + i) * dv] = S[i];
}

// ------------------------------------------------------------------------------------------------ head norm + output gate
// out[n, h, :] = rms(o[n, h, :]) * w * silu(z) (without w: no weight; SIG: sigmoid(z)), one warp per (n, h); z of head h sits at x[n * ldx + zoff + (h / r) * zstride + (h % r) * dv].
// LPR lanes share a row.
template <typename T, int VEC, int LPR, bool SIG>
__global__ void __launch_bounds__(256) gated_head_norm_kernel(const T* __restrict__ o, const T* __restrict__ x, long ldx, long rows, int H, int dv, int r,
                                                              long zoff, long zstride, const T* __restrict__ w, float eps, T* __restrict__ out) {
  const long row = ((long)blockIdx.x * blockDim.x + threadIdx.x) / LPR;
  const int lane = threadIdx.x % LPR;
  const bool in = row < rows;
  const long n = in ? row / H : 0;
  const int h = in ? (int)(row % H) : 0;
  const T* op = o + (in ? row : 0) * dv;
  const T* zp = x + n * ldx + zoff + (long)(h / r) * zstride + (long)(h % r) * dv;
  float ss = 0.f, v[VEC];
  for (int c = lane * VEC; c < dv; c += LPR * VEC) {
    load_vec<VEC>(op + c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
  }
#pragma unroll
  for (int s = LPR / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!in) return;
  const float rstd = rsqrtf(ss / (float)dv + eps);
  const bool once = dv <= LPR * VEC;                     // the row is still in registers
  for (int c = lane * VEC; c < dv; c += LPR * VEC) {
    float z[VEC], g[VEC];
    if (!once) load_vec<VEC>(op + c, v);
    load_vec<VEC>(zp + c, z);
    if (w) load_vec<VEC>(w + c, g);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * (w ? rstd * g[e] : rstd) * (SIG ? sigmoid_t<T>(z[e]) : silu_t<T>(z[e]));
    store_vec<VEC>(out + row * dv + c, v);
  }
}

// ------------------------------------------------------------------------------------------------ launchers
template <typename T, int KIND>
int launch_decode(const RecArgs& a, const DeltaArgs<T>& d, const GlaArgs<T>& g, const RetArgs<T>& rt, const ChanArgs<T>& ch, const void* norm, float eps,
                  void* out, int B, cudaStream_t st) {
  int dvp = 32;
  while (dvp < a.dv) dvp <<= 1;
  if (dvp > DEC_NT) return -1;
  const int nrg = DEC_NT / dvp, rows = ((a.dk + nrg - 1) / nrg + 3) & ~3;
  const size_t state = sizeof(float) * (size_t)a.dk * a.dv;
  const bool tile = state % 16 == 0 && state <= 160 * 1024;
  const size_t smem = (tile ? state : 0) + sizeof(float) * ((KIND == CHAN ? 5 : KIND == GLA ? 3 : 2) * (size_t)rows * nrg + (size_t)a.r * a.dv + 2 * DEC_NT + DEC_NT / 32);
  if (smem > 220 * 1024) return -1;
  auto k1 = recurrent_decode_kernel<T, KIND, true>;
  auto k0 = recurrent_decode_kernel<T, KIND, false>;
  auto k = tile ? k1 : k0;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
  k<<<dim3(a.hk, B), DEC_NT, smem, st>>>(a, d, g, rt, ch, (const T*)norm, eps, (T*)out, dvp, rows);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T, int KIND>
int launch_scan(const RecArgs& a, const void* q, const void* k, const void* v, long ldx, const float* la, const void* ba, long ldb, const void* A,
                const void* dt, const RetArgs<T>& rt, const ChanArgs<T>& ch, void* o, int B, cudaStream_t st) {
  const int need = (a.dk + 7) / 8;
  const int rpt = need <= 4 ? 4 : need <= 8 ? 8 : need <= 16 ? 16 : need <= 32 ? 32 : 0;
  if (!rpt) return -1;
  const size_t smem = sizeof(float) * ((KIND == GLA || KIND == CHAN ? 3 : 2) * (size_t)SCAN_TC * 8 * (rpt + 4) + SCAN_TC * SCAN_COLS + SCAN_TC * 4);
  auto kern = rpt == 4 ? recurrent_scan_kernel<T, KIND, 4> : rpt == 8 ? recurrent_scan_kernel<T, KIND, 8> : rpt == 16
      ? recurrent_scan_kernel<T, KIND, 16> : recurrent_scan_kernel<T, KIND, 32>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -2;
  kern<<<dim3((a.dv + SCAN_COLS - 1) / SCAN_COLS, a.hk * a.r, B), SCAN_NT, smem, st>>>(
      a, (const T*)q, (const T*)k, (const T*)v, ldx, la, (const T*)ba, ldb, (const T*)A, (const T*)dt, rt, ch, (T*)o);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
int launch_conv(const RecArgs& a, const DeltaArgs<T>& d, void* y, int B, cudaStream_t st) {
  const int conv_dim = 2 * a.hk * a.dk + a.hk * a.r * a.dv;
  constexpr int V = 16 / sizeof(T);
  const unsigned tiles = (a.S + CONV_TT - 1) / CONV_TT;
  if (d.taps <= 4 && a.dk % V == 0 && a.dv % V == 0 && d.ldx % V == 0)
    delta_conv_kernel<T, V, 4><<<dim3((conv_dim / V + 127) / 128, tiles, B), 128, 0, st>>>(a, d, (T*)y);
  else if (d.taps <= 8)
    delta_conv_kernel<T, 1, 8><<<dim3((conv_dim + 127) / 128, tiles, B), 128, 0, st>>>(a, d, (T*)y);
  else if (d.taps <= 64)
    delta_conv_kernel<T, 1, 64><<<dim3((conv_dim + 127) / 128, tiles, B), 128, 0, st>>>(a, d, (T*)y);
  else
    return -1;
  if (d.taps > 1) conv_state_kernel<T><<<dim3((conv_dim + 127) / 128, B), 128, 0, st>>>(a, d);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

template <typename T>
int launch_head_norm(const void* o, const void* x, long ldx, long rows, int H, int dv, int r, long zoff, long zstride, const void* w, float eps, int sig,
                     void* out, cudaStream_t st) {
  const bool v8 = dv % 8 == 0 && ldx % 8 == 0 && zoff % 8 == 0 && zstride % 8 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0;
#define GO_(V, L, S) gated_head_norm_kernel<T, V, L, S><<<(unsigned)((rows * L + 255) / 256), 256, 0, st>>>((const T*)o, (const T*)x, ldx, rows, H, dv, r, \
                                                                                                         zoff, zstride, (const T*)w, eps, (T*)out)
#define GO(V, L) do { if (sig) GO_(V, L, true); else GO_(V, L, false); } while (0)
  if (!v8) GO(1, 32);
  else if (dv <= 64) GO(8, 8);
  else if (dv <= 128) GO(8, 16);
  else GO(8, 32);
#undef GO
#undef GO_
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace mt

using namespace mt;

#define MT_BY_TYPE(f32, CALL) ((f32) ? CALL(float) : CALL(__nv_bfloat16))

extern "C" int mt_delta_decode(int f32, const void* x, long ldx, const void* ba, long ldb, const void* conv_w, int taps, const void* A_log,
                               const void* dt_bias, const void* norm, float eps, int hk, int hv, int dk, int dv, float* conv, float* rec,
                               const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st) {
  if (B <= 0) return 0;
  const RecArgs a{hk, hv / hk, dk, dv, 1, slots, lengths, nullptr, rec};
#define CALL(T) launch_decode<T, DELTA>(a, DeltaArgs<T>{(const T*)x, ldx, (const T*)ba, ldb, (const T*)conv_w, taps, conv, (const T*)A_log, \
                                                       (const T*)dt_bias}, GlaArgs<T>{}, RetArgs<T>{}, ChanArgs<T>{}, norm, eps, out, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_gla_decode(int f32, const void* x, long ldx, const void* w, const void* bias, int rank, float inv_tau, const void* norm, float eps,
                             int H, int dk, int dv, float* rec, const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st) {
  if (B <= 0) return 0;
  const RecArgs a{H, 1, dk, dv, 1, slots, lengths, nullptr, rec};
#define CALL(T) launch_decode<T, GLA>(a, DeltaArgs<T>{}, GlaArgs<T>{(const T*)x, ldx, (const T*)w, (const T*)bias, rank, inv_tau}, RetArgs<T>{}, \
                                      ChanArgs<T>{}, norm, eps, out, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_delta_conv(int f32, const void* x, long ldx, const void* conv_w, int taps, int hk, int hv, int dk, int dv, int S, float* conv,
                             const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* y, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const RecArgs a{hk, hv / hk, dk, dv, S, slots, lengths, new_lens, nullptr};
#define CALL(T) launch_conv<T>(a, DeltaArgs<T>{(const T*)x, ldx, nullptr, 0, (const T*)conv_w, taps, conv, nullptr, nullptr}, y, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_delta_scan(int f32, const void* mixed, const void* ba, long ldb, const void* A_log, const void* dt_bias, int hk, int hv, int dk, int dv,
                             int S, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const RecArgs a{hk, hv / hk, dk, dv, S, slots, lengths, new_lens, rec};
  const long ld = 2L * hk * dk + (long)hv * dv;
#define CALL(T) launch_scan<T, DELTA>(a, (const T*)mixed, (const T*)mixed + (long)hk * dk, (const T*)mixed + 2L * hk * dk, ld, nullptr, ba, ldb, A_log, \
                                     dt_bias, RetArgs<T>{}, ChanArgs<T>{}, o, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_gla_scan(int f32, const void* x, long ldx, const float* log_alpha, int H, int dk, int dv, int S, float* rec, const int64_t* slots,
                           const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const RecArgs a{H, 1, dk, dv, S, slots, lengths, new_lens, rec};
#define CALL(T) launch_scan<T, GLA>(a, (const T*)x, (const T*)x + (long)H * dk, (const T*)x + 2L * H * dk, ldx, log_alpha, nullptr, 0, nullptr, nullptr, \
                                      RetArgs<T>{}, ChanArgs<T>{}, o, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_gla_decay(int f32, const void* lo, long ldx, const void* w, const void* bias, int rank, float inv_tau, float* out, long N, int C,
                            cudaStream_t st) {
  if (N <= 0) return 0;
  if (rank % 8) return -1;
  if (!f32 && C % 2 == 0 && ldx % 8 == 0 && reinterpret_cast<uintptr_t>(lo) % 16 == 0 && rank <= 160) {
    const size_t smem = 2 * 2 * 64 * (size_t)(((rank + 15) & ~15) + 8);
    gla_decay_tc_kernel<<<dim3((C + 63) / 64, (unsigned)((N + 63) / 64)), 128, smem, st>>>((const __nv_bfloat16*)lo, ldx, (const __nv_bfloat16*)w,
                                                                                       (const __nv_bfloat16*)bias, rank, inv_tau, out, N, C);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  const dim3 grid((C + 127) / 128, (unsigned)((N + 31) / 32));
  if (f32) gla_decay_kernel<float><<<grid, 128, 0, st>>>((const float*)lo, ldx, (const float*)w, (const float*)bias, rank, inv_tau, out, N, C);
  else gla_decay_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>((const __nv_bfloat16*)lo, ldx, (const __nv_bfloat16*)w, (const __nv_bfloat16*)bias, rank,
                                                             inv_tau, out, N, C);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

extern "C" int mt_gated_head_norm(int f32, const void* o, const void* x, long ldx, long rows, int H, int dv, int r, long zoff, long zstride, const void* w,
                                  float eps, int sig, void* out, cudaStream_t st) {
  if (rows <= 0) return 0;
  return f32 ? launch_head_norm<float>(o, x, ldx, rows, H, dv, r, zoff, zstride, w, eps, sig, out, st)
             : launch_head_norm<__nv_bfloat16>(o, x, ldx, rows, H, dv, r, zoff, zstride, w, eps, sig, out, st);
}

extern "C" int mt_retention_decode(int f32, const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, float eps, int H, int dk, int dv,
                                   float* rec, const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st) {
  if (B <= 0) return 0;
  const RecArgs a{H, 1, dk, dv, 1, slots, lengths, nullptr, rec};
#define CALL(T) launch_decode<T, RET>(a, DeltaArgs<T>{}, GlaArgs<T>{}, RetArgs<T>{(const T*)x, ldx, log_decay, inv_ts, rot}, ChanArgs<T>{}, nullptr, eps, out, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_retention_scan(int f32, const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, int H, int dk, int dv, int S, float* rec,
                                 const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const RecArgs a{H, 1, dk, dv, S, slots, lengths, new_lens, rec};
#define CALL(T) launch_scan<T, RET>(a, (const T*)x, (const T*)x + (long)H * dk, (const T*)x + 2L * H * dk, ldx, nullptr, nullptr, 0, nullptr, nullptr, \
                                    RetArgs<T>{(const T*)x, ldx, log_decay, inv_ts, rot}, ChanArgs<T>{}, o, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

extern "C" int mt_channel_delta_decode(int f32, const void* x, long ldx, const void* beta, long ldb, const void* conv_w, int taps, const float* da,
                                       const void* A_log, const void* dt_bias, const void* z, long ldz, const void* norm, float eps, int hk, int hv, int dk,
                                       int dv, float* conv, float* rec, const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st) {
  if (B <= 0) return 0;
  const RecArgs a{hk, hv / hk, dk, dv, 1, slots, lengths, nullptr, rec};
#define CALL(T) launch_decode<T, CHAN>(a, DeltaArgs<T>{}, GlaArgs<T>{}, RetArgs<T>{}, ChanArgs<T>{(const T*)x, ldx, (const T*)beta, ldb, (const T*)conv_w, \
                                       taps, conv, da, (const T*)A_log, (const T*)dt_bias, (const T*)z, ldz}, norm, eps, out, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}

// mixed [B*S, 2 hk dk + hv dv]: q | k | v after the convolution
extern "C" int mt_channel_delta_scan(int f32, const void* mixed, const void* beta, long ldb, const float* da, const void* A_log, const void* dt_bias, int hk,
                                     int hv, int dk, int dv, int S, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o,
                                     int B, cudaStream_t st) {
  if (B <= 0 || S <= 0) return 0;
  const RecArgs a{hk, hv / hk, dk, dv, S, slots, lengths, new_lens, rec};
  const long ld = 2L * hk * dk + (long)hv * dv;
#define CALL(T) launch_scan<T, CHAN>(a, (const T*)mixed, (const T*)mixed + (long)hk * dk, (const T*)mixed + 2L * hk * dk, ld, nullptr, nullptr, 0, nullptr, \
                                     nullptr, RetArgs<T>{}, ChanArgs<T>{nullptr, 0, (const T*)beta, ldb, nullptr, 1, nullptr, da, (const T*)A_log, \
                                     (const T*)dt_bias, nullptr, 0}, o, B, st)
  return MT_BY_TYPE(f32, CALL);
#undef CALL
}
