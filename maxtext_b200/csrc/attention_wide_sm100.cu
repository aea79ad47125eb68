// Flash attention forward for wide queries on tcgen05 / TMEM: every query head meets ONE key made of all key heads side by side, and the values
// of its own group. That is what attention becomes when the heads' scores are mixed by a matrix before the softmax, s_h <- sum_g T[h, g] s_g: by
// linearity the mixing moves to the queries (qkv_prep), q_h . k -> [.., sum of T[h, g] q_g over the query heads g of key head c, ..] . [.., k_c, ..].
//
// q [B, Sq, H, W], k [B, Skv, W] (W = G * D, any multiple of 8), v [B, Skv, G * Dv], out [B, Sq, H, Dv]; bf16 in / out, fp32 scores and statistics.
//
// A CTA pair (cta_group::2) holds 256 queries of one head, 128 in each CTA of 320 threads:
//   warp 0      TMA producer, in both CTAs
//   warp 1      TMEM owner; MMA issuer in the leader CTA
//   warps 2..9  softmax, two threads per query row (64 keys each)
// The contraction W passes in boxes of 64 lanes with 128-byte swizzle through a ring that keys and values share; each CTA fetches half of the keys (and
// half of the value columns) of a 128-key tile, the products read both halves. That halves what the long contraction costs in shared memory and in
// traffic: with the whole tile in each CTA the products wait for their operands. The query's boxes stay in shared memory when they fit (W <= 512) and
// pass through the ring next to the keys' otherwise. W is several times the head width, so the score products of the next key tiles are long enough to
// cover the softmax of the current one: S has three buffers in tensor memory,
//   S(0), S(1), [S(2), P(0) V], [S(3), P(1) V], ...
// A row's two threads agree on its maximum through shared memory; by then all scores of the tile are in registers, so P may overwrite S as the TMEM
// operand. Masks, the lazy rescaling and the bounded waits are those of attention_fwd_sm100.cu. Boxes that reach into a neighbour head's columns meet
// zero-filled lanes of the other operand (keys), or fill accumulator columns that are not stored (values; their width counts as 128).
#include "attention_mask.cuh"
#include "sm100_ptx.cuh"
#include <cuda_bf16.h>

namespace mt {
namespace wide {

constexpr float LOG2E = 1.4426950408889634f;
constexpr float RESCALE_THRESHOLD = 8.f;     // log2 units
constexpr int QBOX = 128 * 64 * 2, KBOX = 64 * 64 * 2, VBOX = 128 * 64 * 2;      // bytes of a box, per CTA
constexpr int STAGES_MAX = 12, RESIDENT_MAX = 8;

struct Params {
  int B, H, G, Dv, W;
  int boxes;             // of the contraction: ceil(W / 64)
  int resident, stages, stage_bytes;
  int n_pairs;           // of 256 queries
  attn::Mask mk;
  float scale;
  const __nv_bfloat16* sinks;    // [H] or nullptr
  __nv_bfloat16* out;
  int* status;
};

struct alignas(8) Ctl {
  uint64_t bars[10 + 2 * STAGES_MAX];
  uint32_t tmem_base;
  int abort_flag;
  int pad[2];
  float top[2][2][128];  // [parity][half][row] maxima; the row sums at the end
  int pos[2][128], seg[2][128];
};

__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}

__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(320, 1)
wide_flash_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                  const __grid_constant__ Params p) {
  constexpr uint32_t TMEM_COLS = 512, COL_S = 0, COL_O = 384;        // S of tile i at (i % 3) * 128
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sQ = base, sR = base + (p.resident ? p.boxes * QBOX : 0);
  Ctl* ctl = reinterpret_cast<Ctl*>(smem_raw + (sR - smem_u32(smem_raw)) + p.stages * p.stage_bytes);
  const uint32_t bar0 = smem_u32(&ctl->bars[0]);
  // leader only: Q_FULL, P_READY, FULL; in both CTAs: S_FULL, PV_DONE, EMPTY
  enum { Q_FULL = 0, S_FULL0 = 1, P_READY0 = 4, PV_DONE0 = 7, FULL0 = 9, EMPTY0 = 9 + STAGES_MAX };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t rank = cluster_ctarank();               // 0 = leader
  const int hb = p.H * p.B, pi = (int)blockIdx.x >> 1;
  const int pair = p.n_pairs - 1 - pi / hb;              // the last queries see the most keys: they come first
  const int h = pi % hb % p.H, b = pi % hb / p.H, g = h / (p.H / p.G);
  const attn::Mask& mk = p.mk;
  const attn::Span t0 = attn::q_span(mk, b, 2 * pair), t1 = attn::q_span(mk, b, 2 * pair + 1), t = rank ? t1 : t0;
  const int q0 = (2 * pair + (int)rank) * 128;
  int kt_lo, kt_hi, lo1, hi1;
  attn::k_tiles_for(mk, t0, kt_lo, kt_hi);
  attn::k_tiles_for(mk, t1, lo1, hi1);
  if (t1.rows) { kt_lo = min(kt_lo, lo1); kt_hi = max(kt_hi, hi1); }
  // the next key tile from kt on that holds a visible key for either CTA, or kt_hi: every role of the pair walks the same tiles
  auto seek = [&](int kt) {
    if (!mk.pos_k) return kt;                            // without position arrays the bounds are exact
    for (; kt < kt_hi; ++kt) {
      const attn::Span ks = attn::k_span(mk, b, kt);
      if (attn::classify(mk, t0, ks) != 0 || attn::classify(mk, t1, ks) != 0) break;
    }
    return kt;
  };

  if (threadIdx.x == 0) {
    ctl->abort_flag = 0;
    mbar_init(bar(Q_FULL), 1);
    mbar_init(bar(PV_DONE0), 1);
    mbar_init(bar(PV_DONE0 + 1), 1);
    for (int s = 0; s < 3; ++s) {
      mbar_init(bar(S_FULL0 + s), 1);
      mbar_init(bar(P_READY0 + s), 16);                  // one arrival per softmax warp of the pair
    }
    for (int s = 0; s < p.stages; ++s) { mbar_init(bar(FULL0 + s), 1); mbar_init(bar(EMPTY0 + s), 1); }
    fence_barrier_init();
    prefetch_tensormap(&map_q); prefetch_tensormap(&map_k); prefetch_tensormap(&map_v);
  }
  if (warp == 1) { tmem_alloc_2cta(smem_u32(&ctl->tmem_base), TMEM_COLS); tmem_relinquish_2cta(); }
  tc_fence_before();
  __syncthreads();
  cluster_sync_all();                                    // both CTAs' barriers exist before anyone signals across the pair
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&ctl->tmem_base);
  volatile int* abort_flag = &ctl->abort_flag;

  if (warp == 0) {
    // ================================================================ TMA producer: this CTA's part of every operand, counted on the leader's barrier
    if (lane == 0) {
      int s = 0;
      uint32_t ph = 0;
      auto stage = [&](int bytes) {                      // waits for a free stage and announces what both CTAs will put into it
        if (!mbar_wait(bar(EMPTY0 + s), ph ^ 1, abort_flag, p.status, ST_TIMEOUT_PRODUCER)) return false;
        if (rank == 0) mbar_arrive_expect_tx(bar(FULL0 + s), 2 * bytes);
        return true;
      };
      auto advance = [&]() { if (++s == p.stages) { s = 0; ph ^= 1; } };
      auto keys = [&](int kt) {                          // two boxes of the contraction per stage
        for (int j = 0; j < p.boxes; j += 2) {
          const int n = min(2, p.boxes - j);
          if (!stage(n * (p.resident ? KBOX : KBOX + QBOX))) return false;
          const uint32_t dst = sR + s * p.stage_bytes, fb = mapa_shared(bar(FULL0 + s), 0);
          for (int e = 0; e < n; ++e) {
            tma_load_3d_pair(dst + e * KBOX, &map_k, fb, (j + e) * 64, kt * 128 + (int)rank * 64, b);
            if (!p.resident) tma_load_3d_pair(dst + 2 * KBOX + e * QBOX, &map_q, fb, h * p.W + (j + e) * 64, q0, b);
          }
          advance();
        }
        return true;
      };
      int kt = seek(kt_lo);
      bool ok = kt < kt_hi;
      if (ok && p.resident) {
        if (rank == 0) mbar_arrive_expect_tx(bar(Q_FULL), 2 * p.boxes * QBOX);
        const uint32_t qb = mapa_shared(bar(Q_FULL), 0);
        for (int j = 0; j < p.boxes; ++j) tma_load_3d_pair(sQ + j * QBOX, &map_q, qb, h * p.W + j * 64, q0, b);
      }
      ok = ok && keys(kt);
      if (ok && seek(kt + 1) < kt_hi) ok = keys(seek(kt + 1));
      while (ok) {
        const int nx = seek(kt + 1);
        const int ahead = nx < kt_hi ? seek(nx + 1) : kt_hi;
        if (ahead < kt_hi && !keys(ahead)) break;
        if (!stage(VBOX)) break;
        tma_load_3d_pair(sR + s * p.stage_bytes, &map_v, mapa_shared(bar(FULL0 + s), 0), g * p.Dv + (int)rank * 64, kt * 128, b);
        advance();
        kt = nx;
        if (kt >= kt_hi) break;
      }
    }
  } else if (warp == 1) {
    // ================================================================ MMA issuer: the leader's warp walks together, one lane issues, so that
    // descriptors and loop state stay in uniform registers (a lone thread's arithmetic would be slower than the products)
    if (rank == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(256, 128, false, false), idesc_pv = make_idesc_bf16(256, 128, false, true);
      constexpr uint64_t KSTEP = 32 >> 4, VSTEP = 2048 >> 4;           // 16 lanes / 16 keys further, in descriptor units
      int n = 0;
      if (!mk.pos_k) n = kt_hi - kt_lo;
      else for (int kt = seek(kt_lo); kt < kt_hi; kt = seek(kt + 1)) ++n;
      n = __shfl_sync(0xffffffffu, n, 0);
      const uint32_t tm = __shfl_sync(0xffffffffu, tmem, 0);
      const uint64_t dq0 = make_smem_desc(sQ, 16, 1024), dk0 = make_smem_desc(sR, 16, 1024), dv0 = make_smem_desc(sR, VBOX, 1024);
      const bool elected = lane == 0;
      int s = 0;
      uint32_t ph = 0;
      auto wait = [&](int i, uint32_t parity) {
        const bool ok = __all_sync(0xffffffffu, mbar_wait(bar(i), parity, abort_flag, p.status, ST_TIMEOUT_MMA));
        tc_fence_after();
        return ok;
      };
      auto release = [&]() {
        if (elected) umma_commit_pair(bar(EMPTY0 + s));
        if (++s == p.stages) { s = 0; ph ^= 1; }
      };
      auto scores = [&](int buf) {                       // S of a tile
        const uint32_t d = tm + COL_S + buf * 128;
        for (int j = 0; j < p.boxes; j += 2) {
          if (!wait(FULL0 + s, ph)) return false;
          const uint64_t dk = dk0 + (uint64_t)((s * p.stage_bytes) >> 4), dq = p.resident ? dq0 + (uint64_t)(j * (QBOX >> 4)) : dk + (2 * KBOX >> 4);
          if (elected) {
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_f16_ss_2cta(d, dq + k * KSTEP, dk + k * KSTEP, idesc_qk, (j | k) != 0);
            if (j + 1 < p.boxes) {
#pragma unroll
              for (int k = 0; k < 4; ++k) umma_f16_ss_2cta(d, dq + (QBOX >> 4) + k * KSTEP, dk + (KBOX >> 4) + k * KSTEP, idesc_qk, 1);
            }
          }
          release();
        }
        if (elected) umma_commit_pair(bar(S_FULL0 + buf));
        return true;
      };
      bool ok = n > 0;
      if (ok && p.resident) ok = wait(Q_FULL, 0);
      ok = ok && scores(0);
      if (ok && n > 1) ok = scores(1);
      int buf = 0;                                       // of tile i
      uint32_t par = 0;
      for (int i = 0; i < n && ok; ++i) {
        if (i + 2 < n && !scores(buf == 0 ? 2 : buf - 1)) break;
        if (!wait(FULL0 + s, ph) || !wait(P_READY0 + buf, par)) break;
        const uint64_t dv = dv0 + (uint64_t)((s * p.stage_bytes) >> 4);
        const uint32_t tp = tm + COL_S + buf * 128;
        if (elected) {
#pragma unroll
          for (int k = 0; k < 8; ++k) umma_f16_ts_2cta(tm + COL_O, tp + k * 8, dv + k * VSTEP, idesc_pv, (i | k) != 0);
        }
        release();
        if (elected) umma_commit_pair(bar(PV_DONE0 + (i & 1)));
        if (++buf == 3) { buf = 0; par ^= 1; }
      }
    }
  } else {
    // ================================================================ softmax: warps 2..5 keys 0..63 of a tile, warps 6..9 keys 64..127
    const int half = (warp - 2) >> 2, qd = warp & 3;     // TMEM lane quarter this warp may touch
    const int row = qd * 32 + lane, wt = threadIdx.x - 64, qg = q0 + row;
    const uint32_t lane_off = (uint32_t)(qd * 32) << 16, tO = tmem + lane_off + COL_O + half * 64;
    const bool row_ok = row < t.rows, has_seg = mk.seg_q != nullptr, arrays = mk.pos_k != nullptr;
    const int qpos = mk.pos_q ? (row_ok ? mk.pos_q[(long)b * mk.Sq + qg] : 0) : qg + mk.q_off;
    const int my_seg = has_seg && row_ok ? mk.seg_q[(long)b * mk.Sq + qg] : 0;
    int lo_p, hi_p;
    attn::key_interval(mk, qpos, lo_p, hi_p);            // keys this row may attend to, as a closed position interval
    const uint32_t span = (uint32_t)hi_p - (uint32_t)lo_p;
    const bool none = hi_p < lo_p;
    const float a = p.scale * LOG2E;                     // scores in log2 units
    float m = -INFINITY, l = 0.f;                        // reference maximum; this half's part of the row sum
    int cnt = 0, buf = 0;
    uint32_t phase = 0;                                  // of the buffer of tile cnt
    bool ok = true;
    for (int kt = seek(kt_lo); kt < kt_hi; kt = seek(kt + 1), ++cnt) {
      const int par = cnt & 1, k0 = kt * 128 + half * 64;
      const bool masked = attn::classify(mk, t, attn::k_span(mk, b, kt)) != 1;
      const uint32_t tS = tmem + lane_off + COL_S + buf * 128;
      if (arrays || has_seg) {
        if (wt < 128) {
          const int kg = kt * 128 + wt;
          if (arrays) ctl->pos[par][wt] = kg < mk.Skv ? mk.pos_k[(long)b * mk.Skv + kg] : INT_MAX;
          if (has_seg) ctl->seg[par][wt] = kg < mk.Skv ? mk.seg_k[(long)b * mk.Skv + kg] : 0;
        }
        named_bar_sync(1, 256);
      }
      if (ok && !mbar_wait(bar(S_FULL0 + buf), phase, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) ok = false;
      tc_fence_after();
      uint32_t r0[32], r1[32];
      auto mask32 = [&](uint32_t (&r)[32], int c0) {
        if (arrays) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if ((uint32_t)ctl->pos[par][half * 64 + c0 + e] - (uint32_t)lo_p > span || none) r[e] = 0xff800000u;
        } else {
          const uint32_t e_lo = (uint32_t)lo_p - (uint32_t)(k0 + c0);
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if ((uint32_t)e - e_lo > span || none) r[e] = 0xff800000u;
        }
        if (has_seg) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (ctl->seg[par][half * 64 + c0 + e] != my_seg || my_seg == 0) r[e] = 0xff800000u;
        }
      };
      auto max32 = [](const uint32_t (&r)[32]) {
        float v0 = fmax3(__uint_as_float(r[0]), __uint_as_float(r[1]), __uint_as_float(r[2]));
        float v1 = fmax3(__uint_as_float(r[3]), __uint_as_float(r[4]), __uint_as_float(r[5]));
#pragma unroll
        for (int e = 6; e < 30; e += 4) {
          v0 = fmax3(v0, __uint_as_float(r[e]), __uint_as_float(r[e + 1]));
          v1 = fmax3(v1, __uint_as_float(r[e + 2]), __uint_as_float(r[e + 3]));
        }
        return fmax3(v0, v1, fmaxf(__uint_as_float(r[30]), __uint_as_float(r[31])));
      };
      tmem_ld_32x32b_x32(tS + half * 64, r0);
      tmem_ld_32x32b_x32(tS + half * 64 + 32, r1);
      tmem_ld_wait_dep(r0);
      tmem_ld_wait_dep(r1);
      if (masked) { mask32(r0, 0); mask32(r1, 32); }
      ctl->top[par][half][row] = fmaxf(max32(r0), max32(r1));
      named_bar_sync(2, 256);                    // every score of the tile has been read, too
      const float tm = a * fmaxf(ctl->top[par][0][row], ctl->top[par][1][row]);            // -inf when the whole row is masked
      const bool grow = tm > m + RESCALE_THRESHOLD;
      if (__any_sync(0xffffffffu, grow)) {
        const float alpha = grow ? fast_exp2(m - tm) : 1.f;
        if (cnt > 0) {
          // O may only be touched once the previous P V product has retired (the scores of this tile follow the one before that); each half scales
          // its columns
          if (ok && !mbar_wait(bar(PV_DONE0 + (par ^ 1)), ((cnt - 1) >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) ok = false;
          __syncwarp();
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < 64; c += 16) {
            uint32_t o[16];
            tmem_ld_32x32b_x16(tO + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) asm volatile("" : "+r"(o[e]));
#pragma unroll
            for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
            tmem_st_32x32b_x16(tO + c, o);
          }
        }
        if (grow) { l *= alpha; m = tm; }
      }
      const float neg = (m == -INFINITY) ? 0.f : -m;
      const float2 a2 = make_float2(a, a), neg2 = make_float2(neg, neg);
      float2 rsa = make_float2(0.f, 0.f), rsb = make_float2(0.f, 0.f);
      auto exps = [&](uint32_t (&r)[32], int c) {        // probabilities of 32 keys, written over the tile's scores
        uint32_t pk[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float2 x = __ffma2_rn(make_float2(__uint_as_float(r[2 * e]), __uint_as_float(r[2 * e + 1])), a2, neg2);
          const float2 pp = make_float2(fast_exp2(x.x), fast_exp2(x.y));
          if (e & 1) rsb = __fadd2_rn(rsb, pp); else rsa = __fadd2_rn(rsa, pp);
          pk[e] = pack_bf16(pp.x, pp.y);
        }
        tmem_st_32x32b_x16(tS + half * 32 + c * 16, pk);
      };
      exps(r0, 0);
      exps(r1, 1);
      l += (rsa.x + rsa.y) + (rsb.x + rsb.y);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive_cluster_tmem(mapa_shared(bar(P_READY0 + buf), 0));
      if (++buf == 3) { buf = 0; phase ^= 1; }
    }
    // ---------------------------------------------------------------- epilogue: each half stores its columns
    if (ok && cnt > 0 && !mbar_wait(bar(PV_DONE0 + ((cnt - 1) & 1)), ((cnt - 1) >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) ok = false;
    __syncwarp();
    tc_fence_after();
    named_bar_sync(2, 256);                              // the last maxima have been read
    ctl->top[0][half][row] = l;
    named_bar_sync(2, 256);
    l = ctl->top[0][0][row] + ctl->top[0][1][row];
    if (p.sinks) {
      const float sk = __bfloat162float(p.sinks[h]) * LOG2E;
      if (m == -INFINITY) l = 1.f; else l += fast_exp2(sk - m);
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    __nv_bfloat16* dst = p.out + (((long)b * mk.Sq + qg) * p.H + h) * p.Dv + half * 64;
#pragma unroll 1
    for (int c = 0; c < 2; ++c) {
      uint32_t r[32];
      if (cnt > 0) {
        tmem_ld_32x32b_x32(tO + c * 32, r);
        tmem_ld_wait_dep(r);
      } else {
#pragma unroll
        for (int e = 0; e < 32; ++e) r[e] = 0u;
      }
      if (row_ok && ok) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (half * 64 + c * 32 + j * 8 >= p.Dv) continue;
          uint4 o4;
          o4.x = pack_bf16(__uint_as_float(r[8 * j]) * inv, __uint_as_float(r[8 * j + 1]) * inv);
          o4.y = pack_bf16(__uint_as_float(r[8 * j + 2]) * inv, __uint_as_float(r[8 * j + 3]) * inv);
          o4.z = pack_bf16(__uint_as_float(r[8 * j + 4]) * inv, __uint_as_float(r[8 * j + 5]) * inv);
          o4.w = pack_bf16(__uint_as_float(r[8 * j + 6]) * inv, __uint_as_float(r[8 * j + 7]) * inv);
          *reinterpret_cast<uint4*>(dst + c * 32 + j * 8) = o4;
        }
      }
      __syncwarp();
    }
  }
  if (*abort_flag) { const uint64_t w0 = globaltimer_ns(); while (globaltimer_ns() - w0 < 200000ull) { } }
  tc_fence_before();
  __syncthreads();
  cluster_sync_all();                                    // the peer may still read this CTA's shared memory / signal its barriers
  if (warp == 1) { tc_fence_after(); tmem_dealloc_2cta(tmem, TMEM_COLS); }
}

// ================================================================================================ host
typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeFn encode_fn() {
  static EncodeFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || !ptr) return nullptr;
    fn = reinterpret_cast<EncodeFn>(ptr);
  }
  return fn;
}

// {cols, tokens, batch} view with row stride `ld` and batch stride `bs` (elements); box {64 columns, `rows` rows, 1}
static int box_map(CUtensorMap* m, const void* ptr, long batch, long tokens, long cols, long ld, long bs, int rows) {
  EncodeFn enc = encode_fn();
  if (!enc) return -1;
  if (batch == 1) bs = tokens * ld;      // a one-batch view may carry any batch stride
  cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)tokens, (cuuint64_t)batch};
  cuuint64_t strides[2] = {(cuuint64_t)ld * 2, (cuuint64_t)bs * 2};
  cuuint32_t box[3] = {64, (cuuint32_t)rows, 1}, es[3] = {1, 1, 1};
  CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : (int)r;
}

}  // namespace wide
}  // namespace mt

extern "C" {
void mt_attn_tile_minmax(const int* pos, int B, int S, int* out, cudaStream_t st);

// q [B, Sq, H, G * D] dense, k / v views of rows with strides ld* and batch strides bs* (elements), out [B, Sq, H, Dv] dense. D and Dv multiples of 8,
// Dv <= 128, scale > 0. seg_q / seg_k, pos_q / pos_k (with `tiles`) and sinks may be null. Causal.
int mt_wide_flash(const void* q, const void* k, const void* v, void* out, const int* seg_q, const int* seg_k, const int* pos_q, const int* pos_k, int* tiles,
                  const void* sinks, int B, int Sq, int Skv, int H, int G, int D, int Dv, long ldk, long bsk, long ldv, long bsv, float scale, int window,
                  int chunk, int q_off, int* status, cudaStream_t st) {
  using namespace mt::wide;
  if (B < 1 || Sq < 1 || Skv < 1 || H % G || D % 8 || Dv % 8 || Dv > 128 || !(scale > 0.f) || (pos_q == nullptr) != (pos_k == nullptr) ||
      (seg_q == nullptr) != (seg_k == nullptr) || (pos_q && !tiles))
    return -1;
  Params p{};
  p.B = B; p.H = H; p.G = G; p.Dv = Dv; p.W = G * D;
  p.boxes = (p.W + 63) / 64;
  p.resident = p.boxes <= RESIDENT_MAX;
  p.stage_bytes = p.resident ? VBOX : 2 * (KBOX + QBOX);
  const int fixed = 1024 + (int)sizeof(Ctl), held = p.resident ? p.boxes * QBOX : 0;
  p.stages = (227 * 1024 - fixed - held) / p.stage_bytes;
  if (p.stages > STAGES_MAX) p.stages = STAGES_MAX;
  const int smem = fixed + held + p.stages * p.stage_bytes;
  CUtensorMap mq, mk, mv;
  if (box_map(&mq, q, B, Sq, (long)H * p.W, (long)H * p.W, (long)Sq * H * p.W, 128) || box_map(&mk, k, B, Skv, p.W, ldk, bsk, 64) ||
      box_map(&mv, v, B, Skv, (long)G * Dv, ldv, bsv, 128))
    return -3;
  p.n_pairs = (Sq + 255) / 256;
  p.scale = scale; p.sinks = static_cast<const __nv_bfloat16*>(sinks); p.out = static_cast<__nv_bfloat16*>(out); p.status = status;
  mt::attn::Mask& msk = p.mk;
  msk.Sq = Sq; msk.Skv = Skv; msk.n_qt = (Sq + 127) / 128; msk.n_kt = (Skv + 127) / 128;
  msk.q_off = q_off; msk.causal = 1; msk.window = window; msk.chunk = chunk;
  msk.seg_q = seg_q; msk.seg_k = seg_k; msk.pos_q = pos_q; msk.pos_k = pos_k;
  if (pos_q) {
    mt_attn_tile_minmax(pos_q, B, Sq, tiles, st);
    mt_attn_tile_minmax(pos_k, B, Skv, tiles + 2l * B * msk.n_qt, st);
    msk.tile_q = tiles;
    msk.tile_k = tiles + 2l * B * msk.n_qt;
  }
  if (cudaFuncSetAttribute(wide_flash_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  wide_flash_kernel<<<(unsigned)(2l * p.n_pairs * H * B), 320, smem, st>>>(mq, mk, mv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // extern "C"
