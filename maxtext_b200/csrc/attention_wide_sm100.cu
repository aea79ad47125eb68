// Flash attention forward for wide queries on tcgen05 / TMEM: every query head meets ONE key made of all key heads side by side, and the values
// of its own group. That is what attention becomes when the heads' scores are mixed by a matrix before the softmax, s_h <- sum_g T[h, g] s_g: by
// linearity the mixing moves to the queries (qkv_prep), q_h . k -> [.., sum of T[h, g] q_g over the query heads g of key head c, ..] . [.., k_c, ..].
//
// q [B, Sq, H, W], k [B, Skv, W] (W = G * D, any multiple of 8), v [B, Skv, G * Dv], out [B, Sq, H, Dv]; bf16 in / out, fp32 scores and statistics.
//
// CTA = 128 queries of one head, 192 threads:
//   warp 0      TMA producer
//   warp 1      MMA issuer / TMEM owner
//   warps 2..5  softmax, one thread per query row
// The contraction W passes in boxes of 64 lanes, [128 rows x 64] bf16 with 128-byte swizzle, through a ring that keys and values share. The query's
// boxes stay in shared memory when they fit (W <= 512) and pass through the ring next to the keys' otherwise. W is several times the head width, so
// the score products of the next key tile are long enough to cover the softmax of the current one: S is double buffered in tensor memory,
//   S(0), [S(1), P(0) V], [S(2), P(1) V], ...
// and the tensor core never waits for a second query tile. P overwrites its own S as the TMEM operand, in halves of 64 keys. Masks, the lazy
// rescaling and the bounded waits are those of attention_fwd_sm100.cu. Boxes that reach into a neighbour head's columns meet zero-filled lanes of the
// other operand (keys), or fill accumulator columns that are not stored (values).
#include "attention_mask.cuh"
#include "sm100_ptx.cuh"
#include <cuda_bf16.h>

namespace mt {
namespace wide {

constexpr float LOG2E = 1.4426950408889634f;
constexpr float RESCALE_THRESHOLD = 8.f;     // log2 units
constexpr int BOX = 128 * 64 * 2;            // bytes of a box
constexpr int STAGES_MAX = 12, RESIDENT_MAX = 8;

struct Params {
  int B, H, G, Dv, W;
  int boxes;             // of the contraction: ceil(W / 64)
  int resident, stages, stage_bytes;
  int n_qt;
  attn::Mask mk;
  float scale;
  const __nv_bfloat16* sinks;    // [H] or nullptr
  __nv_bfloat16* out;
  int* status;
};

struct alignas(8) Ctl {
  uint64_t bars[8 + 2 * STAGES_MAX];
  uint32_t tmem_base;
  int abort_flag;
  int pad[2];
};

__device__ __forceinline__ uint64_t kmajor(uint32_t box, int k) { return make_smem_desc(box + k * 32, 16, 1024); }
__device__ __forceinline__ uint64_t mnmajor(uint32_t box, int k) { return make_smem_desc(box + k * 2048, BOX, 1024); }

template <int NV>                            // boxes of the value width
__global__ void __launch_bounds__(192, 1)
wide_flash_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                  const __grid_constant__ Params p) {
  constexpr uint32_t TMEM_COLS = 512, COL_S = 0, COL_O = 256;        // S of a tile at (its parity) * 128
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sQ = base, sR = base + (p.resident ? p.boxes * BOX : 0);
  Ctl* ctl = reinterpret_cast<Ctl*>(smem_raw + (sR - smem_u32(smem_raw)) + p.stages * p.stage_bytes);
  int* sk_pos = reinterpret_cast<int*>(ctl + 1);         // [parity][128]
  int* sk_seg = sk_pos + 2 * 128;
  const uint32_t bar0 = smem_u32(&ctl->bars[0]);
  enum { Q_FULL = 0, S_FULL0 = 1, PA_READY0 = 3, PB_READY0 = 5, PV_DONE = 7, FULL0 = 8, EMPTY0 = 8 + STAGES_MAX };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hb = p.H * p.B;
  const int qi = p.n_qt - 1 - (int)(blockIdx.x / hb);    // the last queries see the most keys: they come first
  const int h = (int)(blockIdx.x % hb) % p.H, b = (int)(blockIdx.x % hb) / p.H, g = h / (p.H / p.G);
  const attn::Mask& mk = p.mk;
  const attn::Span t = attn::q_span(mk, b, qi);
  const int q0 = qi * 128;
  int kt_lo, kt_hi;
  attn::k_tiles_for(mk, t, kt_lo, kt_hi);
  // the next key tile from kt on that holds a visible key, or kt_hi: every role walks the same tiles
  auto seek = [&](int kt) {
    while (kt < kt_hi && attn::classify(mk, t, attn::k_span(mk, b, kt)) == 0) ++kt;
    return kt;
  };

  if (threadIdx.x == 0) {
    ctl->abort_flag = 0;
    mbar_init(bar(Q_FULL), 1);
    mbar_init(bar(PV_DONE), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar(S_FULL0 + s), 1);
      mbar_init(bar(PA_READY0 + s), 4); mbar_init(bar(PB_READY0 + s), 4);            // one arrival per softmax warp
    }
    for (int s = 0; s < p.stages; ++s) { mbar_init(bar(FULL0 + s), 1); mbar_init(bar(EMPTY0 + s), 1); }
    fence_barrier_init();
    prefetch_tensormap(&map_q); prefetch_tensormap(&map_k); prefetch_tensormap(&map_v);
  }
  if (warp == 1) { tmem_alloc(smem_u32(&ctl->tmem_base), TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&ctl->tmem_base);
  volatile int* abort_flag = &ctl->abort_flag;

  if (warp == 0) {
    // ================================================================ TMA producer
    if (lane == 0) {
      int s = 0;
      uint32_t ph = 0;
      auto stage = [&](int bytes) {                      // waits for a free stage and announces what will land in it
        if (!mbar_wait(bar(EMPTY0 + s), ph ^ 1, abort_flag, p.status, ST_TIMEOUT_PRODUCER)) return false;
        mbar_arrive_expect_tx(bar(FULL0 + s), bytes);
        return true;
      };
      auto advance = [&]() { if (++s == p.stages) { s = 0; ph ^= 1; } };
      auto keys = [&](int kt) {
        for (int j = 0; j < p.boxes; ++j) {
          if (!stage(p.resident ? BOX : 2 * BOX)) return false;
          const uint32_t dst = sR + s * p.stage_bytes;
          tma_load_3d(dst, &map_k, bar(FULL0 + s), j * 64, kt * 128, b);
          if (!p.resident) tma_load_3d(dst + BOX, &map_q, bar(FULL0 + s), h * p.W + j * 64, q0, b);
          advance();
        }
        return true;
      };
      int kt = seek(kt_lo);
      bool ok = kt < kt_hi;
      if (ok && p.resident) {
        mbar_arrive_expect_tx(bar(Q_FULL), p.boxes * BOX);
        for (int j = 0; j < p.boxes; ++j) tma_load_3d(sQ + j * BOX, &map_q, bar(Q_FULL), h * p.W + j * 64, q0, b);
      }
      ok = ok && keys(kt);
      while (ok) {
        const int nx = seek(kt + 1);
        if (nx < kt_hi) ok = keys(nx);
        for (int j = 0; j < NV && ok; ++j) {
          ok = stage(BOX);
          if (ok) {
            tma_load_3d(sR + s * p.stage_bytes, &map_v, bar(FULL0 + s), g * p.Dv + j * 64, kt * 128, b);
            advance();
          }
        }
        kt = nx;
        if (kt >= kt_hi) break;
      }
    }
  } else if (warp == 1) {
    // ================================================================ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, 64, false, true);
      int s = 0;
      uint32_t ph = 0;
      auto landed = [&]() {
        if (!mbar_wait(bar(FULL0 + s), ph, abort_flag, p.status, ST_TIMEOUT_MMA)) return false;
        tc_fence_after();
        return true;
      };
      auto release = [&]() {
        umma_commit(bar(EMPTY0 + s));
        if (++s == p.stages) { s = 0; ph ^= 1; }
      };
      auto scores = [&](int i) {                         // S of the i-th tile
        for (int j = 0; j < p.boxes; ++j) {
          if (!landed()) return false;
          const uint32_t kb = sR + s * p.stage_bytes, qb = p.resident ? sQ + j * BOX : kb + BOX;
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ss(tmem + COL_S + (i & 1) * 128, kmajor(qb, k), kmajor(kb, k), idesc_qk, (j | k) != 0);
          release();
        }
        umma_commit(bar(S_FULL0 + (i & 1)));
        return true;
      };
      int kt = seek(kt_lo), i = 0;
      bool ok = kt < kt_hi;
      if (ok && p.resident) ok = mbar_wait(bar(Q_FULL), 0, abort_flag, p.status, ST_TIMEOUT_MMA);
      ok = ok && scores(0);
      while (ok) {
        const int nx = seek(kt + 1);
        if (nx < kt_hi && !(ok = scores(i + 1))) break;
        const uint32_t tp = tmem + COL_S + (i & 1) * 128, par = (i >> 1) & 1;
        for (int j = 0; j < NV && ok; ++j) {
          if (!(ok = landed())) break;
          const uint32_t vb = sR + s * p.stage_bytes;
          // the probabilities arrive in two halves of 64 keys; the product starts on the first while the second is computed
          if (j == 0 && !(ok = mbar_wait(bar(PA_READY0 + (i & 1)), par, abort_flag, p.status, ST_TIMEOUT_MMA))) break;
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ts(tmem + COL_O + j * 64, tp + k * 8, mnmajor(vb, k), idesc_pv, (i | k) != 0);
          if (j == 0 && !(ok = mbar_wait(bar(PB_READY0 + (i & 1)), par, abort_flag, p.status, ST_TIMEOUT_MMA))) break;
          tc_fence_after();
#pragma unroll
          for (int k = 4; k < 8; ++k) umma_f16_ts(tmem + COL_O + j * 64, tp + k * 8, mnmajor(vb, k), idesc_pv, 1);
          release();
        }
        if (!ok) break;
        umma_commit(bar(PV_DONE));
        kt = nx;
        ++i;
        if (kt >= kt_hi) break;
      }
    }
  } else {
    // ================================================================ softmax
    const int qd = warp & 3;                             // TMEM lane quarter this warp may touch
    const int row = qd * 32 + lane, wt = threadIdx.x - 64, qg = q0 + row;
    const uint32_t lane_off = (uint32_t)(qd * 32) << 16, tO = tmem + lane_off + COL_O;
    const bool row_ok = row < t.rows, has_seg = mk.seg_q != nullptr, arrays = mk.pos_k != nullptr;
    const int qpos = mk.pos_q ? (row_ok ? mk.pos_q[(long)b * mk.Sq + qg] : 0) : qg + mk.q_off;
    const int my_seg = has_seg && row_ok ? mk.seg_q[(long)b * mk.Sq + qg] : 0;
    int lo_p, hi_p;
    attn::key_interval(mk, qpos, lo_p, hi_p);            // keys this row may attend to, as a closed position interval
    const uint32_t span = (uint32_t)hi_p - (uint32_t)lo_p;
    const bool none = hi_p < lo_p;
    const float a = p.scale * LOG2E;                     // scores in log2 units
    float m = -INFINITY, l = 0.f;                        // reference maximum and row sum
    int cnt = 0;
    bool ok = true;
    for (int kt = seek(kt_lo); kt < kt_hi; kt = seek(kt + 1), ++cnt) {
      const int par = cnt & 1, k0 = kt * 128;
      const bool masked = attn::classify(mk, t, attn::k_span(mk, b, kt)) == 2;
      const uint32_t tS = tmem + lane_off + COL_S + par * 128;
      if (arrays || has_seg) {
        if (masked) {
          const int kg = k0 + wt;
          if (arrays) sk_pos[par * 128 + wt] = kg < mk.Skv ? mk.pos_k[(long)b * mk.Skv + kg] : INT_MAX;
          if (has_seg) sk_seg[par * 128 + wt] = kg < mk.Skv ? mk.seg_k[(long)b * mk.Skv + kg] : 0;
        }
        named_bar_sync(1, 128);                          // on every tile: a warp may not run two tiles ahead of the tables' readers
      }
      if (ok && !mbar_wait(bar(S_FULL0 + par), (cnt >> 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) ok = false;
      if (!ok) continue;
      tc_fence_after();
      auto mask32 = [&](uint32_t (&r)[32], int c0) {
        if (!masked) return;
        if (arrays) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if ((uint32_t)sk_pos[par * 128 + c0 + e] - (uint32_t)lo_p > span || none) r[e] = 0xff800000u;
        } else {
          const uint32_t e_lo = (uint32_t)lo_p - (uint32_t)(k0 + c0);
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if ((uint32_t)e - e_lo > span || none) r[e] = 0xff800000u;
        }
        if (has_seg) {
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (sk_seg[par * 128 + c0 + e] != my_seg || my_seg == 0) r[e] = 0xff800000u;
        }
      };
      // first pass: the row's maximum; the loads run one 32-column chunk ahead of the arithmetic
      float top = -INFINITY;
      uint32_t r0[32], r1[32];
      auto scan = [&](uint32_t (&r)[32], int c0) {
        mask32(r, c0);
        float v0 = -INFINITY, v1 = -INFINITY;
#pragma unroll
        for (int e = 0; e < 32; e += 2) { v0 = fmaxf(v0, __uint_as_float(r[e])); v1 = fmaxf(v1, __uint_as_float(r[e + 1])); }
        top = fmaxf(top, fmaxf(v0, v1));
      };
      tmem_ld_32x32b_x32(tS, r0);
      tmem_ld_wait_dep(r0);
      tmem_ld_32x32b_x32(tS + 32, r1);
      scan(r0, 0);
      tmem_ld_wait_dep(r1);
      tmem_ld_32x32b_x32(tS + 64, r0);
      scan(r1, 32);
      tmem_ld_wait_dep(r0);
      tmem_ld_32x32b_x32(tS + 96, r1);
      scan(r0, 64);
      tmem_ld_wait_dep(r1);
      tmem_ld_32x32b_x32(tS, r0);                // first chunk of the second pass
      scan(r1, 96);
      const float tm = a * top;                  // -inf when the whole row is masked
      const bool grow = tm > m + RESCALE_THRESHOLD;
      if (__any_sync(0xffffffffu, grow)) {
        const float alpha = grow ? fast_exp2(m - tm) : 1.f;
        if (cnt > 0) {
          // O may only be touched once the previous P V product has retired
          if (!mbar_wait(bar(PV_DONE), (cnt - 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) { ok = false; continue; }
          tc_fence_after();
          tmem_ld_wait_dep(r0);
#pragma unroll 1
          for (int c = 0; c < NV * 2; ++c) {
            tmem_ld_32x32b_x32(tO + c * 32, r1);
            tmem_ld_wait_dep(r1);
#pragma unroll
            for (int e = 0; e < 32; ++e) r1[e] = __float_as_uint(__uint_as_float(r1[e]) * alpha);
            tmem_st_32x32b_x32(tO + c * 32, r1);
          }
        }
        if (grow) { l *= alpha; m = tm; }
      }
      const float neg = (m == -INFINITY) ? 0.f : -m;
      const float2 a2 = make_float2(a, a), neg2 = make_float2(neg, neg);
      float2 rsa = make_float2(0.f, 0.f), rsb = make_float2(0.f, 0.f);
      // probabilities, written over the row's own (already read) score columns
      auto exps = [&](uint32_t (&r)[32], int c) {
        mask32(r, c * 32);
        uint32_t pk[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float2 x = __ffma2_rn(make_float2(__uint_as_float(r[2 * e]), __uint_as_float(r[2 * e + 1])), a2, neg2);
          const float2 pp = make_float2(fast_exp2(x.x), fast_exp2(x.y));
          if (e & 1) rsb = __fadd2_rn(rsb, pp); else rsa = __fadd2_rn(rsa, pp);
          pk[e] = pack_bf16(pp.x, pp.y);
        }
        tmem_st_32x32b_x16(tS + c * 16, pk);
      };
      auto announce = [&](int which) {
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar(which + par));
      };
      tmem_ld_wait_dep(r0);
      tmem_ld_32x32b_x32(tS + 32, r1);
      exps(r0, 0);
      tmem_ld_wait_dep(r1);
      tmem_ld_32x32b_x32(tS + 64, r0);
      exps(r1, 1);
      tmem_ld_wait_dep(r0);
      tmem_ld_32x32b_x32(tS + 96, r1);
      announce(PA_READY0);
      exps(r0, 2);
      tmem_ld_wait_dep(r1);
      exps(r1, 3);
      l += (rsa.x + rsa.y) + (rsb.x + rsb.y);
      announce(PB_READY0);
    }
    // ---------------------------------------------------------------- epilogue
    if (ok && cnt > 0 && !mbar_wait(bar(PV_DONE), (cnt - 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPILOGUE)) ok = false;
    if (ok) {
      tc_fence_after();
      if (p.sinks) {
        const float sk = __bfloat162float(p.sinks[h]) * LOG2E;
        if (m == -INFINITY) l = 1.f; else l += fast_exp2(sk - m);
      }
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* dst = p.out + (((long)b * mk.Sq + qg) * p.H + h) * p.Dv;
#pragma unroll 1
      for (int c = 0; c < NV * 2; ++c) {
        uint32_t r[32];
        if (cnt > 0) {
          tmem_ld_32x32b_x32(tO + c * 32, r);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int e = 0; e < 32; ++e) r[e] = 0u;
        }
        if (!row_ok) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (c * 32 + j * 8 >= p.Dv) continue;
          uint4 o4;
          o4.x = pack_bf16(__uint_as_float(r[8 * j]) * inv, __uint_as_float(r[8 * j + 1]) * inv);
          o4.y = pack_bf16(__uint_as_float(r[8 * j + 2]) * inv, __uint_as_float(r[8 * j + 3]) * inv);
          o4.z = pack_bf16(__uint_as_float(r[8 * j + 4]) * inv, __uint_as_float(r[8 * j + 5]) * inv);
          o4.w = pack_bf16(__uint_as_float(r[8 * j + 6]) * inv, __uint_as_float(r[8 * j + 7]) * inv);
          *reinterpret_cast<uint4*>(dst + c * 32 + j * 8) = o4;
        }
      }
    }
  }
  if (*abort_flag) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 200000ull) { } }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem, TMEM_COLS); }
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

// {cols, tokens, batch} view with row stride `ld` and batch stride `bs` (elements); box {64 columns, 128 rows, 1}
static int box_map(CUtensorMap* m, const void* ptr, long batch, long tokens, long cols, long ld, long bs) {
  EncodeFn enc = encode_fn();
  if (!enc) return -1;
  if (batch == 1) bs = tokens * ld;      // a one-batch view may carry any batch stride
  cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)tokens, (cuuint64_t)batch};
  cuuint64_t strides[2] = {(cuuint64_t)ld * 2, (cuuint64_t)bs * 2};
  cuuint32_t box[3] = {64, 128, 1}, es[3] = {1, 1, 1};
  CUresult r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : (int)r;
}

template <int NV>
static int run(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const Params& p, int smem, cudaStream_t st) {
  if (cudaFuncSetAttribute(wide_flash_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -2;
  wide_flash_kernel<NV><<<(unsigned)((long)p.n_qt * p.H * p.B), 192, smem, st>>>(mq, mk, mv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace wide
}  // namespace mt

extern "C" {
void mt_attn_tile_minmax(const int* pos, int B, int S, int* out, cudaStream_t st);

// q [B, Sq, H, G * D] dense, k / v views of rows with strides ld* and batch strides bs* (elements), out [B, Sq, H, Dv] dense. D and Dv multiples of 8,
// Dv <= 128, scale >= 0. seg_q / seg_k, pos_q / pos_k (with `tiles`) and sinks may be null. Causal.
int mt_wide_flash(const void* q, const void* k, const void* v, void* out, const int* seg_q, const int* seg_k, const int* pos_q, const int* pos_k, int* tiles,
                  const void* sinks, int B, int Sq, int Skv, int H, int G, int D, int Dv, long ldk, long bsk, long ldv, long bsv, float scale, int window,
                  int chunk, int q_off, int* status, cudaStream_t st) {
  using namespace mt::wide;
  if (B < 1 || Sq < 1 || Skv < 1 || H % G || D % 8 || Dv % 8 || Dv > 128 || scale < 0.f || (pos_q == nullptr) != (pos_k == nullptr) ||
      (seg_q == nullptr) != (seg_k == nullptr) || (pos_q && !tiles))
    return -1;
  Params p{};
  p.B = B; p.H = H; p.G = G; p.Dv = Dv; p.W = G * D;
  p.boxes = (p.W + 63) / 64;
  p.resident = p.boxes <= RESIDENT_MAX;
  p.stage_bytes = p.resident ? BOX : 2 * BOX;
  const int fixed = 1024 + (int)sizeof(Ctl) + 4 * 128 * 4, room = 227 * 1024 - fixed - (p.resident ? p.boxes * BOX : 0);
  p.stages = room / p.stage_bytes;
  if (p.stages > STAGES_MAX) p.stages = STAGES_MAX;
  const int smem = fixed + (p.resident ? p.boxes * BOX : 0) + p.stages * p.stage_bytes;
  CUtensorMap mq, mk, mv;
  if (box_map(&mq, q, B, Sq, (long)H * p.W, (long)H * p.W, (long)Sq * H * p.W) || box_map(&mk, k, B, Skv, p.W, ldk, bsk) ||
      box_map(&mv, v, B, Skv, (long)G * Dv, ldv, bsv))
    return -3;
  p.n_qt = (Sq + 127) / 128;
  p.scale = scale; p.sinks = static_cast<const __nv_bfloat16*>(sinks); p.out = static_cast<__nv_bfloat16*>(out); p.status = status;
  mt::attn::Mask& msk = p.mk;
  msk.Sq = Sq; msk.Skv = Skv; msk.n_qt = p.n_qt; msk.n_kt = (Skv + 127) / 128;
  msk.q_off = q_off; msk.causal = 1; msk.window = window; msk.chunk = chunk;
  msk.seg_q = seg_q; msk.seg_k = seg_k; msk.pos_q = pos_q; msk.pos_k = pos_k;
  if (pos_q) {
    mt_attn_tile_minmax(pos_q, B, Sq, tiles, st);
    mt_attn_tile_minmax(pos_k, B, Skv, tiles + 2l * B * msk.n_qt, st);
    msk.tile_q = tiles;
    msk.tile_k = tiles + 2l * B * msk.n_qt;
  }
  return Dv <= 64 ? run<1>(mq, mk, mv, p, smem, st) : run<2>(mq, mk, mv, p, smem, st);
}

}  // extern "C"
