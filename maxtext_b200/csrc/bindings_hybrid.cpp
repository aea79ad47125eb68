// Bindings of the inference kernels for several residual streams, selective scans, attention over a key/value cache and routed experts with
// scaled inputs. Every entry checks types, layouts and sizes before it launches; pointers handed to the kernels are in bounds for the sizes
// given with them.
#include <torch/extension.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <cuda_runtime.h>
#include "cached_attention.h"

extern "C" {
int mt_stream_mix(float* x, int k, const void* branch, const int* dest, int per_token, const void* mix, const void* write, const void* read, const void* w,
                  const void* b, void* y, int f32, long rows, int D, float eps, cudaStream_t st);
int mt_ssm_conv(int f32, const void* x, long ldx, const void* w, const void* bias, int taps, int C, int S, float* hist, const int64_t* slots,
                const int64_t* lengths, const int64_t* new_lens, void* y, int B, cudaStream_t st);
int mt_ssm_scan(int f32, const void* x, const void* z, long ldz, const void* q, long ldq, int off, const float* dt, const void* dt_bias, const void* A_log,
                const void* D, int C, int N, int S, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* y, int B,
                cudaStream_t st);
int mt_qkv_prep(int f32, const mt::cattn::PrepArgs* a, long N, cudaStream_t st);
int mt_cached_decode(const void* q, const void* k, const void* v, const int64_t* slots, const int64_t* lengths, long max_len, int B, int H, int G, int D, int Dv,
                     float scale, float cap, int window, int chunk, const void* sinks, const void* gate, long ldg, int per_head,
                     const mt::cattn::DiffArgs* diff, int splits, float* part, float* ml, void* out, cudaStream_t st);
int mt_cached_attention(int f32, const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S, int H,
                        int G, int D, int Dv, float scale, float cap, int window, int chunk, const void* sinks, void* out, cudaStream_t st);
int mt_wide_decode(const void* q, const void* k, const void* v, const int64_t* slots, const int64_t* lengths, long max_len, int B, int H, int G, int D, int Dv,
                   float scale, int window, int chunk, const void* sinks, int splits, float* part, float* ml, void* out, cudaStream_t st);
int mt_wide_attention(int f32, const void* q, const void* k, const void* v, long max_len, const int64_t* slots, const int64_t* lengths, int B, int S, int H, int G,
                      int D, int Dv, float scale, int window, int chunk, const void* sinks, void* out, cudaStream_t st);
int mt_wide_flash(const void* q, const void* k, const void* v, void* out, const int* seg_q, const int* seg_k, const int* pos_q, const int* pos_k, int* tiles,
                  const void* sinks, int B, int Sq, int Skv, int H, int G, int D, int Dv, long ldk, long bsk, long ldv, long bsv, float scale, int window,
                  int chunk, int q_off, int* status, cudaStream_t st);
long mt_attn_tile_ints(int B, int Sq, int Skv);
int mt_head_gate(int f32, const void* o, int dvp, const void* g, long ldg, long rows, int HD, int Dv, int per_head, void* out, int sms, cudaStream_t st);
int mt_diff_combine(int f32, const void* o, int dvp, const mt::cattn::DiffArgs* a, long N, int H, int Dv, const void* gate, long ldg, int per_head, void* out,
                    int sms, cudaStream_t st);
int mt_expert_up(int f32, const void* x, const void* w0, const void* w1, const float* wts, const int* idx, const int* sizes, const int* offs,
                 const int* row_pair, int n, int k, int E, int F, int D, float limit, void* h, int sms, cudaStream_t st);
int mt_expert_down(int f32, const void* h, const void* w, const int* idx, const int* sizes, const int* offs, const int* row_pair, int n, int E, int D, int F,
                   void* y, int sms, cudaStream_t st);
int mt_expert_act(const void* gu, int gated, const float* wts, const int* row_pair, const int* offs, int E, int F, float limit, void* h, int rows_max, int sms,
                  cudaStream_t st);
}

void mt_count_launches(int n); // defined in bindings.cpp
int mt_num_sms();              // defined in bindings.cpp
int* mt_status_ptr();          // defined in bindings.cpp

namespace {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

cudaStream_t stream() { return at::cuda::getCurrentCUDAStream().stream(); }

void done(int rc, const char* what, int launches = 1) {
  TORCH_CHECK(rc == 0, what, " failed with code ", rc);
  mt_count_launches(launches);
}
bool f32(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == torch::kFloat32 || t.scalar_type() == torch::kBFloat16), "bf16 or fp32 CUDA tensor expected");
  return t.scalar_type() == torch::kFloat32;
}
void same(const Tensor& t, const Tensor& like, int64_t numel, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == like.scalar_type() && t.is_contiguous() && t.numel() == numel, what, ": contiguous tensor of ", numel,
              " elements of the compute type expected");
}
const void* same(const OptTensor& t, const Tensor& like, int64_t numel, const char* what) {
  if (!t) return nullptr;
  same(*t, like, numel, what);
  return t->data_ptr();
}
void rows2d(const Tensor& t, const Tensor& like, int64_t n, int64_t cols, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == like.scalar_type() && t.dim() == 2 && t.size(0) == n && t.size(1) >= cols && t.stride(1) == 1, what,
              ": [", n, ", >= ", cols, "] rows expected");
}
void floats(const Tensor& t, int64_t numel, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.is_contiguous() && t.numel() == numel, what, ": contiguous fp32 tensor of ", numel,
              " elements expected");
}
const int64_t* longs(const Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt64 && t.is_contiguous() && t.numel() == n, what, ": int64 [", n, "] expected");
  return t.data_ptr<int64_t>();
}
const int64_t* longs(const OptTensor& t, int64_t n, const char* what) { return t ? longs(*t, n, what) : nullptr; }
const int* ints(const Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt32 && t.is_contiguous() && t.numel() == n, what, ": int32 [", n, "] expected");
  return t.data_ptr<int>();
}

void stream_mix(Tensor& x, const OptTensor& branch, const OptTensor& dest, int64_t per_token, const OptTensor& mix, const OptTensor& write,
                const OptTensor& read, const OptTensor& w, const OptTensor& b, const OptTensor& y, double eps) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 3 && x.is_contiguous() && x.scalar_type() == torch::kFloat32, "stream_mix: x fp32 [rows, k, D]");
  const int64_t N = x.size(0), k = x.size(1), D = x.size(2);
  TORCH_CHECK(branch || y, "stream_mix: nothing to do");
  TORCH_CHECK(bool(branch) == bool(mix) && bool(branch) == bool(write) && bool(w) == bool(y) && bool(b) == bool(y) && per_token >= 1);
  const Tensor& like = branch ? *branch : *y;
  const bool f = f32(like);
  if (branch) {
    TORCH_CHECK(branch->dim() == 2 && branch->is_contiguous() && branch->size(1) == D, "stream_mix: branch rows of the model width");
    if (dest) ints(*dest, N * per_token, "dest");
    else TORCH_CHECK(branch->size(0) == N * per_token, "stream_mix: ", per_token, " branch rows per token");
    same(*mix, like, k * k, "mix");
    same(*write, like, k, "write");
  }
  if (y) { same(*y, like, N * D, "y"); same(*w, like, D, "norm weight"); same(*b, like, D, "norm bias"); }
  const void* rd = same(read, like, k, "read");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_stream_mix(x.data_ptr<float>(), (int)k, branch ? branch->data_ptr() : nullptr, dest ? dest->data_ptr<int>() : nullptr, (int)per_token,
                     mix ? mix->data_ptr() : nullptr, write ? write->data_ptr() : nullptr, rd, w ? w->data_ptr() : nullptr, b ? b->data_ptr() : nullptr,
                     y ? y->data_ptr() : nullptr, f, N, (int)D, (float)eps, stream()), "stream_mix");
}

// x [B*S, >= C] projection rows, w [taps, C], bias [C] or None, hist [slots, taps-1, C] -> y [B*S, C]
void ssm_conv(const Tensor& x, const Tensor& w, const OptTensor& bias, int64_t S, Tensor& hist, const Tensor& slots, const Tensor& lengths,
              const OptTensor& new_lens, Tensor& y) {
  const bool f = f32(x);
  TORCH_CHECK(w.dim() == 2 && w.size(0) >= 1);
  const int64_t B = slots.numel(), taps = w.size(0), C = w.size(1);
  rows2d(x, x, B * S, C, "projection");
  TORCH_CHECK((reinterpret_cast<uintptr_t>(x.data_ptr()) % 16) == 0);
  same(w, x, taps * C, "filter"); same(y, x, B * S * C, "y");
  TORCH_CHECK(hist.is_cuda() && hist.scalar_type() == torch::kFloat32 && hist.is_contiguous() && hist.dim() == 3 && hist.size(1) == taps - 1 && hist.size(2) == C);
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_ssm_conv(f, x.data_ptr(), x.stride(0), w.data_ptr(), same(bias, x, C, "bias"), (int)taps, (int)C, (int)S, hist.data_ptr<float>(), longs(slots, B, "slots"),
                   longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), y.data_ptr(), (int)B, stream()), "ssm_conv");
}

// x [B*S, C]; p [B*S, 2C] projection rows whose second half is the gate; q [B*S, >= off + 2N]; dt fp32 [B*S, C]; rec [slots, 1, C, N] -> y [B*S, C]
void ssm_scan(const Tensor& x, const Tensor& p, const Tensor& q, const Tensor& dt, const Tensor& dt_bias, const Tensor& A_log, const Tensor& D, int64_t off,
              int64_t N, int64_t S, Tensor& rec, const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& y) {
  const bool f = f32(x);
  const int64_t B = slots.numel(), C = D.numel();
  same(x, x, B * S * C, "x"); same(y, x, B * S * C, "y");
  rows2d(p, x, B * S, 2 * C, "projection");
  rows2d(q, x, B * S, off + 2 * N, "step size, B, C");
  floats(dt, B * S * C, "dt");
  same(dt_bias, x, C, "dt bias"); same(A_log, x, C * N, "A_log"); same(D, x, C, "D");
  TORCH_CHECK(rec.is_cuda() && rec.scalar_type() == torch::kFloat32 && rec.is_contiguous() && rec.dim() == 4 && rec.size(1) == 1 && rec.size(2) == C &&
              rec.size(3) == N, "ssm_scan: state of the wrong size");
  c10::cuda::CUDAGuard guard(x.device());
  const char* z = static_cast<const char*>(p.data_ptr()) + C * p.element_size();
  done(mt_ssm_scan(f, x.data_ptr(), z, p.stride(0), q.data_ptr(), q.stride(0), (int)off, dt.data_ptr<float>(), dt_bias.data_ptr(), A_log.data_ptr(),
                   D.data_ptr(), (int)C, (int)N, (int)S, rec.data_ptr<float>(), longs(slots, B, "slots"), longs(lengths, B, "lengths"),
                   longs(new_lens, B, "new_lens"), y.data_ptr(), (int)B, stream()), "ssm_scan");
}

void check_cache(const Tensor& k, const Tensor& v, const Tensor& like, int64_t D) {
  TORCH_CHECK(k.dim() == 4 && v.dim() == 4 && k.size(0) == v.size(0) && k.size(1) == v.size(1) && k.size(2) == v.size(2) && k.size(3) == D,
              "cache: keys and values of different shapes");
  same(k, like, k.numel(), "key cache");
  same(v, like, v.numel(), "value cache");
}

// q / k / v rows of the projections -> qp [N, H * maps, dq], kp [N, G, dq] or None, vp [N, G, dvp] or None, cache rows. rot: rotated lanes;
// eps < 0: no norm; without norm weights the norm follows the rotation, with them it precedes it (one head's weights, or all heads').
// temp_every 0: no query temperature. maps 2: differential attention, D being the width of one map.
void qkv_prep(const Tensor& q, const Tensor& k, const Tensor& v, int64_t D, int64_t Dv, const Tensor& pos, const OptTensor& inv_ts, int64_t rot, double eps,
              Tensor& qp, const OptTensor& kp, const OptTensor& vp, Tensor& kc, Tensor& vc, const Tensor& slots, const Tensor& lengths,
              const OptTensor& new_lens, const OptTensor& bq, const OptTensor& bk, const OptTensor& bv, const OptTensor& wq, const OptTensor& wk, bool paired,
              int64_t maps, double temp_coef, double temp_every, const OptTensor& talk) {
  const bool f = f32(q);
  TORCH_CHECK(qp.dim() == 3 && rot % 2 == 0 && rot >= 0 && rot <= D && bool(inv_ts) == (rot > 0) && maps >= 1 && qp.size(1) % maps == 0);
  const int64_t N = q.size(0), H = qp.size(1) / maps, dq = qp.size(2), B = slots.numel();
  check_cache(kc, vc, q, D * maps);
  const int64_t G = kc.size(2);
  TORCH_CHECK(vc.size(3) == Dv && B > 0 && N % B == 0 && dq >= D * maps && H % G == 0 && (!talk || (maps == 1 && dq == G * D)));
  rows2d(q, q, N, H * maps * D, "q"); rows2d(k, q, N, G * maps * D, "k"); rows2d(v, q, N, G * Dv, "v");
  same(qp, q, N * H * maps * dq, "packed q");
  if (kp) same(*kp, q, N * G * (talk ? D : dq), "packed k");
  int64_t dvp = Dv;
  if (vp) { dvp = vp->size(vp->dim() - 1); TORCH_CHECK(dvp >= Dv); same(*vp, q, N * G * dvp, "packed v"); }
  if (inv_ts) floats(*inv_ts, rot / 2, "inverse timescales");
  TORCH_CHECK(bool(wq) == bool(wk) && (!wq || eps >= 0));
  const bool all = wq && (wq->numel() != D || wk->numel() != D || (H * maps == 1 && G * maps == 1));
  mt::cattn::PrepArgs a{};
  a.q = q.data_ptr(); a.k = k.data_ptr(); a.v = v.data_ptr();
  a.ldq = q.stride(0); a.ldk = k.stride(0); a.ldv = v.stride(0);
  a.bq = same(bq, q, H * maps * D, "q bias"); a.bk = same(bk, q, G * maps * D, "k bias"); a.bv = same(bv, q, G * Dv, "v bias");
  a.wq = same(wq, q, all ? H * maps * D : D, "q norm"); a.wk = same(wk, q, all ? G * maps * D : D, "k norm");
  a.norm = eps < 0 ? mt::cattn::NORM_NONE : !wq ? mt::cattn::NORM_AFTER : all ? mt::cattn::NORM_ALL : mt::cattn::NORM_HEAD;
  a.H = (int)H; a.G = (int)G; a.D = (int)D; a.Dv = (int)Dv; a.maps = (int)maps;
  a.pos = longs(pos, N, "positions");
  a.inv_ts = inv_ts ? inv_ts->data_ptr<float>() : nullptr;
  a.rot = (int)rot; a.paired = paired;
  a.eps = (float)eps; a.temp_coef = (float)temp_coef; a.temp_every = (float)temp_every;
  a.S = (int)(N / B);
  a.talk = same(talk, q, H * H, "mixing matrix");
  a.qp = qp.data_ptr(); a.kp = kp ? kp->data_ptr() : nullptr; a.vp = vp ? vp->data_ptr() : nullptr;
  a.dq = (int)dq; a.dvp = (int)dvp;
  a.kc = kc.data_ptr(); a.vc = vc.data_ptr(); a.max_len = kc.size(1);
  a.slots = longs(slots, B, "slots"); a.lengths = longs(lengths, B, "lengths"); a.new_lens = longs(new_lens, B, "new_lens");
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_qkv_prep(f, &a, N, stream()), "qkv_prep");
}

// lam: the four lambda vectors of differential attention
mt::cattn::DiffArgs diff_args(const std::vector<Tensor>& lam, const Tensor& like, double diff, double eps) {
  TORCH_CHECK(lam.size() == 4, "differential attention: four lambda vectors");
  const int64_t D = lam[0].numel();
  for (const Tensor& t : lam) same(t, like, D, "lambda");
  return {lam[0].data_ptr(), lam[1].data_ptr(), lam[2].data_ptr(), lam[3].data_ptr(), (int)D, (float)diff, (float)eps};
}

// gate rows [N, >= H * Dv], or [N, >= H] with one gate per head
const void* gate_rows(const OptTensor& gate, const Tensor& like, int64_t N, int64_t H, int64_t Dv, bool per_head) {
  if (!gate) return nullptr;
  rows2d(*gate, like, N, per_head ? H : H * Dv, "gate");
  return gate->data_ptr();
}

// parts of the key range that fill the machine twice over without making a part shorter than four tiles; long ranges are cut up to four times
// anyway, so that the last wave of CTAs is short
int64_t cached_decode_splits(int64_t B, int64_t H, int64_t G, int64_t span) {
  const int64_t ctas = std::max<int64_t>(1, B * G * ((H / G + 15) / 16));
  const int64_t fill = 2 * mt_num_sms() / ctas, even = std::min<int64_t>(4, span / 1024);
  return std::max<int64_t>(1, std::min<int64_t>({64, std::max(fill, even), (span + 63) / 64}));
}

void cached_decode(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& slots, const Tensor& lengths, double scale, double cap, int64_t window,
                   const OptTensor& sinks, const OptTensor& gate, int64_t splits, Tensor& part, Tensor& ml, Tensor& out, int64_t chunk, bool per_head,
                   const std::vector<Tensor>& lam, double diff, double eps) {
  TORCH_CHECK(!f32(q) && q.dim() == 3 && q.is_contiguous());
  const int64_t B = q.size(0), H = q.size(1), D = q.size(2), heads = lam.empty() ? H : H / 2;
  check_cache(k, v, q, D);
  const int64_t G = k.size(2), Dv = v.size(3);
  TORCH_CHECK(H % G == 0 && splits >= 1 && (lam.empty() || H % 2 == 0));
  floats(part, B * H * splits * Dv, "part"); floats(ml, B * H * splits * 2, "ml");
  same(out, q, B * heads * Dv, "out");
  const void* sk = same(sinks, q, H, "sinks");
  const void* gp = gate_rows(gate, q, B, heads, Dv, per_head);
  mt::cattn::DiffArgs d{};
  if (!lam.empty()) d = diff_args(lam, q, diff, eps);
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_cached_decode(q.data_ptr(), k.data_ptr(), v.data_ptr(), longs(slots, B, "slots"), longs(lengths, B, "lengths"), k.size(1), (int)B, (int)H, (int)G,
                        (int)D, (int)Dv, (float)scale, (float)cap, (int)window, (int)chunk, sk, gp, gate ? gate->stride(0) : 0, per_head,
                        lam.empty() ? nullptr : &d, (int)splits, part.data_ptr<float>(), ml.data_ptr<float>(), out.data_ptr(), stream()), "cached_decode", 2);
}

void cached_attention(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& slots, const Tensor& lengths, int64_t S, double scale, double cap,
                      int64_t window, const OptTensor& sinks, Tensor& out, int64_t chunk) {
  const bool f = f32(q);
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous());
  const int64_t B = slots.numel(), H = q.size(1), D = q.size(2);
  check_cache(k, v, q, D);
  const int64_t G = k.size(2), Dv = v.size(3);
  TORCH_CHECK(q.size(0) == B * S && H % G == 0);
  same(out, q, B * S * H * Dv, "out");
  const void* sk = same(sinks, q, H, "sinks");
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_cached_attention(f, q.data_ptr(), k.data_ptr(), v.data_ptr(), k.size(1), longs(slots, B, "slots"), longs(lengths, B, "lengths"), (int)B, (int)S, (int)H,
                           (int)G, (int)D, (int)Dv, (float)scale, (float)cap, (int)window, (int)chunk, sk, out.data_ptr(), stream()), "cached_attention");
}

// q [B, H, G * D] (one key of all key heads side by side), k [slots, max_len, G, D], v [.., G, Dv] -> out [B, H * Dv]
void wide_decode(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& slots, const Tensor& lengths, double scale, int64_t window, int64_t chunk,
                 const OptTensor& sinks, int64_t splits, Tensor& part, Tensor& ml, Tensor& out) {
  TORCH_CHECK(!f32(q) && q.dim() == 3 && q.is_contiguous() && k.dim() == 4 && v.dim() == 4);
  const int64_t B = q.size(0), H = q.size(1), G = k.size(2), D = k.size(3), Dv = v.size(3);
  check_cache(k, v, q, D);
  TORCH_CHECK(q.size(2) == G * D && H % G == 0 && splits >= 1);
  floats(part, B * H * splits * Dv, "part"); floats(ml, B * H * splits * 2, "ml");
  same(out, q, B * H * Dv, "out");
  const void* sk = same(sinks, q, H, "sinks");
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_wide_decode(q.data_ptr(), k.data_ptr(), v.data_ptr(), longs(slots, B, "slots"), longs(lengths, B, "lengths"), k.size(1), (int)B, (int)H, (int)G,
                      (int)D, (int)Dv, (float)scale, (int)window, (int)chunk, sk, (int)splits, part.data_ptr<float>(), ml.data_ptr<float>(), out.data_ptr(),
                      stream()), "wide_decode", 2);
}

void wide_attention(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& slots, const Tensor& lengths, int64_t S, double scale, int64_t window,
                    int64_t chunk, const OptTensor& sinks, Tensor& out) {
  const bool f = f32(q);
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && k.dim() == 4 && v.dim() == 4);
  const int64_t B = slots.numel(), H = q.size(1), G = k.size(2), D = k.size(3), Dv = v.size(3);
  check_cache(k, v, q, D);
  TORCH_CHECK(q.size(0) == B * S && q.size(2) == G * D && H % G == 0);
  same(out, q, B * S * H * Dv, "out");
  const void* sk = same(sinks, q, H, "sinks");
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_wide_attention(f, q.data_ptr(), k.data_ptr(), v.data_ptr(), k.size(1), longs(slots, B, "slots"), longs(lengths, B, "lengths"), (int)B, (int)S, (int)H,
                         (int)G, (int)D, (int)Dv, (float)scale, (int)window, (int)chunk, sk, out.data_ptr(), stream()), "wide_attention");
}

// q [B, Sq, H, G * D] contiguous, k [B, Skv, G, D] and v [B, Skv, G, Dv] rows whose heads lie side by side -> out [B, Sq, H * Dv]
void wide_flash(const Tensor& q, const Tensor& k, const Tensor& v, Tensor& out, const OptTensor& seg_q, const OptTensor& seg_k, const OptTensor& pos_q,
                const OptTensor& pos_k, const OptTensor& sinks, double scale, int64_t window, int64_t chunk, int64_t q_off) {
  TORCH_CHECK(!f32(q) && q.dim() == 4 && q.is_contiguous() && k.dim() == 4 && v.dim() == 4);
  const int64_t B = q.size(0), Sq = q.size(1), H = q.size(2), Skv = k.size(1), G = k.size(2), D = k.size(3), Dv = v.size(3);
  auto rows = [&](const Tensor& t, int64_t w) {
    return t.is_cuda() && t.scalar_type() == torch::kBFloat16 && t.size(0) == B && t.size(1) == Skv && t.size(2) == G && t.size(3) == w && t.stride(3) == 1 &&
           (G == 1 || t.stride(2) == w) && t.stride(1) % 8 == 0 && t.stride(1) >= G * w && (B == 1 || t.stride(0) % 8 == 0) &&
           reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0;
  };
  TORCH_CHECK(rows(k, D) && rows(v, Dv) && q.size(3) == G * D && H % G == 0 && D % 8 == 0 && Dv % 8 == 0 && Dv <= 128 && Skv >= 1 && Sq >= 1,
              "wide_flash: unsupported operands");
  same(out, q, B * Sq * H * Dv, "out");
  TORCH_CHECK(bool(seg_q) == bool(seg_k) && bool(pos_q) == bool(pos_k));
  auto opt = [&](const OptTensor& t, int64_t n, const char* what) { return t ? ints(*t, n, what) : nullptr; };
  const void* sk = same(sinks, q, H, "sinks");
  c10::cuda::CUDAGuard guard(q.device());
  Tensor tiles;
  if (pos_q) tiles = torch::empty({mt_attn_tile_ints((int)B, (int)Sq, (int)Skv)}, torch::dtype(torch::kInt32).device(q.device()));
  done(mt_wide_flash(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), opt(seg_q, B * Sq, "seg_q"), opt(seg_k, B * Skv, "seg_k"),
                     opt(pos_q, B * Sq, "pos_q"), opt(pos_k, B * Skv, "pos_k"), pos_q ? tiles.data_ptr<int>() : nullptr, sk, (int)B, (int)Sq, (int)Skv, (int)H,
                     (int)G, (int)D, (int)Dv, k.stride(1), k.stride(0), v.stride(1), v.stride(0), (float)scale, (int)window, (int)chunk, (int)q_off,
                     mt_status_ptr(), stream()), "wide_flash", pos_q ? 3 : 1);
}

// o [N, H, >= dv], g [N, >= H * dv] (or [N, >= H]) -> out [N, H * dv]
void head_gate(const Tensor& o, const Tensor& g, int64_t dv, Tensor& out, bool per_head) {
  const bool f = f32(o);
  TORCH_CHECK(o.dim() == 3 && o.is_contiguous() && o.size(2) >= dv);
  const int64_t N = o.size(0), H = o.size(1);
  gate_rows(g, o, N, H, dv, per_head);
  same(out, o, N * H * dv, "out");
  c10::cuda::CUDAGuard guard(o.device());
  done(mt_head_gate(f, o.data_ptr(), (int)o.size(2), g.data_ptr(), g.stride(0), N, (int)(H * dv), (int)dv, per_head, out.data_ptr(), mt_num_sms(), stream()),
       "head_gate");
}

// o [N, 2 H, >= dv] (two maps per head) -> out [N, H * dv]
void diff_combine(const Tensor& o, const std::vector<Tensor>& lam, double diff, double eps, const OptTensor& gate, int64_t dv, Tensor& out, bool per_head) {
  const bool f = f32(o);
  TORCH_CHECK(o.dim() == 3 && o.is_contiguous() && o.size(2) >= dv && o.size(1) % 2 == 0);
  const int64_t N = o.size(0), H = o.size(1) / 2;
  const void* gp = gate_rows(gate, o, N, H, dv, per_head);
  same(out, o, N * H * dv, "out");
  const auto d = diff_args(lam, o, diff, eps);
  c10::cuda::CUDAGuard guard(o.device());
  done(mt_diff_combine(f, o.data_ptr(), (int)o.size(2), &d, N, (int)H, (int)dv, gp, gate ? gate->stride(0) : 0, per_head, out.data_ptr(), mt_num_sms(),
                       stream()), "diff_combine");
}

void check_plan(const Tensor& sizes, const Tensor& offs, const Tensor& row_pair, int64_t E) {
  ints(sizes, E, "sizes"); ints(offs, E + 1, "offs"); ints(row_pair, row_pair.numel(), "row_pair");
}

// w1 absent: ungated experts
void expert_up(const Tensor& x, const Tensor& w0, const OptTensor& w1, const Tensor& wts, const Tensor& idx, const Tensor& sizes, const Tensor& offs,
               const Tensor& row_pair, int64_t k, double limit, Tensor& h) {
  const bool f = f32(x);
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && w0.dim() == 3 && w0.size(2) == x.size(1));
  const int64_t E = w0.size(0), F = w0.size(1), D = w0.size(2), n = x.size(0) * k;
  same(w0, x, E * F * D, "w0"); same(w1, x, E * F * D, "w1"); same(h, x, n * F, "h");
  floats(wts, n, "scores");
  check_plan(sizes, offs, row_pair, E);
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_expert_up(f, x.data_ptr(), w0.data_ptr(), w1 ? w1->data_ptr() : nullptr, wts.data_ptr<float>(), ints(idx, n, "idx"), sizes.data_ptr<int>(), offs.data_ptr<int>(),
                    row_pair.data_ptr<int>(), (int)n, (int)k, (int)E, (int)F, (int)D, (float)limit, h.data_ptr(), mt_num_sms(), stream()), "expert_up");
}

void expert_down(const Tensor& h, const Tensor& w, const Tensor& idx, const Tensor& sizes, const Tensor& offs, const Tensor& row_pair, Tensor& y) {
  const bool f = f32(h);
  TORCH_CHECK(h.dim() == 2 && h.is_contiguous() && w.dim() == 3 && w.size(2) == h.size(1));
  const int64_t E = w.size(0), D = w.size(1), F = w.size(2), n = h.size(0);
  same(w, h, E * F * D, "w"); same(y, h, n * D, "y");
  check_plan(sizes, offs, row_pair, E);
  c10::cuda::CUDAGuard guard(h.device());
  done(mt_expert_down(f, h.data_ptr(), w.data_ptr(), ints(idx, n, "idx"), sizes.data_ptr<int>(), offs.data_ptr<int>(), row_pair.data_ptr<int>(), (int)n, (int)E,
                      (int)D, (int)F, y.data_ptr(), mt_num_sms(), stream()), "expert_down");
}

// gu [rows_max, 2F] (ungated experts: [rows_max, F]) of the padded layout -> h [rows_max, F]
void expert_act(const Tensor& gu, const Tensor& wts, const Tensor& row_pair, const Tensor& offs, double limit, Tensor& h) {
  TORCH_CHECK(!f32(gu) && gu.dim() == 2 && gu.is_contiguous() && h.dim() == 2 && (gu.size(1) == 2 * h.size(1) || gu.size(1) == h.size(1)) && h.size(1) % 8 == 0);
  same(h, gu, gu.size(0) * h.size(1), "h");
  ints(row_pair, gu.size(0), "row_pair"); ints(offs, offs.numel(), "offs"); floats(wts, wts.numel(), "scores");
  c10::cuda::CUDAGuard guard(gu.device());
  done(mt_expert_act(gu.data_ptr(), gu.size(1) == 2 * h.size(1), wts.data_ptr<float>(), row_pair.data_ptr<int>(), offs.data_ptr<int>(), (int)offs.numel() - 1, (int)h.size(1), (float)limit,
                     h.data_ptr(), (int)gu.size(0), mt_num_sms(), stream()), "expert_act");
}

}  // namespace

void register_hybrid(pybind11::module_& m) {
  m.def("stream_mix", &stream_mix);
  m.def("ssm_conv", &ssm_conv);
  m.def("ssm_scan", &ssm_scan);
  using pybind11::arg;
  const auto none = pybind11::none();
  m.def("qkv_prep", &qkv_prep, arg("q"), arg("k"), arg("v"), arg("D"), arg("Dv"), arg("pos"), arg("inv_ts"), arg("rot"), arg("eps"), arg("qp"), arg("kp"),
        arg("vp"), arg("kc"), arg("vc"), arg("slots"), arg("lengths"), arg("new_lens"), arg("bq") = none, arg("bk") = none, arg("bv") = none, arg("wq") = none,
        arg("wk") = none, arg("paired") = false, arg("maps") = 1, arg("temp_coef") = 0.0, arg("temp_every") = 0.0, arg("talk") = none);
  m.def("cached_decode_splits", &cached_decode_splits);
  m.def("cached_decode", &cached_decode, arg("q"), arg("k"), arg("v"), arg("slots"), arg("lengths"), arg("scale"), arg("cap"), arg("window"), arg("sinks"),
        arg("gate"), arg("splits"), arg("part"), arg("ml"), arg("out"), arg("chunk") = 0, arg("per_head") = false, arg("lam") = std::vector<Tensor>{},
        arg("diff") = 0.0, arg("eps") = 0.0);
  m.def("cached_attention", &cached_attention, arg("q"), arg("k"), arg("v"), arg("slots"), arg("lengths"), arg("S"), arg("scale"), arg("cap"), arg("window"),
        arg("sinks"), arg("out"), arg("chunk") = 0);
  m.def("wide_decode", &wide_decode);
  m.def("wide_attention", &wide_attention);
  m.def("wide_flash", &wide_flash);
  m.def("head_gate", &head_gate, arg("o"), arg("g"), arg("dv"), arg("out"), arg("per_head") = false);
  m.def("diff_combine", &diff_combine);
  m.def("expert_up", &expert_up);
  m.def("expert_down", &expert_down);
  m.def("expert_act", &expert_act);
}
