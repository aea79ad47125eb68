// Bindings of the inference kernels for fp32 residual streams, recurrent layers and latent attention. Every entry checks types, layouts and
// sizes before it launches; pointers handed to the kernels are in bounds for the sizes given with them.
#include <torch/extension.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <cuda_runtime.h>
#include "residual_gate.h"

extern "C" {
int mt_residual_gate(const mt::ResidualGate* a, int f32, long rows, int D, cudaStream_t st);
int mt_act_rows(const void* x, long ldx, void* y, int f32, long rows, int F, int code, const void* par, int sms, cudaStream_t st);
int mt_residual_norm(float* x, const void* branch, const void* w_post, float mult, const void* w_next, void* y, int f32, long rows, int D, float eps_post,
                     float eps_next, float offset, cudaStream_t st);
int mt_residual_join(float* x, const void* a, const void* a_bias, const void* a_norm, float a_factor, const void* b, const void* b_bias, const void* b_norm,
                     float b_factor, const void* lanes, const void* w_next, void* y, int f32, long rows, int D, float eps, cudaStream_t st);
int mt_token_gate(const void* g, const void* table, const int64_t* tokens, void* out, int f32, long N, int dim, long vocab, int sms, cudaStream_t st);
int mt_act_fwd(const void* x, void* y, int f32, long n, int code, int sms, cudaStream_t st);
int mt_delta_decode(int f32, const void* x, long ldx, const void* ba, long ldb, const void* conv_w, int taps, const void* A_log, const void* dt_bias,
                    const void* norm, float eps, int hk, int hv, int dk, int dv, float* conv, float* rec, const int64_t* slots, const int64_t* lengths,
                    void* out, int B, cudaStream_t st);
int mt_gla_decode(int f32, const void* x, long ldx, const void* w, const void* bias, int rank, float inv_tau, const void* norm, float eps, int H, int dk,
                  int dv, float* rec, const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st);
int mt_delta_conv(int f32, const void* x, long ldx, const void* conv_w, int taps, int hk, int hv, int dk, int dv, int S, float* conv, const int64_t* slots,
                  const int64_t* lengths, const int64_t* new_lens, void* y, int B, cudaStream_t st);
int mt_delta_scan(int f32, const void* mixed, const void* ba, long ldb, const void* A_log, const void* dt_bias, int hk, int hv, int dk, int dv, int S,
                  float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st);
int mt_gla_scan(int f32, const void* x, long ldx, const float* log_alpha, int H, int dk, int dv, int S, float* rec, const int64_t* slots,
                const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st);
int mt_chunk_supported(int dk, int dv);
int mt_delta_chunks(const void* mixed, long ldx, const void* ba, long ldb, const void* A_log, const void* dt_bias, int hk, int hv, int dk, int dv, int S,
                    int t_lo, int t_hi, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* tp, float* gates, float* ends,
                    void* o, int B, cudaStream_t st);
int mt_gla_chunks(const void* x, long ldx, const float* log_alpha, int H, int dk, int dv, int S, int t_lo, int t_hi, float* rec, const int64_t* slots,
                  const int64_t* lengths, const int64_t* new_lens, void* aa, void* qkg, float* ends, void* o, int B, cudaStream_t st);
int mt_gla_decay(int f32, const void* lo, long ldx, const void* w, const void* bias, int rank, float inv_tau, float* out, long N, int C, cudaStream_t st);
int mt_gated_head_norm(int f32, const void* o, const void* x, long ldx, long rows, int H, int dv, int r, long zoff, long zstride, const void* w, float eps,
                       int sig, void* out, cudaStream_t st);
int mt_retention_decode(int f32, const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, float eps, int H, int dk, int dv, float* rec,
                        const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st);
int mt_retention_scan(int f32, const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, int H, int dk, int dv, int S, float* rec,
                      const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o, int B, cudaStream_t st);
int mt_retention_chunks(const void* x, long ldx, const float* log_decay, const float* inv_ts, int rot, int H, int dk, int dv, int S, int t_lo, int t_hi,
                        float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* aa, void* qkg, float* ends, void* o, int B,
                        cudaStream_t st);
int mt_channel_delta_decode(int f32, const void* x, long ldx, const void* beta, long ldb, const void* conv_w, int taps, const float* da, const void* A_log,
                            const void* dt_bias, const void* z, long ldz, const void* norm, float eps, int hk, int hv, int dk, int dv, float* conv, float* rec,
                            const int64_t* slots, const int64_t* lengths, void* out, int B, cudaStream_t st);
int mt_channel_delta_scan(int f32, const void* mixed, const void* beta, long ldb, const float* da, const void* A_log, const void* dt_bias, int hk, int hv,
                          int dk, int dv, int S, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, void* o, int B,
                          cudaStream_t st);
int mt_channel_delta_chunks(const void* mixed, long ldx, const void* beta, long ldb, const float* da, const void* A_log, const void* dt_bias, int hk, int hv,
                            int dk, int dv, int S, int t_lo, int t_hi, float* rec, const int64_t* slots, const int64_t* lengths, const int64_t* new_lens,
                            void* tp, void* qkg, float* betas, float* ends, void* o, int B, cudaStream_t st);
int mt_mla_prep(int f32, const void* qa, long ldq, const void* qw, int Q, const void* kva, long ldk, const void* kw, int R, int dr, float eps,
                const int64_t* pos, const float* inv_ts, int interleaved, int S, void* cq, void* lat, void* kr, void* cache_lat, void* cache_kr, long max_len,
                const int64_t* slots, const int64_t* lengths, const int64_t* new_lens, long N, cudaStream_t st);
int mt_mla_pack(const void* q, const void* kv, const void* kr, const int64_t* pos, const float* inv_ts, int interleaved, long NQ, long NK, int H, int nope,
                int dr, int vd, int DQ, int DV, void* qp, void* kp, void* vp, cudaStream_t st);
int mt_mla_absorb(int f32, const void* q, const void* w, const int64_t* pos, const float* inv_ts, int interleaved, int B, int H, int nope, int dr, int vd,
                  int R, void* qa, cudaStream_t st);
int mt_mla_decode_attn(int f32, const void* qa, const void* lat, const void* kr, long max_len, const int64_t* slots, const int64_t* lengths, int B, int H,
                       int R, int dr, float scale, int window, int splits, float* part, float* ml, cudaStream_t st);
int mt_mla_value_up(int f32, const float* part, const float* ml, const void* w, int B, int H, int nope, int vd, int R, int splits, void* out,
                    cudaStream_t st);
}

int* mt_status_ptr();          // defined in bindings.cpp
void mt_count_launches(int n); // defined in bindings.cpp
int mt_num_sms();              // defined in bindings.cpp

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
void rows2d(const Tensor& t, const Tensor& like, int64_t n, int64_t cols, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == like.scalar_type() && t.dim() == 2 && t.size(0) == n && t.size(1) >= cols && t.stride(1) == 1, what,
              ": [", n, ", >= ", cols, "] rows expected");
}
const int64_t* longs(const Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt64 && t.is_contiguous() && t.numel() == n, what, ": int64 [", n, "] expected");
  return t.data_ptr<int64_t>();
}
const int64_t* longs(const OptTensor& t, int64_t n, const char* what) { return t ? longs(*t, n, what) : nullptr; }
float* state(const Tensor& t, std::vector<int64_t> tail, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.is_contiguous() && t.dim() == (int64_t)tail.size() + 1, what, ": fp32 state expected");
  for (size_t i = 0; i < tail.size(); ++i) TORCH_CHECK(t.size(i + 1) == tail[i], what, ": state of the wrong size");
  return t.data_ptr<float>();
}

void residual_norm(Tensor& x, const OptTensor& branch, const OptTensor& w_post, double mult, const OptTensor& w_next, const OptTensor& y, double eps_post,
                   double eps_next, double offset) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.is_contiguous() && x.scalar_type() == torch::kFloat32);
  TORCH_CHECK((branch && w_post) || (w_next && y), "residual_norm: nothing to do");
  TORCH_CHECK(bool(w_next) == bool(y) && bool(branch) == bool(w_post));
  const Tensor& like = branch ? *branch : *y;
  const bool f = f32(like);
  if (branch) { same(*branch, like, x.numel(), "branch"); same(*w_post, like, x.size(1), "w_post"); }
  if (y) { same(*y, like, x.numel(), "y"); same(*w_next, like, x.size(1), "w_next"); }
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_residual_norm(x.data_ptr<float>(), branch ? branch->data_ptr() : nullptr, w_post ? w_post->data_ptr() : nullptr, (float)mult,
                        w_next ? w_next->data_ptr() : nullptr, y ? y->data_ptr() : nullptr, f, x.size(0), (int)x.size(1), (float)eps_post, (float)eps_next,
                        (float)offset, stream()), "residual_norm");
}

const void* lane_vector(const OptTensor& t, const Tensor& like, int64_t D, const char* what) {
  if (!t) return nullptr;
  same(*t, like, D, what);
  return t->data_ptr();
}

// x [rows, D] fp32 += lanes * (a + b), each branch [norm of](out + bias) * factor; y: rms(x) * w_next, x itself without w_next, or None
void residual_join(Tensor& x, const Tensor& a, const OptTensor& a_bias, const OptTensor& a_norm, double a_factor, const OptTensor& b, const OptTensor& b_bias,
                   const OptTensor& b_norm, double b_factor, const OptTensor& lanes, const OptTensor& w_next, const OptTensor& y, double eps) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.is_contiguous() && x.scalar_type() == torch::kFloat32 && x.size(1) <= 8192, "residual_join: x fp32 [rows, <= 8192]");
  const bool f = f32(a);
  const int64_t D = x.size(1);
  TORCH_CHECK(y || !w_next, "residual_join: a norm without a result");
  same(a, a, x.numel(), "branch");
  if (b) same(*b, a, x.numel(), "second branch");
  if (y) same(*y, a, x.numel(), "y");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_residual_join(x.data_ptr<float>(), a.data_ptr(), lane_vector(a_bias, a, D, "bias"), lane_vector(a_norm, a, D, "norm"), (float)a_factor,
                        b ? b->data_ptr() : nullptr, lane_vector(b_bias, a, D, "bias"), lane_vector(b_norm, a, D, "norm"), (float)b_factor,
                        lane_vector(lanes, a, D, "lane factors"), lane_vector(w_next, a, D, "next norm"), y ? y->data_ptr() : nullptr, f, x.size(0), (int)D,
                        (float)eps, stream()), "residual_join");
}

// x [N, D] fp32 += norm(b * sigmoid(gate + bias)) * w_post with b the sum of `per_token` of `rows` (dest: which) and `extra`; y: norm(x) * w_next, x itself
// without w_next, or None. gate and y may be columns of wider matrices. centred: layer norms, otherwise RMS norms. fresh: x is only written.
void residual_gate(Tensor& x, const OptTensor& rows, const OptTensor& dest, int64_t per_token, const OptTensor& extra, const OptTensor& gate,
                   const OptTensor& bias, const OptTensor& w_post, const OptTensor& w_next, const OptTensor& y, double eps, bool centred, bool fresh) {
  TORCH_CHECK(x.is_cuda() && x.dim() == 2 && x.is_contiguous() && x.scalar_type() == torch::kFloat32 && x.size(1) <= 8192, "residual_gate: x fp32 [rows, <= 8192]");
  TORCH_CHECK((rows && w_post) || (y && !rows && !fresh), "residual_gate: nothing to do");
  TORCH_CHECK(bool(rows) == bool(w_post) && (!w_next || y) && bool(gate) == bool(bias) && (rows || !(gate || extra || dest)) && per_token >= 1);
  const Tensor& like = rows ? *rows : *y;
  const bool f = f32(like);
  const int64_t N = x.size(0), D = x.size(1);
  mt::ResidualGate a{};
  a.x = x.data_ptr<float>(); a.per_token = (int)per_token; a.eps = (float)eps; a.centred = centred; a.fresh = fresh;
  if (rows) {
    TORCH_CHECK(rows->dim() == 2 && rows->is_contiguous() && rows->size(1) == D && rows->size(0) >= 1, "residual_gate: branch rows of the model width");
    a.rows = rows->data_ptr(); a.n_rows = rows->size(0);
    if (dest) {
      TORCH_CHECK(dest->is_cuda() && dest->scalar_type() == torch::kInt32 && dest->is_contiguous() && dest->numel() == N * per_token, "residual_gate: int32 row numbers");
      a.dest = dest->data_ptr<int>();
    } else {
      TORCH_CHECK(rows->size(0) == N * per_token, "residual_gate: ", per_token, " branch rows per token");
    }
    same(*w_post, like, D, "w_post"); a.w_post = w_post->data_ptr();
    a.extra = lane_vector(extra, like, N * D, "extra rows");
    if (gate) {
      TORCH_CHECK(gate->is_cuda() && gate->scalar_type() == like.scalar_type() && gate->dim() == 2 && gate->size(0) == N && gate->size(1) == D &&
                  gate->stride(1) == 1, "residual_gate: gate [rows, D]");
      a.gate = gate->data_ptr(); a.ldg = gate->stride(0);
      a.bias = lane_vector(bias, like, D, "gate bias");
    }
  }
  a.w_next = lane_vector(w_next, like, D, "w_next");
  if (y) {
    TORCH_CHECK(y->is_cuda() && y->scalar_type() == like.scalar_type() && y->dim() == 2 && y->size(0) == N && y->size(1) == D && y->stride(1) == 1,
                "residual_gate: y [rows, D]");
    a.y = y->data_ptr(); a.ldy = y->stride(0);
  }
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_residual_gate(&a, f, N, (int)D, stream()), "residual_gate");
}

// x [N, F] rows (columns of a wider matrix allowed) -> y [N, F]; par: the two numbers of xIELU (code 6)
void act_rows(const Tensor& x, Tensor& y, int64_t code, const OptTensor& par) {
  const bool f = f32(x);
  TORCH_CHECK(x.dim() == 2 && (x.size(1) == 1 || x.stride(1) == 1) && bool(par) == (code == 6));
  same(y, x, x.numel(), "act_rows output");
  const void* pp = lane_vector(par, x, 2, "activation parameters");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_act_rows(x.data_ptr(), x.stride(0), y.data_ptr(), f, x.size(0), (int)x.size(1), (int)code, pp, mt_num_sms(), stream()), "act_rows");
}

// g [N, dim], table [V, dim], tokens [N] -> out [N, dim]
void token_gate(const Tensor& g, const Tensor& table, const Tensor& tokens, Tensor& out) {
  const bool f = f32(g);
  TORCH_CHECK(g.dim() == 2 && table.dim() == 2 && table.size(1) == g.size(1) && table.size(0) > 0);
  same(g, g, g.numel(), "g"); same(table, g, table.numel(), "table"); same(out, g, g.numel(), "out");
  c10::cuda::CUDAGuard guard(g.device());
  done(mt_token_gate(g.data_ptr(), table.data_ptr(), longs(tokens, g.size(0), "tokens"), out.data_ptr(), f, g.size(0), (int)g.size(1), table.size(0),
                     mt_num_sms(), stream()), "token_gate");
}

void act_fwd(const Tensor& x, Tensor& y, int64_t code) {
  const bool f = f32(x);
  TORCH_CHECK(x.is_contiguous() && (reinterpret_cast<uintptr_t>(x.data_ptr()) % 16) == 0);
  same(y, x, x.numel(), "act_fwd output");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_act_fwd(x.data_ptr(), y.data_ptr(), f, x.numel(), (int)code, mt_num_sms(), stream()), "act_fwd");
}

void check_delta(const Tensor& x, int64_t n, int64_t hk, int64_t hv, int64_t dk, int64_t dv) {
  TORCH_CHECK(hk > 0 && hv % hk == 0 && dk > 0 && dv > 0, "gated delta: bad head counts");
  rows2d(x, x, n, 2 * hk * dk + 2 * hv * dv, "packed projection");
}

void delta_decode(const Tensor& x, const Tensor& ba, const Tensor& conv_w, const Tensor& A_log, const Tensor& dt_bias, const Tensor& norm, double eps,
                  int64_t hk, int64_t hv, int64_t dk, int64_t dv, Tensor& conv, Tensor& rec, const Tensor& slots, const Tensor& lengths, Tensor& out) {
  const bool f = f32(x);
  const int64_t B = x.size(0), cd = 2 * hk * dk + hv * dv;
  check_delta(x, B, hk, hv, dk, dv);
  rows2d(ba, x, B, 2 * hv, "gates");
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(0) >= 1);
  const int64_t taps = conv_w.size(0);
  same(conv_w, x, taps * cd, "convolution"); same(A_log, x, hv, "A_log"); same(dt_bias, x, hv, "dt_bias"); same(norm, x, dv, "norm");
  same(out, x, B * hv * dv, "out");
  float* cp = state(conv, {taps - 1, cd}, "conv");
  float* rp = state(rec, {hv, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_delta_decode(f, x.data_ptr(), x.stride(0), ba.data_ptr(), ba.stride(0), conv_w.data_ptr(), (int)taps, A_log.data_ptr(), dt_bias.data_ptr(),
                       norm.data_ptr(), (float)eps, (int)hk, (int)hv, (int)dk, (int)dv, cp, rp, longs(slots, B, "slots"), longs(lengths, B, "lengths"),
                       out.data_ptr(), (int)B, stream()), "delta_decode");
}

void gla_decode(const Tensor& x, const Tensor& w, const Tensor& bias, const Tensor& norm, double eps, double tau, int64_t H, int64_t dk, int64_t dv,
                Tensor& rec, const Tensor& slots, const Tensor& lengths, Tensor& out) {
  const bool f = f32(x);
  const int64_t B = x.size(0);
  TORCH_CHECK(w.dim() == 2 && w.size(0) == H * dk && w.size(1) % 8 == 0, "gla_decode: the rank is padded to a multiple of 8");
  rows2d(x, x, B, 2 * H * (dk + dv) + w.size(1), "packed projection");
  same(w, x, H * dk * w.size(1), "decay projection"); same(bias, x, H * dk, "decay bias"); same(norm, x, dv, "norm"); same(out, x, B * H * dv, "out");
  float* rp = state(rec, {H, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_gla_decode(f, x.data_ptr(), x.stride(0), w.data_ptr(), bias.data_ptr(), (int)w.size(1), (float)(1.0 / tau), norm.data_ptr(), (float)eps, (int)H,
                     (int)dk, (int)dv, rp, longs(slots, B, "slots"), longs(lengths, B, "lengths"), out.data_ptr(), (int)B, stream()), "gla_decode");
}

void delta_conv(const Tensor& x, const Tensor& conv_w, int64_t hk, int64_t hv, int64_t dk, int64_t dv, int64_t S, Tensor& conv, const Tensor& slots,
                const Tensor& lengths, const OptTensor& new_lens, Tensor& y) {
  const bool f = f32(x);
  const int64_t B = slots.numel(), cd = 2 * hk * dk + hv * dv;
  check_delta(x, B * S, hk, hv, dk, dv);
  TORCH_CHECK(conv_w.dim() == 2 && conv_w.size(0) >= 1 && (reinterpret_cast<uintptr_t>(x.data_ptr()) % 16) == 0);
  const int64_t taps = conv_w.size(0);
  same(conv_w, x, taps * cd, "convolution"); same(y, x, B * S * cd, "y");
  float* cp = state(conv, {taps - 1, cd}, "conv");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_delta_conv(f, x.data_ptr(), x.stride(0), conv_w.data_ptr(), (int)taps, (int)hk, (int)hv, (int)dk, (int)dv, (int)S, cp, longs(slots, B, "slots"),
                     longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), y.data_ptr(), (int)B, stream()), "delta_conv", 2);
}

void delta_scan(const Tensor& mixed, const Tensor& ba, const Tensor& A_log, const Tensor& dt_bias, int64_t hk, int64_t hv, int64_t dk, int64_t dv, int64_t S,
                Tensor& rec, const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  const bool f = f32(mixed);
  const int64_t B = slots.numel(), cd = 2 * hk * dk + hv * dv;
  same(mixed, mixed, B * S * cd, "mixed");
  rows2d(ba, mixed, B * S, 2 * hv, "gates");
  same(A_log, mixed, hv, "A_log"); same(dt_bias, mixed, hv, "dt_bias"); same(o, mixed, B * S * hv * dv, "o");
  float* rp = state(rec, {hv, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(mixed.device());
  done(mt_delta_scan(f, mixed.data_ptr(), ba.data_ptr(), ba.stride(0), A_log.data_ptr(), dt_bias.data_ptr(), (int)hk, (int)hv, (int)dk, (int)dv, (int)S, rp,
                     longs(slots, B, "slots"), longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), o.data_ptr(), (int)B, stream()), "delta_scan");
}

void gla_decay(const Tensor& x, int64_t at, const Tensor& w, const Tensor& bias, double tau, Tensor& out) {
  const bool f = f32(x);
  TORCH_CHECK(w.dim() == 2 && w.size(1) % 8 == 0, "gla_decay: the rank is padded to a multiple of 8");
  const int64_t N = x.size(0), C = w.size(0), rank = w.size(1);
  rows2d(x, x, N, at + rank, "packed projection");
  same(w, x, C * rank, "decay projection"); same(bias, x, C, "decay bias");
  TORCH_CHECK(out.is_cuda() && out.scalar_type() == torch::kFloat32 && out.is_contiguous() && out.numel() == N * C);
  c10::cuda::CUDAGuard guard(x.device());
  const char* lo = static_cast<const char*>(x.data_ptr()) + at * x.element_size();
  done(mt_gla_decay(f, lo, x.stride(0), w.data_ptr(), bias.data_ptr(), (int)rank, (float)(1.0 / tau), out.data_ptr<float>(), N, (int)C, stream()),
       "gla_decay");
}

void gla_scan(const Tensor& x, const Tensor& log_alpha, int64_t H, int64_t dk, int64_t dv, int64_t S, Tensor& rec, const Tensor& slots,
              const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  const bool f = f32(x);
  const int64_t B = slots.numel();
  rows2d(x, x, B * S, 2 * H * (dk + dv), "packed projection");
  TORCH_CHECK(log_alpha.is_cuda() && log_alpha.scalar_type() == torch::kFloat32 && log_alpha.is_contiguous() && log_alpha.numel() == B * S * H * dk);
  same(o, x, B * S * H * dv, "o");
  float* rp = state(rec, {H, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_gla_scan(f, x.data_ptr(), x.stride(0), log_alpha.data_ptr<float>(), (int)H, (int)dk, (int)dv, (int)S, rp, longs(slots, B, "slots"),
                   longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), o.data_ptr(), (int)B, stream()), "gla_scan");
}

// tokens of every row handled per launch pair, so that the per-chunk scratch stays near 256 MB
int64_t chunk_segment(int64_t B, int64_t H, int64_t S, int64_t bytes_per_token_head) {
  const int64_t fit = (int64_t(256) << 20) / std::max<int64_t>(1, B * H * bytes_per_token_head);
  return std::min((S + 63) / 64 * 64, std::max<int64_t>(64, fit / 64 * 64));
}

bool chunk_supported(int64_t dk, int64_t dv) { return mt_chunk_supported((int)dk, (int)dv) != 0; }

// the chunked form of delta_scan (bf16)
void delta_chunks(const Tensor& mixed, const Tensor& ba, const Tensor& A_log, const Tensor& dt_bias, int64_t hk, int64_t hv, int64_t dk, int64_t dv,
                  int64_t S, Tensor& rec, const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  TORCH_CHECK(!f32(mixed) && chunk_supported(dk, dv), "delta_chunks: bf16 and head widths of 16 .. 128 in steps of 16");
  const int64_t B = slots.numel(), cd = 2 * hk * dk + hv * dv;
  same(mixed, mixed, B * S * cd, "mixed");
  TORCH_CHECK((reinterpret_cast<uintptr_t>(mixed.data_ptr()) % 16) == 0);
  rows2d(ba, mixed, B * S, 2 * hv, "gates");
  same(A_log, mixed, hv, "A_log"); same(dt_bias, mixed, hv, "dt_bias"); same(o, mixed, B * S * hv * dv, "o");
  float* rp = state(rec, {hv, dk, dv}, "rec");
  const int64_t *sl = longs(slots, B, "slots"), *le = longs(lengths, B, "lengths"), *nl = longs(new_lens, B, "new_lens");
  c10::cuda::CUDAGuard guard(mixed.device());
  const int64_t seg = chunk_segment(B, hv, S, 4 * 64 * 2), tiles = B * (seg / 64) * hv;
  auto fo = torch::dtype(torch::kFloat32).device(mixed.device());
  auto tp = torch::empty({tiles * 4 * 64 * 64}, mixed.options());
  auto gates = torch::empty({tiles * 4 * 64}, fo), ends = torch::empty({tiles}, fo);
  for (int64_t t = 0; t < S; t += seg)
    done(mt_delta_chunks(mixed.data_ptr(), cd, ba.data_ptr(), ba.stride(0), A_log.data_ptr(), dt_bias.data_ptr(), (int)hk, (int)hv, (int)dk, (int)dv, (int)S,
                         (int)t, (int)std::min(S, t + seg), rp, sl, le, nl, tp.data_ptr(), gates.data_ptr<float>(), ends.data_ptr<float>(), o.data_ptr(), (int)B,
                         stream()), "delta_chunks", 2);
}

// the chunked form of gla_scan (bf16)
void gla_chunks(const Tensor& x, const Tensor& log_alpha, int64_t H, int64_t dk, int64_t dv, int64_t S, Tensor& rec, const Tensor& slots,
                const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  TORCH_CHECK(!f32(x) && chunk_supported(dk, dv), "gla_chunks: bf16 and head widths of 16 .. 128 in steps of 16");
  const int64_t B = slots.numel();
  rows2d(x, x, B * S, 2 * H * (dk + dv), "packed projection");
  TORCH_CHECK((reinterpret_cast<uintptr_t>(x.data_ptr()) % 16) == 0 && x.stride(0) % 8 == 0);
  TORCH_CHECK(log_alpha.is_cuda() && log_alpha.scalar_type() == torch::kFloat32 && log_alpha.is_contiguous() && log_alpha.numel() == B * S * H * dk);
  same(o, x, B * S * H * dv, "o");
  float* rp = state(rec, {H, dk, dv}, "rec");
  const int64_t *sl = longs(slots, B, "slots"), *le = longs(lengths, B, "lengths"), *nl = longs(new_lens, B, "new_lens");
  c10::cuda::CUDAGuard guard(x.device());
  const int64_t seg = chunk_segment(B, H, S, 2 * 64 * 2 + 4 * dk * 2), tiles = B * (seg / 64) * H;
  auto aa = torch::empty({tiles * 2 * 64 * 64}, x.options()), qkg = torch::empty({tiles * 4 * 64 * dk}, x.options());
  auto ends = torch::empty({tiles * dk}, torch::dtype(torch::kFloat32).device(x.device()));
  for (int64_t t = 0; t < S; t += seg)
    done(mt_gla_chunks(x.data_ptr(), x.stride(0), log_alpha.data_ptr<float>(), (int)H, (int)dk, (int)dv, (int)S, (int)t, (int)std::min(S, t + seg), rp, sl, le,
                       nl, aa.data_ptr(), qkg.data_ptr(), ends.data_ptr<float>(), o.data_ptr(), (int)B, stream()), "gla_chunks", 2);
}

// out = rms(o) [* w] * silu(z), or sigmoid(z) with `sig`; z at column zoff + (h / r) * zstride + (h % r) * dv of x
void gated_head_norm(const Tensor& o, const Tensor& x, int64_t H, int64_t dv, int64_t r, int64_t zoff, int64_t zstride, const OptTensor& w, double eps,
                     Tensor& out, bool sig) {
  const bool f = f32(o);
  const int64_t N = x.size(0);
  rows2d(x, o, N, zoff + (H / r - 1) * zstride + r * dv, "packed projection");
  same(o, o, N * H * dv, "o"); same(out, o, N * H * dv, "out");
  if (w) same(*w, o, dv, "norm");
  c10::cuda::CUDAGuard guard(o.device());
  done(mt_gated_head_norm(f, o.data_ptr(), x.data_ptr(), x.stride(0), N * H, (int)H, (int)dv, (int)r, zoff, zstride, w ? w->data_ptr() : nullptr, (float)eps,
                          sig, out.data_ptr(), stream()), "gated_head_norm");
}

void check_fp32(const Tensor& t, int64_t numel, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kFloat32 && t.is_contiguous() && t.numel() == numel, what, ": contiguous fp32 tensor of ", numel,
              " elements expected");
}
const float* turns(const OptTensor& inv_ts, int64_t rot, int64_t dk) {
  TORCH_CHECK(rot >= 0 && rot % 2 == 0 && rot <= dk && bool(inv_ts) == (rot > 0), "retention: bad rotation");
  if (!inv_ts) return nullptr;
  check_fp32(*inv_ts, rot / 2, "inverse timescales");
  return inv_ts->data_ptr<float>();
}

// x rows: q H*dk | k H*dk | v H*dv | gate H*dv -> out [B, H * dv], normalised and gated
void retention_decode(const Tensor& x, const Tensor& log_decay, const OptTensor& inv_ts, int64_t rot, double eps, int64_t H, int64_t dk, int64_t dv, Tensor& rec,
                      const Tensor& slots, const Tensor& lengths, Tensor& out) {
  const bool f = f32(x);
  const int64_t B = x.size(0);
  rows2d(x, x, B, 2 * H * (dk + dv), "packed projection");
  check_fp32(log_decay, H, "log decay");
  same(out, x, B * H * dv, "out");
  float* rp = state(rec, {H, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_retention_decode(f, x.data_ptr(), x.stride(0), log_decay.data_ptr<float>(), turns(inv_ts, rot, dk), (int)rot, (float)eps, (int)H, (int)dk, (int)dv,
                           rp, longs(slots, B, "slots"), longs(lengths, B, "lengths"), out.data_ptr(), (int)B, stream()), "retention_decode");
}

// token scan, any widths up to 256: x rows as above -> o [B*S, H * dv]
void retention_scan(const Tensor& x, const Tensor& log_decay, const OptTensor& inv_ts, int64_t rot, int64_t H, int64_t dk, int64_t dv, int64_t S, Tensor& rec,
                    const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  const bool f = f32(x);
  const int64_t B = slots.numel();
  rows2d(x, x, B * S, 2 * H * (dk + dv), "packed projection");
  check_fp32(log_decay, H, "log decay");
  same(o, x, B * S * H * dv, "o");
  float* rp = state(rec, {H, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_retention_scan(f, x.data_ptr(), x.stride(0), log_decay.data_ptr<float>(), turns(inv_ts, rot, dk), (int)rot, (int)H, (int)dk, (int)dv, (int)S, rp,
                         longs(slots, B, "slots"), longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), o.data_ptr(), (int)B, stream()),
       "retention_scan");
}

// the chunked form of retention_scan (bf16)
void retention_chunks(const Tensor& x, const Tensor& log_decay, const OptTensor& inv_ts, int64_t rot, int64_t H, int64_t dk, int64_t dv, int64_t S, Tensor& rec,
                      const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& o) {
  TORCH_CHECK(!f32(x) && chunk_supported(dk, dv), "retention_chunks: bf16 and head widths of 16 .. 128 in steps of 16");
  const int64_t B = slots.numel();
  rows2d(x, x, B * S, 2 * H * (dk + dv), "packed projection");
  TORCH_CHECK((reinterpret_cast<uintptr_t>(x.data_ptr()) % 16) == 0 && x.stride(0) % 8 == 0);
  check_fp32(log_decay, H, "log decay");
  same(o, x, B * S * H * dv, "o");
  float* rp = state(rec, {H, dk, dv}, "rec");
  const int64_t *sl = longs(slots, B, "slots"), *le = longs(lengths, B, "lengths"), *nl = longs(new_lens, B, "new_lens");
  const float* iv = turns(inv_ts, rot, dk);
  c10::cuda::CUDAGuard guard(x.device());
  const int64_t seg = chunk_segment(B, H, S, 2 * 64 * 2 + 4 * dk * 2), tiles = B * (seg / 64) * H;
  auto aa = torch::empty({tiles * 2 * 64 * 64}, x.options()), qkg = torch::empty({tiles * 4 * 64 * dk}, x.options());
  auto ends = torch::empty({tiles * dk}, torch::dtype(torch::kFloat32).device(x.device()));
  for (int64_t t = 0; t < S; t += seg)
    done(mt_retention_chunks(x.data_ptr(), x.stride(0), log_decay.data_ptr<float>(), iv, (int)rot, (int)H, (int)dk, (int)dv, (int)S, (int)t,
                             (int)std::min(S, t + seg), rp, sl, le, nl, aa.data_ptr(), qkg.data_ptr(), ends.data_ptr<float>(), o.data_ptr(), (int)B, stream()),
         "retention_chunks", 2);
}

// x rows: q hk*dk | k hk*dk | v hv*dv; beta rows [B, >= hv]; da fp32 [B, hv*dk]; z rows [B, >= hv*dv] -> out [B, hv * dv], normalised and gated
void channel_delta_decode(const Tensor& x, const Tensor& beta, const Tensor& conv_w, const Tensor& da, const Tensor& A_log, const Tensor& dt_bias,
                          const Tensor& z, const Tensor& norm, double eps, int64_t hk, int64_t hv, int64_t dk, int64_t dv, Tensor& conv, Tensor& rec,
                          const Tensor& slots, const Tensor& lengths, Tensor& out) {
  const bool f = f32(x);
  const int64_t B = x.size(0), cd = 2 * hk * dk + hv * dv;
  TORCH_CHECK(hk > 0 && hv % hk == 0 && conv_w.dim() == 2 && conv_w.size(0) >= 1, "channel-wise gated delta: bad sizes");
  const int64_t taps = conv_w.size(0);
  rows2d(x, x, B, cd, "packed projection"); rows2d(beta, x, B, hv, "beta"); rows2d(z, x, B, hv * dv, "gate");
  same(conv_w, x, taps * cd, "convolution"); same(A_log, x, hv, "A_log"); same(dt_bias, x, hv * dk, "dt_bias"); same(norm, x, dv, "norm");
  same(out, x, B * hv * dv, "out");
  check_fp32(da, B * hv * dk, "decay");
  float* cp = state(conv, {taps - 1, cd}, "conv");
  float* rp = state(rec, {hv, dk, dv}, "rec");
  c10::cuda::CUDAGuard guard(x.device());
  done(mt_channel_delta_decode(f, x.data_ptr(), x.stride(0), beta.data_ptr(), beta.stride(0), conv_w.data_ptr(), (int)taps, da.data_ptr<float>(),
                               A_log.data_ptr(), dt_bias.data_ptr(), z.data_ptr(), z.stride(0), norm.data_ptr(), (float)eps, (int)hk, (int)hv, (int)dk, (int)dv,
                               cp, rp, longs(slots, B, "slots"), longs(lengths, B, "lengths"), out.data_ptr(), (int)B, stream()), "channel_delta_decode");
}

// mixed [B*S, 2 hk dk + hv dv] after the convolution -> o [B*S, hv * dv]; `chunked` (bf16, head widths of 16 .. 128 in steps of 16): in chunks of 64 tokens
void channel_delta_scan(const Tensor& mixed, const Tensor& beta, const Tensor& da, const Tensor& A_log, const Tensor& dt_bias, int64_t hk, int64_t hv,
                        int64_t dk, int64_t dv, int64_t S, Tensor& rec, const Tensor& slots, const Tensor& lengths, const OptTensor& new_lens, Tensor& o,
                        bool chunked) {
  const bool f = f32(mixed);
  const int64_t B = slots.numel(), cd = 2 * hk * dk + hv * dv;
  TORCH_CHECK(hk > 0 && hv % hk == 0, "channel-wise gated delta: bad sizes");
  same(mixed, mixed, B * S * cd, "mixed");
  rows2d(beta, mixed, B * S, hv, "beta");
  same(A_log, mixed, hv, "A_log"); same(dt_bias, mixed, hv * dk, "dt_bias"); same(o, mixed, B * S * hv * dv, "o");
  check_fp32(da, B * S * hv * dk, "decay");
  float* rp = state(rec, {hv, dk, dv}, "rec");
  const int64_t *sl = longs(slots, B, "slots"), *le = longs(lengths, B, "lengths"), *nl = longs(new_lens, B, "new_lens");
  c10::cuda::CUDAGuard guard(mixed.device());
  if (!chunked) {
    done(mt_channel_delta_scan(f, mixed.data_ptr(), beta.data_ptr(), beta.stride(0), da.data_ptr<float>(), A_log.data_ptr(), dt_bias.data_ptr(), (int)hk, (int)hv,
                               (int)dk, (int)dv, (int)S, rp, sl, le, nl, o.data_ptr(), (int)B, stream()), "channel_delta_scan");
    return;
  }
  TORCH_CHECK(!f && chunk_supported(dk, dv) && cd % 8 == 0 && (reinterpret_cast<uintptr_t>(mixed.data_ptr()) % 16) == 0, "channel_delta_scan: not chunkable");
  const int64_t seg = chunk_segment(B, hv, S, 4 * 64 * 2 + 6 * dk * 2), tiles = B * (seg / 64) * hv;
  auto tp = torch::empty({tiles * 4 * 64 * 64}, mixed.options()), qkg = torch::empty({tiles * 6 * 64 * dk}, mixed.options());
  auto fo = torch::dtype(torch::kFloat32).device(mixed.device());
  auto betas = torch::empty({tiles * 64}, fo), ends = torch::empty({tiles * dk}, fo);
  for (int64_t t = 0; t < S; t += seg)
    done(mt_channel_delta_chunks(mixed.data_ptr(), cd, beta.data_ptr(), beta.stride(0), da.data_ptr<float>(), A_log.data_ptr(), dt_bias.data_ptr(), (int)hk,
                                 (int)hv, (int)dk, (int)dv, (int)S, (int)t, (int)std::min(S, t + seg), rp, sl, le, nl, tp.data_ptr(), qkg.data_ptr(),
                                 betas.data_ptr<float>(), ends.data_ptr<float>(), o.data_ptr(), (int)B, stream()), "channel_delta_chunks", 2);
}

void mla_prep(const OptTensor& qa, const OptTensor& qw, const Tensor& kva, const Tensor& kw, double eps, const Tensor& pos, const Tensor& inv_ts,
              bool interleaved, const OptTensor& cq, Tensor& lat, Tensor& kr, Tensor& cache_lat, Tensor& cache_kr, const Tensor& slots, const Tensor& lengths,
              const OptTensor& new_lens) {
  const bool f = f32(kva);
  const int64_t N = kva.size(0), R = lat.size(1), dr = kr.size(1), B = slots.numel();
  TORCH_CHECK(B > 0 && N % B == 0 && dr % 2 == 0 && bool(qa) == bool(cq) && bool(qa) == bool(qw));
  rows2d(kva, kva, N, R + dr, "kv down-projection");
  same(kw, kva, R, "kv norm"); same(lat, kva, N * R, "latent"); same(kr, kva, N * dr, "rotated key");
  TORCH_CHECK(cache_lat.dim() == 3 && cache_lat.size(2) == R && cache_kr.dim() == 3 && cache_kr.size(2) == dr && cache_kr.size(1) == cache_lat.size(1));
  same(cache_lat, kva, cache_lat.numel(), "latent cache"); same(cache_kr, kva, cache_kr.numel(), "key cache");
  TORCH_CHECK(inv_ts.is_cuda() && inv_ts.scalar_type() == torch::kFloat32 && inv_ts.is_contiguous() && inv_ts.numel() >= dr / 2);
  int64_t Q = 0;
  if (qa) { Q = cq->size(1); rows2d(*qa, kva, N, Q, "q down-projection"); same(*qw, kva, Q, "q norm"); same(*cq, kva, N * Q, "query latent"); }
  c10::cuda::CUDAGuard guard(kva.device());
  done(mt_mla_prep(f, qa ? qa->data_ptr() : nullptr, qa ? qa->stride(0) : 0, qw ? qw->data_ptr() : nullptr, (int)Q, kva.data_ptr(), kva.stride(0),
                   kw.data_ptr(), (int)R, (int)dr, (float)eps, longs(pos, N, "positions"), inv_ts.data_ptr<float>(), interleaved, (int)(N / B),
                   cq ? cq->data_ptr() : nullptr, lat.data_ptr(), kr.data_ptr(), cache_lat.data_ptr(), cache_kr.data_ptr(), cache_lat.size(1),
                   longs(slots, B, "slots"), longs(lengths, B, "lengths"), longs(new_lens, B, "new_lens"), N, stream()), "mla_prep");
}

void mla_pack(const Tensor& q, const Tensor& kv, const Tensor& kr, const Tensor& pos, const Tensor& inv_ts, bool interleaved, int64_t nope, int64_t vd,
              Tensor& qp, Tensor& kp, Tensor& vp) {
  TORCH_CHECK(q.is_cuda() && q.scalar_type() == torch::kBFloat16 && q.dim() == 3 && qp.dim() == 3 && kp.dim() == 3 && vp.dim() == 3);
  const int64_t NQ = q.size(0), H = q.size(1), dr = q.size(2) - nope, NK = kr.size(0), DQ = qp.size(2), DV = vp.size(2);
  TORCH_CHECK(dr > 0 && dr % 2 == 0 && DQ >= nope + dr && DV >= vd && kp.size(2) == DQ);
  same(q, q, NQ * H * (nope + dr), "q"); same(kv, q, NK * H * (nope + vd), "kv"); same(kr, q, NK * dr, "kr");
  same(qp, q, NQ * H * DQ, "qp"); same(kp, q, NK * H * DQ, "kp"); same(vp, q, NK * H * DV, "vp");
  TORCH_CHECK(inv_ts.is_cuda() && inv_ts.scalar_type() == torch::kFloat32 && inv_ts.is_contiguous() && inv_ts.numel() >= dr / 2);
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_mla_pack(q.data_ptr(), kv.data_ptr(), kr.data_ptr(), longs(pos, NQ, "positions"), inv_ts.data_ptr<float>(), interleaved, NQ, NK, (int)H, (int)nope,
                   (int)dr, (int)vd, (int)DQ, (int)DV, qp.data_ptr(), kp.data_ptr(), vp.data_ptr(), stream()), "mla_pack", 2);
}

void mla_absorb(const Tensor& q, const Tensor& w, const Tensor& pos, const Tensor& inv_ts, bool interleaved, int64_t nope, int64_t vd, Tensor& qa) {
  const bool f = f32(q);
  TORCH_CHECK(q.dim() == 3 && qa.dim() == 3);
  const int64_t B = q.size(0), H = q.size(1), dr = q.size(2) - nope, R = qa.size(2) - dr;
  TORCH_CHECK(dr > 0 && dr % 2 == 0 && R > 0);
  same(q, q, B * H * (nope + dr), "q"); same(w, q, H * (nope + vd) * R, "wkv_b"); same(qa, q, B * H * (R + dr), "qa");
  TORCH_CHECK(inv_ts.is_cuda() && inv_ts.scalar_type() == torch::kFloat32 && inv_ts.is_contiguous() && inv_ts.numel() >= dr / 2);
  c10::cuda::CUDAGuard guard(q.device());
  done(mt_mla_absorb(f, q.data_ptr(), w.data_ptr(), longs(pos, B, "positions"), inv_ts.data_ptr<float>(), interleaved, (int)B, (int)H, (int)nope, (int)dr,
                     (int)vd, (int)R, qa.data_ptr(), stream()), "mla_absorb");
}

// splits of the key range that fill the machine without making parts shorter than one tile
int64_t mla_decode_splits(int64_t B, int64_t H, int64_t span) {
  const int64_t ctas = std::max<int64_t>(1, B * ((H + 15) / 16));
  return std::max<int64_t>(1, std::min<int64_t>({64, mt_num_sms() / ctas, (span + 63) / 64}));
}

void mla_decode_attn(const Tensor& qa, const Tensor& lat, const Tensor& kr, const Tensor& slots, const Tensor& lengths, double scale, int64_t window,
                     int64_t splits, Tensor& part, Tensor& ml) {
  const bool f = f32(qa);
  TORCH_CHECK(qa.dim() == 3 && lat.dim() == 3 && kr.dim() == 3 && lat.size(1) == kr.size(1) && lat.size(0) == kr.size(0));
  const int64_t B = qa.size(0), H = qa.size(1), R = lat.size(2), dr = kr.size(2);
  same(qa, qa, B * H * (R + dr), "qa"); same(lat, qa, lat.numel(), "latent cache"); same(kr, qa, kr.numel(), "key cache");
  TORCH_CHECK(part.is_cuda() && part.scalar_type() == torch::kFloat32 && part.is_contiguous() && part.numel() == B * H * splits * R);
  TORCH_CHECK(ml.is_cuda() && ml.scalar_type() == torch::kFloat32 && ml.is_contiguous() && ml.numel() == B * H * splits * 2);
  c10::cuda::CUDAGuard guard(qa.device());
  done(mt_mla_decode_attn(f, qa.data_ptr(), lat.data_ptr(), kr.data_ptr(), lat.size(1), longs(slots, B, "slots"), longs(lengths, B, "lengths"), (int)B, (int)H,
                          (int)R, (int)dr, (float)scale, (int)window, (int)splits, part.data_ptr<float>(), ml.data_ptr<float>(), stream()),
       "mla_decode_attn");
}

void mla_value_up(const Tensor& part, const Tensor& ml, const Tensor& w, int64_t nope, Tensor& out) {
  const bool f = f32(w);
  TORCH_CHECK(part.dim() == 4 && out.dim() == 3 && part.is_contiguous() && part.scalar_type() == torch::kFloat32);
  const int64_t B = part.size(0), H = part.size(1), splits = part.size(2), R = part.size(3), vd = out.size(2);
  TORCH_CHECK(ml.is_contiguous() && ml.scalar_type() == torch::kFloat32 && ml.numel() == B * H * splits * 2);
  same(w, w, H * (nope + vd) * R, "wkv_b"); same(out, w, B * H * vd, "out");
  c10::cuda::CUDAGuard guard(w.device());
  done(mt_mla_value_up(f, part.data_ptr<float>(), ml.data_ptr<float>(), w.data_ptr(), (int)B, (int)H, (int)nope, (int)vd, (int)R, (int)splits, out.data_ptr(),
                       stream()), "mla_value_up");
}

}  // namespace

void register_serving(pybind11::module_& m) {
  m.def("residual_norm", &residual_norm);
  m.def("residual_join", &residual_join);
  m.def("residual_gate", &residual_gate);
  m.def("act_rows", &act_rows);
  m.def("token_gate", &token_gate);
  m.def("act_fwd", &act_fwd);
  m.def("delta_decode", &delta_decode);
  m.def("delta_conv", &delta_conv);
  m.def("delta_scan", &delta_scan);
  m.def("gla_decode", &gla_decode);
  m.def("gla_decay", &gla_decay);
  m.def("gla_scan", &gla_scan);
  m.def("chunk_supported", &chunk_supported);
  m.def("delta_chunks", &delta_chunks);
  m.def("gla_chunks", &gla_chunks);
  using pybind11::arg;
  m.def("gated_head_norm", &gated_head_norm, arg("o"), arg("x"), arg("H"), arg("dv"), arg("r"), arg("zoff"), arg("zstride"), arg("w"), arg("eps"), arg("out"),
        arg("sig") = false);
  m.def("retention_decode", &retention_decode);
  m.def("retention_scan", &retention_scan);
  m.def("retention_chunks", &retention_chunks);
  m.def("channel_delta_decode", &channel_delta_decode);
  m.def("channel_delta_scan", &channel_delta_scan);
  m.def("mla_prep", &mla_prep);
  m.def("mla_pack", &mla_pack);
  m.def("mla_absorb", &mla_absorb);
  m.def("mla_decode_splits", &mla_decode_splits);
  m.def("mla_decode_attn", &mla_decode_attn);
  m.def("mla_value_up", &mla_value_up);
}
