// Arguments of the gated residual step (residual_norm.cu), shared with its binding.
#pragma once

namespace mt {

struct ResidualGate {
  float* x;                            // fp32 stream [rows, D]
  const void* rows;                    // branch rows [n_rows, D] or null
  const int* dest;                     // numbers of a token's rows, or null: t * per_token ..
  long n_rows;
  int per_token;
  const void* extra;                   // [rows, D] or null: added to the branch
  const void* gate;                    // gate logits [rows, ldg] or null ...
  long ldg;
  const void* bias;                    // ... and their bias [D]
  const void *w_post, *w_next;         // norm weights [D]; w_next null: y is x itself
  void* y;                             // [rows, ldy] or null
  long ldy;
  float eps;
  int centred, fresh;
};

}  // namespace mt
