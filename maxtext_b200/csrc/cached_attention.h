// Arguments that the attention kernels over the cache (cached_attention_sm100.cu) share with their bindings.
#pragma once
#include <stdint.h>

namespace mt {
namespace cattn {

enum { NORM_NONE = 0, NORM_AFTER = 1, NORM_HEAD = 2, NORM_ALL = 3 };

struct PrepArgs {
  const void *q, *k, *v;               // projection rows
  long ldq, ldk, ldv;
  const void *bq, *bk, *bv;            // biases or null
  const void *wq, *wk;                 // norm weights (NORM_HEAD: one head, NORM_ALL: the whole projection)
  int H, G, D, Dv, maps, norm;
  const int64_t* pos;
  const float* inv_ts;
  int rot, paired;                     // rotated lanes; paired: neighbouring lanes turn together
  float eps, temp_coef, temp_every;    // temp_every 0: no query temperature
  int S;
  void *qp, *kp, *vp;                  // q [N, H * maps, dq]; k [N, G, dq] and v [N, G, dvp] or null
  int dq, dvp;
  void *kc, *vc;                       // cache [slots, max_len, G, maps * D], [.., Dv]
  long max_len;
  const int64_t *slots, *lengths, *new_lens;
  const void* talk;                    // [H, H] or null: the heads' scores are mixed by this matrix. Then qp is [N, H, G * D]: a query over the keys of
                                       // all key heads side by side (dq = G * D, no operand padding, one map)
};

// differential attention: lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
struct DiffArgs {
  const void *lq1, *lk1, *lq2, *lk2;   // [D]
  int D;
  float diff, eps;
};

}  // namespace cattn
}  // namespace mt
