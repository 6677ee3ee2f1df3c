// Linear recurrences with one decay per head and token: S_t = a_t S_(t-1) + k_t (s_t v_t)^T, o_t = S_t^T q_t + d v_t.
// Retention has a constant a per head and s = 1, d = 0; the state-space layers (SSD) have a_t = exp(-A dt_t), s_t = dt_t,
// k and q shared by the heads of a group, and a skip weight d per head.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

struct LinrecParams {
  const void* q; int64_t q_stride;      // element strides between tokens; head h reads columns [(h / (heads/groups)) * n, + n)
  const void* k; int64_t k_stride;
  const void* v; int64_t v_stride;      // head h reads columns [h * p, + p)
  const float* log_decay;               // [tokens, heads] logarithm of a, or NULL: head_decay / head_log_decay
  const float* head_decay;              // [heads]
  const float* head_log_decay;          // [heads]
  const float* v_scale;                 // [tokens, heads] or NULL (1)
  const float* skip;                    // [heads] or NULL (0)
  void* out;                            // [tokens, heads * p], model type
  float* state;                         // [slots, heads, n, p] fp32
  const int32_t* slots; const int32_t* cu; const int32_t* pos0;   // [batch], [batch + 1] or NULL (one token each), [batch]
  int batch, heads, groups, n, p;
};

}  // namespace tkv
