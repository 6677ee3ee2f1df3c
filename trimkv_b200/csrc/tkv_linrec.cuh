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

// A long sequence cut into segments that run side by side: a first pass computes every segment's own state, a small kernel
// chains them, the main pass starts each segment from its true state.
struct LinrecSegs {
  int count, tokens;                                      // segments per request, tokens per segment
  float* start;                                           // [batch, heads, count, n, p]
  float* log_sum;                                         // [batch, heads, count], log2
};

int launch_linrec_chain(const LinrecParams& a, const LinrecSegs& sg, cudaStream_t st);
// The tcgen05 form (tkv_linrec_tc.cu): shapes it takes, and its segments.
bool linrec_tc_shape(int n, int p, int max_tokens, int64_t tokens);
LinrecSegs linrec_tc_segments(int batch, int max_tokens, int heads, int p);
int launch_linrec_tc(const LinrecParams& a, const LinrecSegs& sg, int64_t tokens, int32_t* status, cudaStream_t st);

}  // namespace tkv
