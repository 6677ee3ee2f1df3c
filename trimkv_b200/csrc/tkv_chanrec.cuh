// Linear recurrences with one decay per state row (channel of q) and token, in which the forget gate also writes:
//   f = lower + (1 - lower) sigmoid(z_f + bias),  S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,  o_t = S_t^T silu(z_q).
// The gate, its complement and the state are fp32 whatever the type of the projections z_q, z_f, v.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

struct ChanrecParams {
  const void* q; const void* f; const void* v;        // [tokens, heads * n], same, [tokens, heads * p]: columns of projection rows
  int64_t row_stride;                                 // of all three, in elements
  const float* f_bias; const float* lower;            // [heads * n]
  void* out;                                          // [tokens, heads * p], model type
  float* state;                                       // [slots, heads, n, p] fp32
  const int32_t* slots; const int32_t* cu; const int32_t* pos0;
  int batch, heads, n, p;
};

// f and 1 - f, each to fp32 accuracy (1 - f is (1 - lower) sigmoid(-x), not a difference).
__device__ __forceinline__ void forget_gate(float x, float lower, float* f, float* k) {
  const float e = expf(-fabsf(x)), r = 1.0f / (1.0f + e);
  const float big = r, small = e * r;                 // sigmoid(|x|), sigmoid(-|x|)
  *f = fmaf(1.0f - lower, x >= 0.f ? big : small, lower);
  *k = (1.0f - lower) * (x >= 0.f ? small : big);
}

// A long sequence cut into segments that run side by side (see LinrecSegs), with a decay per state row.  The pass over states
// alone, which leaves the last segment out, cuts each segment into pieces of its own, so that it too fills the GPU.
struct ChanrecSegs {
  int count, tokens, pieces;                          // segments per request, tokens per segment, pieces per segment
  float* start;                                       // [batch, heads, count * pieces, n, p]
  float* decay;                                       // [batch, heads, count * pieces, n]: product of f over the piece
};

int launch_chanrec_chain(const ChanrecParams& a, const ChanrecSegs& sg, cudaStream_t st);
// The tcgen05 form (tkv_chanrec_tc.cu): shapes it takes, value columns of a CTA.
bool chanrec_tc_shape(int n, int p, int max_tokens);
int chanrec_tc_columns();
int launch_chanrec_tc(const ChanrecParams& a, const ChanrecSegs& sg, int32_t* status, cudaStream_t st);

}  // namespace tkv
