// Parameters shared by the differential-attention kernels (storage and masks: tkv_diffattn.cu).
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

struct DiffAttnParams {
  const void* q;                                          // [tokens, heads, 2, dp]
  const void* k_ring; const void* v_ring; int ring_rows;  // decode
  const void* k_lin; const void* v_lin; const int32_t* kv_start;   // prompts: first linear row of every request
  const int32_t* cu; const int32_t* slots; const int32_t* pos0;
  const float* lambda; float diff, scale, scale_log2, eps;
  const void* gate; int64_t gate_stride;                  // [tokens, heads] within a wider row
  void* out;                                              // [tokens, heads, vdim]
  float* part_o; float* part_ml;                          // split-KV partials
  int batch, tokens, heads, kv_heads, dim, vdim, dp, pp, window, chunk;
  int32_t* status;
};

int launch_diff_any(const DiffAttnParams& p, int dtype, cudaStream_t st);
int launch_diff_prefill_tc(const DiffAttnParams& p, int64_t kv_rows, int max_tokens, cudaStream_t st);

}  // namespace tkv
