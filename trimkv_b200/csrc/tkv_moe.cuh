// Mixture of experts: tokens are routed, the rows of every expert gathered into consecutive places, two grouped products run
// over them, and whoever consumes the result adds each token's rows up with their weights.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

// out[r, :] = act(a[src ? src[r] : r, :] . w[e]^T) for the rows r of expert e: offsets[e] .. offsets[e + 1).
struct GroupedGemm {
  const void* a; int64_t a_stride; int64_t a_rows;
  const int32_t* src;
  const void* w;                                          // [experts, n, k]
  const int32_t* offsets;                                 // [experts + 1], device
  void* out;                                              // [rows, n]
  int experts, n, k, act;                                 // act: 0 none, 1 GELU (erf)
  int64_t max_rows;                                       // host bound on offsets[experts]
  int32_t* status;
};

__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }

// Expert and first row of row tile `tile` when every expert's rows are cut into tiles of `rows` (the last one short): tiles are
// counted expert by expert.  False beyond the last tile.
__device__ __forceinline__ bool find_tile(const int32_t* offsets, int experts, int rows, int tile, int* expert, int* row0) {
  int at = 0;
  for (int e = 0; e < experts; ++e) {
    const int n = (offsets[e + 1] - offsets[e] + rows - 1) / rows;
    if (tile < at + n) {
      *expert = e;
      *row0 = offsets[e] + (tile - at) * rows;
      return true;
    }
    at += n;
  }
  return false;
}

bool moe_tc_shape(const GroupedGemm& p, int dtype);       // tcgen05 (tkv_moe_tc.cu)
int launch_moe_tc(const GroupedGemm& p, cudaStream_t st);

}  // namespace tkv
