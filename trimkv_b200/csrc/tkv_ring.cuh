// Windows of keys and values: ring storage (position p in row p mod rows) and the linear buffers of a step of several tokens.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

constexpr int kFetchThreads = 128;

// The positions before a request's step that its window still reaches, from the ring into the linear buffers: rows of kp
// elements of k and pp of v (0: none), multiples of 16 bytes.  One warp
// per (history row, kv head); grid.y = request.
template <typename T>
__global__ void __launch_bounds__(kFetchThreads) ring_fetch_kernel(const T* k_ring, const T* v_ring, int ring_rows, T* k_lin, T* v_lin,
                                                                 const int32_t* kv_start, const int32_t* slots,
                                                                 const int32_t* pos0, int kv_heads, int kp, int pp, int window) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = threadIdx.x & 31, b = blockIdx.y;
  const int hist = min(pos0[b], window - 1);
  const int item = blockIdx.x * (kFetchThreads / 32) + (threadIdx.x >> 5);
  const int r = item / kv_heads, g = item - r * kv_heads;
  if (r >= hist) return;
  const int64_t src = ((int64_t)slots[b] * kv_heads + g) * ring_rows + (pos0[b] - hist + r) % ring_rows;
  const int64_t dst = ((int64_t)kv_start[b] + r) * kv_heads + g;
  constexpr int kPer = 16 / (int)sizeof(T);
  for (int i = lane * kPer; i < kp; i += 32 * kPer) st16(k_lin + dst * kp + i, ld16(k_ring + src * kp + i));
  for (int i = lane * kPer; i < pp; i += 32 * kPer) st16(v_lin + dst * pp + i, ld16(v_ring + src * pp + i));
}

}  // namespace tkv
