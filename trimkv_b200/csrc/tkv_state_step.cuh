// One-token state update of a linear recurrence, shared by its one-token kernels.
#pragma once
#include "tkv_elem.cuh"

namespace tkv {

constexpr int kStepThreads = 256;

// S <- diag(decay) S + k v^T and o = S^T q for one head: S [n, p] fp32 in global memory, k / q [n], v [p], o [p] in shared
// memory.  Threads cover columns in vectors of V and rows in an interleaved fashion.  The first rows are requested by
// `prefetch` before the step's k, q, v are known, so that their latency overlaps the producers' work.
template <int V> struct StateStep {
  static constexpr int U = 8;
  float* S; int n, p, nc, cb, rg, r, c0; bool fresh;
  float s[U][V];

  __device__ __forceinline__ void load(int row, int c) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int rr = row + u * rg;
      if (rr < n && !fresh) {
        if constexpr (V == 4) {
          const float4 x = *reinterpret_cast<const float4*>(S + (int64_t)rr * p + c * V);
          s[u][0] = x.x; s[u][1] = x.y; s[u][2] = x.z; s[u][3] = x.w;
        } else {
          s[u][0] = S[(int64_t)rr * p + c];
        }
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) s[u][e] = 0.f;
      }
    }
  }
  __device__ __forceinline__ void prefetch(float* S_, int n_, int p_, bool fresh_) {
    S = S_; n = n_; p = p_; fresh = fresh_;
    nc = p / V; cb = min(nc, kStepThreads); rg = kStepThreads / cb;
    r = threadIdx.x / cb; c0 = threadIdx.x - r * cb;
    if (r < rg) load(r, c0);
  }
  // All threads of the CTA call it; k, q, v must be visible (a barrier before), o is visible on return.  decay(row): the
  // factor of a row of the state.  red holds kStepThreads * V floats.
  template <typename Decay>
  __device__ __forceinline__ void run(Decay decay, const float* k, const float* q, const float* v, float* o, float* red) {
    const bool active = r < rg;
    for (int cbase = 0; cbase < nc; cbase += cb) {
      const int c = cbase + c0;
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = 0.f;
      if (active && c < nc) {
        float vv[V];
#pragma unroll
        for (int e = 0; e < V; ++e) vv[e] = v[c * V + e];
        for (int row = r; row < n; row += rg * U) {
          if (row != r || cbase != 0) load(row, c);
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int rr = row + u * rg;
            if (rr < n) {
              const float a = decay(rr), kk = k[rr], qq = q[rr];
#pragma unroll
              for (int e = 0; e < V; ++e) {
                s[u][e] = fmaf(a, s[u][e], kk * vv[e]);
                acc[e] = fmaf(qq, s[u][e], acc[e]);
              }
              if constexpr (V == 4)
                *reinterpret_cast<float4*>(S + (int64_t)rr * p + c * V) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
              else
                S[(int64_t)rr * p + c] = s[u][0];
            }
          }
        }
      }
      if (active) {
#pragma unroll
        for (int e = 0; e < V; ++e) red[(r * cb + c0) * V + e] = acc[e];
      }
      __syncthreads();
      for (int i = threadIdx.x; i < cb * V && cbase * V + i < p; i += kStepThreads) {
        float a = 0.f;
        for (int g = 0; g < rg; ++g) a += red[g * cb * V + i];
        o[cbase * V + i] = a;
      }
      __syncthreads();
    }
  }
};

// Raises a kernel's dynamic shared memory limit (once per kernel and size); false if the size is out of reach.
template <typename K> inline bool allow_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return true;
  if (bytes > 220 * 1024) return false;
  return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}
}  // namespace tkv
