// Element access for kernels that run in the model's 16-bit type or in true fp32: vectors of V elements as fp32.
#pragma once
#include "tkv_common.cuh"

namespace tkv {

template <typename T> __device__ __forceinline__ float to_f32(T x);
template <> __device__ __forceinline__ float to_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T> __device__ __forceinline__ T from_f32(float x);
template <> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }
// The value as the model's type would hold it.
template <typename T> __device__ __forceinline__ float round_as(float x) { return to_f32<T>(from_f32<T>(x)); }

// V = 8 (addresses 16-byte aligned) or 1 (no alignment assumed).
template <int V> __device__ __forceinline__ void load_vec(const float* p, float* v) {
  if constexpr (V == 1) {
    v[0] = p[0];
  } else {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(p + i);
      v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
    }
  }
}
template <int V> __device__ __forceinline__ void store_vec(float* p, const float* v) {
  if constexpr (V == 1) {
    p[0] = v[0];
  } else {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  }
}
template <int V> __device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float* v) {
  if constexpr (V == 1) {
    v[0] = __bfloat162float(p[0]);
  } else {
    const uint4 r = ld16(p);
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { v[2 * i] = __uint_as_float(w[i] << 16); v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
  }
}
template <int V> __device__ __forceinline__ void store_vec(__nv_bfloat16* p, const float* v) {
  if constexpr (V == 1) {
    p[0] = __float2bfloat16_rn(v[0]);
  } else {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      w[i] = *reinterpret_cast<const uint32_t*>(&h);
    }
    st16(p, make_uint4(w[0], w[1], w[2], w[3]));
  }
}

__device__ __forceinline__ float warp_add(float x) {
#pragma unroll
  for (int o = 16; o >= 1; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
  return x;
}
// Sum over a block of kThreads; `red` holds kThreads / 32 floats and may be reused after the next __syncthreads().
template <int kThreads> __device__ __forceinline__ float block_add(float x, float* red) {
  x = warp_add(x);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = x;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) t += red[i];
  return t;
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// SiLU and GELU of values that are then used in the model type: full precision for fp32 models, the hardware's exponential
// and division (errors far below a 16-bit rounding) for 16-bit ones.
template <typename T> __device__ __forceinline__ float silu_act(float x) {
  if constexpr (sizeof(T) == 4) return silu_f32(x);
  else return __fdividef(x, 1.0f + __expf(fminf(-x, 80.f)));
}
template <typename T> __device__ __forceinline__ float gelu_tanh_act(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  if constexpr (sizeof(T) == 4) return 0.5f * z * (1.0f + tanhf(u));
  else return __fdividef(z, 1.0f + __expf(fminf(-2.0f * u, 80.f)));      // (1 + tanh u) / 2 = 1 / (1 + e^(-2u))
}

// sin and cos of pos * (f_hi + f_lo): the fp32 product's rounding error and the frequency's low part are carried as a
// first-order correction, so that the angle keeps its accuracy at large positions.
__device__ __forceinline__ void turn(int pos, float f_hi, float f_lo, float* s, float* c) {
  const float p = (float)pos;
  const float a = p * f_hi;
  const float e = fmaf(p, f_hi, -a) + p * f_lo;
  float s0, c0;
  sincosf(a, &s0, &c0);
  *s = fmaf(c0, e, s0);
  *c = fmaf(-s0, e, c0);
}

// Request that owns packed row t: largest b with cu[b] <= t (cu == nullptr: one row per request).
__device__ __forceinline__ int owner_of(const int32_t* cu, int batch, int t) {
  if (cu == nullptr) return t;
  int lo = 0, hi = batch;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid;
  }
  return lo;
}

inline bool is_model_dtype(int dtype) { return dtype == TKV_BF16 || dtype == TKV_F32; }

}  // namespace tkv

// Runs `body` with the C++ element type of a run-time dtype code bound to `T`.
#define TKV_WITH_TYPE(dtype, T, ...)                              \
  do {                                                            \
    if ((dtype) == TKV_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
    else { using T = float; __VA_ARGS__; }                        \
  } while (0)
