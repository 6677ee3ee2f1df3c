// The residual stream of decoders that keep it in fp32 and norm the OUTPUT of a sublayer, and the elementwise steps
// around their products:
//   embed_stream_kernel  : token rows of the embedding as fp32 stream + its copy in the model type;
//   postnorm_add_kernel  : stream += mult * RMSNorm(y) * (w_offset + w), and the copy the next product reads;
//   gated_sum_norm_kernel: stream = group RMSNorm(alpha * stream + sigmoid(g + b) * y) * w and that copy; y may be a
//                          weighted sum of expert outputs (and of the stream itself), gathered here;
//   stream_norm_kernel   : (group) RMSNorm of the stream itself (before the output projection);
//   gated_norm_kernel    : group RMSNorm, a SiLU gate before or after it or none, optional weight;
//   swiglu_kernel        : silu(gate) * up of one projection row;
//   gelu_tanh_kernel     : the tanh form of GELU, in place;
//   batch_begin_kernel   : start positions of a step's requests, and the lengths after it.
// All statistics are fp32.  Every kernel runs for the 16-bit model type and for fp32.
#include <type_traits>
#include "tkv_elem.cuh"

namespace tkv {

constexpr int kRowThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) embed_stream_kernel(const int64_t* ids, const T* table, int64_t vocab, float* x,
                                                                  T* copy, int width, float scale, int32_t* status) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int64_t row = blockIdx.x;
  int64_t id = ids[row];
  if (id < 0 || id >= vocab) {          // reported, and the row reads as zeros
    if (threadIdx.x == 0) report(status, TKV_DEV_BAD_INDEX);
    id = -1;
  }
  for (int c = threadIdx.x * V; c < width; c += kRowThreads * V) {
    float v[V];
    if (id >= 0) load_vec<V>(table + id * width + c, v);
    else
      for (int i = 0; i < V; ++i) v[i] = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= scale;
    store_vec<V>(x + row * width + c, v);
    if (copy != nullptr) store_vec<V>(copy + row * width + c, v);
  }
}

// One CTA per row.  Rows of up to kRowThreads * kKeep vectors stay in registers between the two passes.
template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) postnorm_add_kernel(float* x, const T* y, const float* w, T* copy, int width,
                                                                  float eps, float mult, float w_offset) {
  constexpr int kKeep = V == 8 ? 2 : 8;
  __shared__ float red[kRowThreads / 32];
  const int64_t off = (int64_t)blockIdx.x * width;
  const int nvec = width / V;
  const bool keep = nvec <= kRowThreads * kKeep;
  float yv[kKeep][V], xv[kKeep][V];
  float ss = 0.f;
  grid_dependency_wait();
  grid_launch_dependents();
  if (keep) {
#pragma unroll
    for (int j = 0; j < kKeep; ++j) {
      const int i = threadIdx.x + j * kRowThreads;
      if (i < nvec) {
        load_vec<V>(y + off + (int64_t)i * V, yv[j]);
        load_vec<V>(x + off + (int64_t)i * V, xv[j]);
#pragma unroll
        for (int e = 0; e < V; ++e) ss += yv[j][e] * yv[j][e];
      }
    }
  } else {
    for (int i = threadIdx.x; i < nvec; i += kRowThreads) {
      float a[V];
      load_vec<V>(y + off + (int64_t)i * V, a);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += a[e] * a[e];
    }
  }
  const float rstd = mult / sqrtf(block_add<kRowThreads>(ss, red) / (float)width + eps);
  auto finish = [&](int i, const float* a, const float* r) {
    float g[V], o[V];
    load_vec<V>(w + (int64_t)i * V, g);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = r[e] + a[e] * rstd * (w_offset + g[e]);
    store_vec<V>(x + off + (int64_t)i * V, o);
    if (copy != nullptr) store_vec<V>(copy + off + (int64_t)i * V, o);
  };
  if (keep) {
#pragma unroll
    for (int j = 0; j < kKeep; ++j) {
      const int i = threadIdx.x + j * kRowThreads;
      if (i < nvec) finish(i, yv[j], xv[j]);
    }
  } else {
    for (int i = threadIdx.x; i < nvec; i += kRowThreads) {
      float a[V], r[V];
      load_vec<V>(y + off + (int64_t)i * V, a);
      load_vec<V>(x + off + (int64_t)i * V, r);
      finish(i, a, r);
    }
  }
}

// Sums of squares of a row's groups.  A thread adds its share of group g (`share(g)`); the result of group g is read back
// with total(g) after the barrier inside.  red: groups * kRowThreads / 32 floats.
template <typename F> __device__ __forceinline__ void group_sums(int groups, float* red, F share) {
  constexpr int kWarps = kRowThreads / 32;
  for (int g = 0; g < groups; ++g) {
    const float x = warp_add(share(g));
    if ((threadIdx.x & 31) == 0) red[g * kWarps + (threadIdx.x >> 5)] = x;
  }
  __syncthreads();
}
__device__ __forceinline__ float group_total(const float* red, int g) {
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRowThreads / 32; ++i) t += red[g * (kRowThreads / 32) + i];
  return t;
}

// One CTA per row.  x <- RMS over each of `groups` equal parts of (alpha x + gate y) times w, gate = sigmoid(g + b) or 1.
// kRouted: y = sum over the row's `top` choices of choice_w * (place >= 0 ? y[place] : x), place < 0 standing for an
// expert that returns its input.  kKeep vectors per thread stay in registers between the passes; kKeep = 0: in shared memory.
struct GatedSumNorm {
  float* x; const void* y; const void* gate; int64_t gate_stride; const float* gate_bias; const float* w; void* copy;
  const int32_t* place; const float* choice_w; int top;
  int width, groups; float eps, alpha;
};

template <typename T, int V, int kKeep, bool kRouted>
__global__ void __launch_bounds__(kRowThreads) gated_sum_norm_kernel(GatedSumNorm p) {
  extern __shared__ float dyn[];                          // red [groups][warps], then (kKeep = 0) the row
  constexpr int kN = kKeep > 0 ? kKeep : 1, kAhead = V == 8 ? 4 : 2;
  const int64_t row = blockIdx.x, off = row * p.width;
  const int nvec = p.width / V, glen = p.width / p.groups;
  float* held = dyn + p.groups * (kRowThreads / 32);
  float sv[kN][V];
  grid_dependency_wait();
  grid_launch_dependents();
  auto value = [&](int i, float* s) {                      // alpha x + gate y of vector i
    float xv[V], yv[V];
    load_vec<V>(p.x + off + (int64_t)i * V, xv);
    if (kRouted) {
#pragma unroll
      for (int e = 0; e < V; ++e) yv[e] = 0.f;
      for (int c0 = 0; c0 < p.top; c0 += kAhead) {         // kAhead rows requested before the first is used
        float r[kAhead][V], cw[kAhead];
        int32_t at[kAhead];
#pragma unroll
        for (int c = 0; c < kAhead; ++c) {
          at[c] = c0 + c < p.top ? p.place[row * p.top + c0 + c] : -1;
          cw[c] = c0 + c < p.top ? p.choice_w[row * p.top + c0 + c] : 0.f;
        }
#pragma unroll
        for (int c = 0; c < kAhead; ++c)
          if (at[c] >= 0) load_vec<V>((const T*)p.y + (int64_t)at[c] * p.width + (int64_t)i * V, r[c]);
#pragma unroll
        for (int c = 0; c < kAhead; ++c)
#pragma unroll
          for (int e = 0; e < V; ++e) yv[e] = fmaf(cw[c], at[c] >= 0 ? r[c][e] : xv[e], yv[e]);
      }
    } else {
      load_vec<V>((const T*)p.y + off + (int64_t)i * V, yv);
    }
    if (p.gate != nullptr) {
      float gv[V], bv[V];
      load_vec<V>((const T*)p.gate + row * p.gate_stride + (int64_t)i * V, gv);
      load_vec<V>(p.gate_bias + (int64_t)i * V, bv);
#pragma unroll
      for (int e = 0; e < V; ++e) yv[e] *= sigmoid_f32(gv[e] + bv[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) s[e] = fmaf(p.alpha, xv[e], yv[e]);
  };
  if (kKeep > 0) {
#pragma unroll
    for (int j = 0; j < kN; ++j) {
      const int i = threadIdx.x + j * kRowThreads;
      if (i < nvec) value(i, sv[j]);
    }
  } else {
    for (int i = threadIdx.x; i < nvec; i += kRowThreads) {
      value(i, sv[0]);
#pragma unroll
      for (int e = 0; e < V; ++e) held[i * V + e] = sv[0][e];
    }
  }
  // Where a group is made of whole rounds of a warp, a round's sum belongs to one group: entry j * warps + warp, in order.
  const bool whole = kKeep > 0 && glen % (32 * V) == 0;
  if (whole) {
#pragma unroll
    for (int j = 0; j < kN; ++j) {
      float ss = 0.f;
      if (threadIdx.x + j * kRowThreads < nvec)
#pragma unroll
        for (int e = 0; e < V; ++e) ss += sv[j][e] * sv[j][e];
      ss = warp_add(ss);
      if ((threadIdx.x & 31) == 0) dyn[j * (kRowThreads / 32) + (threadIdx.x >> 5)] = ss;
    }
    __syncthreads();
  } else group_sums(p.groups, dyn, [&](int g) {            // a vector lies in one group (the host chooses V so)
    float ss = 0.f;
    if (kKeep > 0) {
#pragma unroll
      for (int j = 0; j < kN; ++j) {
        const int i = threadIdx.x + j * kRowThreads;
        if (i < nvec && (p.groups == 1 || i * V / glen == g))
#pragma unroll
          for (int e = 0; e < V; ++e) ss += sv[j][e] * sv[j][e];
      }
    } else {
      for (int i = threadIdx.x; i < nvec; i += kRowThreads)
        if (i * V / glen == g)
#pragma unroll
          for (int e = 0; e < V; ++e) ss += held[i * V + e] * held[i * V + e];
    }
    return ss;
  });
  auto finish = [&](int i, const float* s) {
    const int g = p.groups == 1 ? 0 : i * V / glen;
    float total = 0.f;
    if (whole) for (int m = g * (glen / (32 * V)); m < (g + 1) * (glen / (32 * V)); ++m) total += dyn[m];
    else total = group_total(dyn, g);
    const float rstd = 1.0f / sqrtf(total / (float)glen + p.eps);
    float o[V];
    load_vec<V>(p.w + (int64_t)i * V, o);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] *= s[e] * rstd;
    store_vec<V>(p.x + off + (int64_t)i * V, o);
    if (p.copy != nullptr) store_vec<V>((T*)p.copy + off + (int64_t)i * V, o);
  };
  if (kKeep > 0) {
#pragma unroll
    for (int j = 0; j < kN; ++j) {
      const int i = threadIdx.x + j * kRowThreads;
      if (i < nvec) finish(i, sv[j]);
    }
  } else {
    for (int i = threadIdx.x; i < nvec; i += kRowThreads) {
#pragma unroll
      for (int e = 0; e < V; ++e) sv[0][e] = held[i * V + e];
      finish(i, sv[0]);
    }
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) stream_norm_kernel(const float* x, const int32_t* rows, const float* w, T* out,
                                                                 int width, int groups, float eps, float w_offset) {
  extern __shared__ float red[];                          // [groups][warps]
  grid_dependency_wait();
  grid_launch_dependents();
  const float* src = x + (int64_t)(rows != nullptr ? rows[blockIdx.x] : (int)blockIdx.x) * width;
  const int glen = width / groups;
  group_sums(groups, red, [&](int g) {
    float ss = 0.f;
    for (int c = g * glen + threadIdx.x * V; c < (g + 1) * glen; c += kRowThreads * V) {
      float a[V];
      load_vec<V>(src + c, a);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += a[e] * a[e];
    }
    return ss;
  });
  for (int c = threadIdx.x * V; c < width; c += kRowThreads * V) {
    const float rstd = 1.0f / sqrtf(group_total(red, c / glen) / (float)glen + eps);
    float a[V], g[V];
    load_vec<V>(src + c, a);
    load_vec<V>(w + c, g);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = a[e] * rstd * (w_offset + g[e]);
    store_vec<V>(out + (int64_t)blockIdx.x * width + c, a);
  }
}

// kLanes lanes per (row, group) of `len` elements.  gate_first: RMS(y * silu(z)) * w, else RMS(y) * w * silu(z); z may be
// NULL (no gate).  w has one weight per channel, or (w_shared) one set of `len` for all groups.
template <typename T, int V, int kLanes>
__global__ void __launch_bounds__(kRowThreads) gated_norm_kernel(const T* y, int64_t y_stride, const T* z, int64_t z_stride,
                                                                const float* w, int w_shared, T* out, int rows, int groups,
                                                                int len, float eps, int gate_first) {
  constexpr int kKeep = V == 8 ? 2 : 4;          // vectors per lane held in registers
  const int lane = threadIdx.x & (kLanes - 1);
  const int64_t items = (int64_t)rows * groups;
  const int64_t item_rt = (int64_t)blockIdx.x * (kRowThreads / kLanes) + threadIdx.x / kLanes;
  const bool live = item_rt < items;             // the rest of a warp takes part in its shuffles
  const int64_t item = live ? item_rt : items - 1;
  grid_dependency_wait();
  grid_launch_dependents();
  const int64_t row = item / groups;
  const int grp = (int)(item - row * groups);
  const T* yr = y + row * y_stride + (int64_t)grp * len;
  const bool has_gate = z != nullptr;
  const T* zr = has_gate ? z + row * z_stride + (int64_t)grp * len : yr;
  T* o = out + (row * groups + grp) * (int64_t)len;
  const int nvec = len / V;
  float a[kKeep][V], g[kKeep][V], ss = 0.f;
  auto gate = [&](float* av, float* gv) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      gv[e] = has_gate ? silu_act<T>(gv[e]) : 1.0f;
      if (gate_first) av[e] *= gv[e];
      ss += av[e] * av[e];
    }
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (lane + kLanes * j < nvec) {
      load_vec<V>(yr + (int64_t)(lane + kLanes * j) * V, a[j]);
      if (has_gate) load_vec<V>(zr + (int64_t)(lane + kLanes * j) * V, g[j]);
    }
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (lane + kLanes * j < nvec) gate(a[j], g[j]);
  for (int i = lane + kLanes * kKeep; i < nvec; i += kLanes) {
    float av[V], gv[V];
    load_vec<V>(yr + (int64_t)i * V, av);
    if (has_gate) load_vec<V>(zr + (int64_t)i * V, gv);
    gate(av, gv);
  }
#pragma unroll
  for (int d = kLanes / 2; d >= 1; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  const float rstd = 1.0f / sqrtf(ss / (float)len + eps);
  if (!live) return;
  auto finish = [&](int i, float* av, const float* gv) {
    float wv[V];
    if (w != nullptr) load_vec<V>(w + (w_shared ? 0 : (int64_t)grp * len) + (int64_t)i * V, wv);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      av[e] *= rstd;
      if (w != nullptr) av[e] *= wv[e];
      if (!gate_first) av[e] *= gv[e];
    }
    store_vec<V>(o + (int64_t)i * V, av);
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (lane + kLanes * j < nvec) finish(lane + kLanes * j, a[j], g[j]);
  for (int i = lane + kLanes * kKeep; i < nvec; i += kLanes) {
    float av[V], gv[V];
    load_vec<V>(yr + (int64_t)i * V, av);
    if (has_gate) load_vec<V>(zr + (int64_t)i * V, gv);
    const float keep = ss;
    gate(av, gv);
    ss = keep;
    finish(i, av, gv);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) gelu_tanh_kernel(T* u, int64_t n) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int64_t nvec = n / V;
  for (int64_t i = (int64_t)blockIdx.x * kRowThreads + threadIdx.x; i < nvec; i += (int64_t)gridDim.x * kRowThreads) {
    float a[V];
    load_vec<V>(u + i * V, a);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = gelu_tanh_act<T>(a[e]);
    store_vec<V>(u + i * V, a);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) swiglu_kernel(const T* u, int64_t u_stride, T* out, int64_t rows, int ff) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int per = ff / V;
  const int64_t n = rows * per;
  for (int64_t i = (int64_t)blockIdx.x * kRowThreads + threadIdx.x; i < n; i += (int64_t)gridDim.x * kRowThreads) {
    const int64_t r = i / per;
    const int c = (int)(i - r * per) * V;
    float a[V], b[V];
    load_vec<V>(u + r * u_stride + c, a);
    load_vec<V>(u + r * u_stride + ff + c, b);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = silu_act<T>(a[e]) * b[e];
    store_vec<V>(out + r * ff + c, a);
  }
}

__global__ void batch_begin_kernel(int32_t* lens, const int32_t* slots, const int32_t* cu, int32_t* pos0, int batch) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= batch) return;
  const int s = slots[b], n = cu != nullptr ? cu[b + 1] - cu[b] : 1;
  const int at = lens[s];
  pos0[b] = at;
  lens[s] = at + n;
}

static int rows_grid(const char* what, int64_t rows) {
  return rows > INT32_MAX ? fail(TKV_ERR_UNSUPPORTED, "%s: %lld rows", what, (long long)rows) : TKV_OK;
}

}  // namespace tkv

#define TKV_LAUNCH_V(vec, kernel, grid, threads, ...)                                                            \
  cudaError_t e_ = (vec) ? launch_pdl(kernel<T, 8>, dim3((unsigned)(grid)), dim3(threads), 0, (cudaStream_t)stream, __VA_ARGS__) \
                         : launch_pdl(kernel<T, 1>, dim3((unsigned)(grid)), dim3(threads), 0, (cudaStream_t)stream, __VA_ARGS__); \
  if (e_ != cudaSuccess) return fail(TKV_ERR_LAUNCH, #kernel ": %s", cudaGetErrorString(e_))

extern "C" int tkv_embed_stream(const int64_t* ids, const void* table, int64_t vocab, float* stream_out, void* copy_out, int rows,
                                int width, float scale, int dtype, int32_t* status, tkv_stream_t stream) {
  using namespace tkv;
  if (!ids || !table || !stream_out) return fail(TKV_ERR_ARG, "tkv_embed_stream: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_embed_stream: dtype %d", dtype);
  if (rows < 0 || width <= 0 || vocab <= 0) return fail(TKV_ERR_ARG, "tkv_embed_stream: bad sizes");
  if (rows == 0) return TKV_OK;
  const bool vec = width % 8 == 0 && aligned16(table) && aligned16(stream_out) && (!copy_out || aligned16(copy_out));
  TKV_WITH_TYPE(dtype, T, {
    TKV_LAUNCH_V(vec, embed_stream_kernel, rows, kRowThreads, ids, (const T*)table, vocab, stream_out, (T*)copy_out, width, scale, status);
  });
  return check_launch("tkv_embed_stream");
}

extern "C" int tkv_postnorm_add(float* x, const void* y, const float* weight, void* copy_out, int rows, int width, float eps,
                                float mult, float weight_offset, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!x || !y || !weight) return fail(TKV_ERR_ARG, "tkv_postnorm_add: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_postnorm_add: dtype %d", dtype);
  if (rows < 0 || width <= 0) return fail(TKV_ERR_ARG, "tkv_postnorm_add: bad sizes");
  if (rows == 0) return TKV_OK;
  const bool vec = width % 8 == 0 && aligned16(x) && aligned16(y) && aligned16(weight) && (!copy_out || aligned16(copy_out));
  TKV_WITH_TYPE(dtype, T, {
    TKV_LAUNCH_V(vec, postnorm_add_kernel, rows, kRowThreads, x, (const T*)y, weight, (T*)copy_out, width, eps, mult, weight_offset);
  });
  return check_launch("tkv_postnorm_add");
}

extern "C" int tkv_gated_sum_norm(float* x, const void* y, const int32_t* place, const float* choice_w, int top, const void* gate,
                                  int64_t gate_stride, const float* gate_bias, const float* weight, void* copy_out, int rows,
                                  int width, int groups, float eps, float alpha, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!x || !y || !weight || (place && !choice_w) || (gate && !gate_bias)) return fail(TKV_ERR_ARG, "tkv_gated_sum_norm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_gated_sum_norm: dtype %d", dtype);
  if (rows < 0 || width <= 0 || groups <= 0 || width % groups || (place && top <= 0) || (gate && gate_stride < width))
    return fail(TKV_ERR_ARG, "tkv_gated_sum_norm: bad sizes rows=%d width=%d groups=%d top=%d", rows, width, groups, top);
  if (rows == 0) return TKV_OK;
  const bool vec = (width / groups) % 8 == 0 && aligned16(x) && aligned16(y) && aligned16(weight) && (!copy_out || aligned16(copy_out)) &&
                   (!gate || (aligned16(gate) && aligned16(gate_bias) && (gate_stride * elem_size(dtype)) % 16 == 0));
  const int per_thread = (width / (vec ? 8 : 1) + kRowThreads - 1) / kRowThreads;
  const int keep = !vec ? (per_thread <= 8 ? 8 : 0) : per_thread <= 1 ? 1 : per_thread <= 2 ? 2 : per_thread <= 4 ? 4 : 0;
  const size_t smem = ((size_t)(groups > keep ? groups : keep) * (kRowThreads / 32) + (keep ? 0 : width)) * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "tkv_gated_sum_norm: width=%d groups=%d", width, groups);
  GatedSumNorm p = {x, y, gate, gate_stride, gate_bias, weight, copy_out, place, choice_w, top, width, groups, eps, alpha};
  TKV_WITH_TYPE(dtype, T, {
    auto pick = [&](auto routed) {
      constexpr bool R = decltype(routed)::value;
      if (!vec) return keep ? gated_sum_norm_kernel<T, 1, 8, R> : gated_sum_norm_kernel<T, 1, 0, R>;
      return keep == 1 ? gated_sum_norm_kernel<T, 8, 1, R> : keep == 2 ? gated_sum_norm_kernel<T, 8, 2, R>
             : keep == 4 ? gated_sum_norm_kernel<T, 8, 4, R> : gated_sum_norm_kernel<T, 8, 0, R>;
    };
    auto kern = place != nullptr ? pick(std::true_type{}) : pick(std::false_type{});
    cudaError_t e = launch_pdl(kern, dim3((unsigned)rows), dim3(kRowThreads), smem, (cudaStream_t)stream, p);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_gated_sum_norm: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_gated_sum_norm");
}

extern "C" int tkv_stream_norm(const float* x, const int32_t* row_idx, const float* weight, void* out, int rows, int width,
                               int groups, float eps, float weight_offset, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!x || !weight || !out) return fail(TKV_ERR_ARG, "tkv_stream_norm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_stream_norm: dtype %d", dtype);
  if (rows < 0 || width <= 0 || groups <= 0 || width % groups) return fail(TKV_ERR_ARG, "tkv_stream_norm: bad sizes");
  if (rows == 0) return TKV_OK;
  const size_t smem = (size_t)groups * (kRowThreads / 32) * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "tkv_stream_norm: groups=%d", groups);
  const bool vec = (width / groups) % 8 == 0 && aligned16(x) && aligned16(weight) && aligned16(out);
  TKV_WITH_TYPE(dtype, T, {
    cudaError_t e = launch_pdl(vec ? stream_norm_kernel<T, 8> : stream_norm_kernel<T, 1>, dim3((unsigned)rows), dim3(kRowThreads), smem,
                               (cudaStream_t)stream, x, row_idx, weight, (T*)out, width, groups, eps, weight_offset);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_stream_norm: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_stream_norm");
}

extern "C" int tkv_gated_norm(const void* y, int64_t y_stride, const void* z, int64_t z_stride, const float* weight,
                              int weight_shared, void* out, int rows, int groups, int group_len, float eps, int gate_first,
                              int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!y || !out) return fail(TKV_ERR_ARG, "tkv_gated_norm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_gated_norm: dtype %d", dtype);
  if (rows < 0 || groups <= 0 || group_len <= 0) return fail(TKV_ERR_ARG, "tkv_gated_norm: bad sizes");
  const int64_t width = (int64_t)groups * group_len;
  if (y_stride < width || (z && z_stride < width)) return fail(TKV_ERR_ARG, "tkv_gated_norm: row strides shorter than a row");
  if (rows == 0) return TKV_OK;
  const int64_t es = elem_size(dtype);
  const bool vec = group_len % 8 == 0 && (y_stride * es) % 16 == 0 && (!z || ((z_stride * es) % 16 == 0 && aligned16(z))) && aligned16(y) &&
                   aligned16(out) && (!weight || aligned16(weight));
  const int lanes = !vec || group_len > 256 ? 32 : group_len > 128 ? 16 : 8;
  const int64_t grid = ((int64_t)rows * groups + kRowThreads / lanes - 1) / (kRowThreads / lanes);
  int rc = rows_grid("tkv_gated_norm", grid);
  if (rc != TKV_OK) return rc;
  TKV_WITH_TYPE(dtype, T, {
    auto k = !vec ? gated_norm_kernel<T, 1, 32> : lanes == 8 ? gated_norm_kernel<T, 8, 8> : lanes == 16 ? gated_norm_kernel<T, 8, 16> : gated_norm_kernel<T, 8, 32>;
    cudaError_t e = launch_pdl(k, dim3((unsigned)grid), dim3(kRowThreads), 0, (cudaStream_t)stream, (const T*)y, y_stride, (const T*)z,
                               z_stride, weight, weight_shared, (T*)out, rows, groups, group_len, eps, gate_first);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_gated_norm: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_gated_norm");
}

extern "C" int tkv_gelu_tanh(void* u, int64_t n, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!u) return fail(TKV_ERR_ARG, "tkv_gelu_tanh: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_gelu_tanh: dtype %d", dtype);
  if (n < 0) return fail(TKV_ERR_ARG, "tkv_gelu_tanh: bad size");
  if (n == 0) return TKV_OK;
  const bool vec = n % 8 == 0 && aligned16(u);
  const int64_t blocks = (n / (vec ? 8 : 1) + kRowThreads - 1) / kRowThreads;
  const int grid = (int)(blocks < 148 * 16 ? blocks : 148 * 16);
  TKV_WITH_TYPE(dtype, T, { TKV_LAUNCH_V(vec, gelu_tanh_kernel, grid, kRowThreads, (T*)u, n); });
  return check_launch("tkv_gelu_tanh");
}

extern "C" int tkv_swiglu(const void* u, int64_t u_stride, void* out, int rows, int ff, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!u || !out) return fail(TKV_ERR_ARG, "tkv_swiglu: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_swiglu: dtype %d", dtype);
  if (rows < 0 || ff <= 0 || u_stride < (int64_t)2 * ff) return fail(TKV_ERR_ARG, "tkv_swiglu: bad sizes");
  if (rows == 0) return TKV_OK;
  const bool vec = ff % 8 == 0 && (u_stride * elem_size(dtype)) % 16 == 0 && aligned16(u) && aligned16(out);
  const int64_t blocks = ((int64_t)rows * (ff / (vec ? 8 : 1)) + kRowThreads - 1) / kRowThreads;
  const int grid = (int)(blocks < 148 * 16 ? blocks : 148 * 16);
  TKV_WITH_TYPE(dtype, T, { TKV_LAUNCH_V(vec, swiglu_kernel, grid, kRowThreads, (const T*)u, u_stride, (T*)out, (int64_t)rows, ff); });
  return check_launch("tkv_swiglu");
}

extern "C" int tkv_batch_begin(int32_t* lens, const int32_t* slots, const int32_t* cu_tokens, int32_t* pos0, int batch,
                               tkv_stream_t stream) {
  using namespace tkv;
  if (!lens || !slots || !pos0) return fail(TKV_ERR_ARG, "tkv_batch_begin: NULL pointer argument");
  if (batch < 0) return fail(TKV_ERR_ARG, "tkv_batch_begin: bad size");
  if (batch == 0) return TKV_OK;
  cudaError_t e = launch_pdl(batch_begin_kernel, dim3((batch + 127) / 128), dim3(128), 0, (cudaStream_t)stream, lens, slots, cu_tokens,
                             pos0, batch);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_batch_begin: %s", cudaGetErrorString(e));
  return check_launch("tkv_batch_begin");
}
