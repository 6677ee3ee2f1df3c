// The residual stream of decoders that keep it in fp32 and norm the OUTPUT of a sublayer, and the elementwise steps
// around their products:
//   embed_stream_kernel  : token rows of the embedding as fp32 stream + its copy in the model type;
//   postnorm_add_kernel  : stream += mult * RMSNorm(y) * (w_offset + w), and the copy the next product reads;
//   stream_norm_kernel   : RMSNorm of the stream itself (before the output projection);
//   gated_norm_kernel    : group RMSNorm with a SiLU gate before or after it, optional weight;
//   gelu_tanh_kernel     : the tanh form of GELU, in place;
//   batch_begin_kernel   : start positions of a step's requests, and the lengths after it.
// All statistics are fp32.  Every kernel runs for the 16-bit model type and for fp32.
#include "tkv_elem.cuh"

namespace tkv {

constexpr int kRowThreads = 256;

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) embed_stream_kernel(const int64_t* ids, const T* table, int64_t vocab, float* x,
                                                                  T* copy, int width, int32_t* status) {
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

template <typename T, int V>
__global__ void __launch_bounds__(kRowThreads) stream_norm_kernel(const float* x, const int32_t* rows, const float* w, T* out,
                                                                 int width, float eps, float w_offset) {
  __shared__ float red[kRowThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const float* src = x + (int64_t)(rows != nullptr ? rows[blockIdx.x] : (int)blockIdx.x) * width;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < width; c += kRowThreads * V) {
    float a[V];
    load_vec<V>(src + c, a);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += a[e] * a[e];
  }
  const float rstd = 1.0f / sqrtf(block_add<kRowThreads>(ss, red) / (float)width + eps);
  for (int c = threadIdx.x * V; c < width; c += kRowThreads * V) {
    float a[V], g[V];
    load_vec<V>(src + c, a);
    load_vec<V>(w + c, g);
#pragma unroll
    for (int e = 0; e < V; ++e) a[e] = a[e] * rstd * (w_offset + g[e]);
    store_vec<V>(out + (int64_t)blockIdx.x * width + c, a);
  }
}

// kLanes lanes per (row, group) of `len` elements.  gate_first: RMS(y * silu(z)) * w, else RMS(y) * w * silu(z).
template <typename T, int V, int kLanes>
__global__ void __launch_bounds__(kRowThreads) gated_norm_kernel(const T* y, int64_t y_stride, const T* z, int64_t z_stride,
                                                                const float* w, T* out, int rows, int groups, int len,
                                                                float eps, int gate_first) {
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
  const T* zr = z + row * z_stride + (int64_t)grp * len;
  T* o = out + (row * groups + grp) * (int64_t)len;
  const int nvec = len / V;
  float a[kKeep][V], g[kKeep][V], ss = 0.f;
  auto gate = [&](float* av, float* gv) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      gv[e] = silu_act<T>(gv[e]);
      if (gate_first) av[e] *= gv[e];
      ss += av[e] * av[e];
    }
  };
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (lane + kLanes * j < nvec) {
      load_vec<V>(yr + (int64_t)(lane + kLanes * j) * V, a[j]);
      load_vec<V>(zr + (int64_t)(lane + kLanes * j) * V, g[j]);
    }
#pragma unroll
  for (int j = 0; j < kKeep; ++j)
    if (lane + kLanes * j < nvec) gate(a[j], g[j]);
  for (int i = lane + kLanes * kKeep; i < nvec; i += kLanes) {
    float av[V], gv[V];
    load_vec<V>(yr + (int64_t)i * V, av);
    load_vec<V>(zr + (int64_t)i * V, gv);
    gate(av, gv);
  }
#pragma unroll
  for (int d = kLanes / 2; d >= 1; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  const float rstd = 1.0f / sqrtf(ss / (float)len + eps);
  if (!live) return;
  auto finish = [&](int i, float* av, const float* gv) {
    float wv[V];
    if (w != nullptr) load_vec<V>(w + (int64_t)grp * len + (int64_t)i * V, wv);
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
    load_vec<V>(zr + (int64_t)i * V, gv);
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
                                int width, int dtype, int32_t* status, tkv_stream_t stream) {
  using namespace tkv;
  if (!ids || !table || !stream_out) return fail(TKV_ERR_ARG, "tkv_embed_stream: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_embed_stream: dtype %d", dtype);
  if (rows < 0 || width <= 0 || vocab <= 0) return fail(TKV_ERR_ARG, "tkv_embed_stream: bad sizes");
  if (rows == 0) return TKV_OK;
  const bool vec = width % 8 == 0 && aligned16(table) && aligned16(stream_out) && (!copy_out || aligned16(copy_out));
  TKV_WITH_TYPE(dtype, T, {
    TKV_LAUNCH_V(vec, embed_stream_kernel, rows, kRowThreads, ids, (const T*)table, vocab, stream_out, (T*)copy_out, width, status);
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

extern "C" int tkv_stream_norm(const float* x, const int32_t* row_idx, const float* weight, void* out, int rows, int width,
                               float eps, float weight_offset, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!x || !weight || !out) return fail(TKV_ERR_ARG, "tkv_stream_norm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_stream_norm: dtype %d", dtype);
  if (rows < 0 || width <= 0) return fail(TKV_ERR_ARG, "tkv_stream_norm: bad sizes");
  if (rows == 0) return TKV_OK;
  const bool vec = width % 8 == 0 && aligned16(x) && aligned16(weight) && aligned16(out);
  TKV_WITH_TYPE(dtype, T, {
    TKV_LAUNCH_V(vec, stream_norm_kernel, rows, kRowThreads, x, row_idx, weight, (T*)out, width, eps, weight_offset);
  });
  return check_launch("tkv_stream_norm");
}

extern "C" int tkv_gated_norm(const void* y, int64_t y_stride, const void* z, int64_t z_stride, const float* weight, void* out,
                              int rows, int groups, int group_len, float eps, int gate_first, int dtype, tkv_stream_t stream) {
  using namespace tkv;
  if (!y || !z || !out) return fail(TKV_ERR_ARG, "tkv_gated_norm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_gated_norm: dtype %d", dtype);
  if (rows < 0 || groups <= 0 || group_len <= 0) return fail(TKV_ERR_ARG, "tkv_gated_norm: bad sizes");
  const int64_t width = (int64_t)groups * group_len;
  if (y_stride < width || z_stride < width) return fail(TKV_ERR_ARG, "tkv_gated_norm: row strides shorter than a row");
  if (rows == 0) return TKV_OK;
  const int64_t es = elem_size(dtype);
  const bool vec = group_len % 8 == 0 && (y_stride * es) % 16 == 0 && (z_stride * es) % 16 == 0 && aligned16(y) && aligned16(z) &&
                   aligned16(out) && (!weight || aligned16(weight));
  const int lanes = !vec || group_len > 256 ? 32 : group_len > 128 ? 16 : 8;
  const int64_t grid = ((int64_t)rows * groups + kRowThreads / lanes - 1) / (kRowThreads / lanes);
  int rc = rows_grid("tkv_gated_norm", grid);
  if (rc != TKV_OK) return rc;
  TKV_WITH_TYPE(dtype, T, {
    auto k = !vec ? gated_norm_kernel<T, 1, 32> : lanes == 8 ? gated_norm_kernel<T, 8, 8> : lanes == 16 ? gated_norm_kernel<T, 8, 16> : gated_norm_kernel<T, 8, 32>;
    cudaError_t e = launch_pdl(k, dim3((unsigned)grid), dim3(kRowThreads), 0, (cudaStream_t)stream, (const T*)y, y_stride, (const T*)z,
                               z_stride, weight, (T*)out, rows, groups, group_len, eps, gate_first);
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
