// Producers and one-token steps of the linear-recurrence layers, and a token-by-token scan for every size and type.
//
//   rotate_qk_kernel       : rotary positions on q and k of a packed batch (first rot_dims dims, pair i with i + rot_dims/2);
//   conv_silu_kernel       : causal depthwise convolution + bias + SiLU over a packed batch; earlier inputs of a request
//                            come from its ring of `taps` inputs (input of position p in row p mod taps);
//   conv_tail_kernel       : the last inputs of every request into its ring;
//   ssd_steps_kernel       : dt = softplus(dt + bias), log a = -exp(A_log) dt;
//   retention_step_kernel  : one token: rotation, state update, read-out, per-head RMS and the SiLU gate in one pass;
//   ssd_step_kernel        : one token: convolution (and its ring), dt, state update, read-out with the skip weight;
//   linrec_scan_kernel     : any number of tokens, one after the other, state in shared memory.
// A request whose start position is 0 starts from the zero state whatever its slot held before.  The state is fp32 and
// is read and written once per step; its 8 n p bytes per head are what a decode step costs.
#include "tkv_linrec.cuh"
#include "tkv_state_step.cuh"

namespace tkv {

constexpr int kRotThreads = 128;

// One CTA per token.  proj row: q [heads, dim] at column 0, k [heads, dim] behind it.  out row: the same, contiguous.
template <typename T, int V>
__global__ void __launch_bounds__(kRotThreads) rotate_qk_kernel(const T* proj, int64_t row_stride, T* out, const int32_t* cu,
                                                               const int32_t* pos0, int batch, int heads, int dim, int rot_dims,
                                                               const float2* freq, float k_scale) {
  extern __shared__ float tab[];                      // sin [half], cos [half]
  grid_dependency_wait();
  grid_launch_dependents();
  const int t = blockIdx.x, half = rot_dims / 2;
  const int b = owner_of(cu, batch, t);
  const int pos = pos0[b] + (cu != nullptr ? t - cu[b] : 0);
  for (int i = threadIdx.x; i < half; i += kRotThreads) turn(pos, freq[i].x, freq[i].y, &tab[i], &tab[half + i]);
  __syncthreads();
  const int per_head = half / V, tail = (dim - rot_dims) / V;      // work items of a head: rotated pairs, then the rest
  const int items = per_head + tail;
  const T* src = proj + (int64_t)t * row_stride;
  T* dst = out + (int64_t)t * 2 * heads * dim;
  for (int i = threadIdx.x; i < 2 * heads * items; i += kRotThreads) {
    const int hh = i / items, w = i - hh * items;
    const float scale = hh < heads ? 1.0f : k_scale;
    const int64_t base = (int64_t)hh * dim;
    if (w < per_head) {
      float u[V], v[V];
      load_vec<V>(src + base + w * V, u);
      load_vec<V>(src + base + half + w * V, v);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float s = tab[w * V + e], c = tab[half + w * V + e];
        const float a = (u[e] * c - v[e] * s) * scale, bb = (v[e] * c + u[e] * s) * scale;
        u[e] = a; v[e] = bb;
      }
      store_vec<V>(dst + base + w * V, u);
      store_vec<V>(dst + base + half + w * V, v);
    } else {
      float u[V];
      const int64_t at = base + rot_dims + (w - per_head) * V;
      load_vec<V>(src + at, u);
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] *= scale;
      store_vec<V>(dst + at, u);
    }
  }
}

constexpr int kConvThreads = 128, kConvStrip = 32;

// grid: (channel blocks, strips of kConvStrip tokens, requests).  kTaps = 0: any number of taps, inputs re-read per tap.
template <typename T, int V, int kTaps>
__global__ void __launch_bounds__(kConvThreads) conv_silu_kernel(const T* proj, int64_t row_stride, const T* ring, const float* w,
                                                                const float* bias, T* out, const int32_t* cu, const int32_t* slots,
                                                                const int32_t* pos0, int channels, int taps_rt) {
  const int taps = kTaps > 0 ? kTaps : taps_rt;
  const int ch = (blockIdx.x * kConvThreads + threadIdx.x) * V;
  const int b = blockIdx.z;
  grid_dependency_wait();
  grid_launch_dependents();
  const int t0 = cu[b], n = cu[b + 1] - t0;
  const int i0 = blockIdx.y * kConvStrip, i1 = min(n, i0 + kConvStrip);
  if (ch >= channels || i0 >= n) return;
  const int p0 = pos0[b];
  const T* hist = ring + (int64_t)slots[b] * taps * channels;
  auto input = [&](int i, float* v) {                 // input of the request's i-th token of this step (i < 0: earlier)
    if (i >= 0) load_vec<V>(proj + (int64_t)(t0 + i) * row_stride + ch, v);
    else if (p0 + i >= 0) load_vec<V>(hist + (int64_t)((p0 + i) % taps) * channels + ch, v);
    else
      for (int e = 0; e < V; ++e) v[e] = 0.f;
  };
  float bs[V];
#pragma unroll
  for (int e = 0; e < V; ++e) bs[e] = bias[ch + e];
  if (kTaps > 0) {
    constexpr int kT = kTaps > 0 ? kTaps : 1;
    float wt[kT][V], win[kT][V];                       // win[k]: input k places before the newest
#pragma unroll
    for (int k = 0; k < kT; ++k)
#pragma unroll
      for (int e = 0; e < V; ++e) wt[k][e] = w[(int64_t)(ch + e) * kT + kT - 1 - k];
#pragma unroll
    for (int k = 1; k < kT; ++k) input(i0 - k, win[k - 1]);
    for (int i = i0; i < i1; ++i) {
#pragma unroll
      for (int k = kT - 1; k > 0; --k)
#pragma unroll
        for (int e = 0; e < V; ++e) win[k][e] = win[k - 1][e];
      input(i, win[0]);
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        acc[e] = bs[e];
#pragma unroll
        for (int k = kT - 1; k >= 0; --k) acc[e] = fmaf(wt[k][e], win[k][e], acc[e]);
        acc[e] = silu_act<T>(acc[e]);
      }
      store_vec<V>(out + (int64_t)(t0 + i) * channels + ch, acc);
    }
  } else {
    for (int i = i0; i < i1; ++i) {
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = bs[e];
      for (int k = taps - 1; k >= 0; --k) {
        float v[V];
        input(i - k, v);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[(int64_t)(ch + e) * taps + taps - 1 - k], v[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = silu_act<T>(acc[e]);
      store_vec<V>(out + (int64_t)(t0 + i) * channels + ch, acc);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kConvThreads) conv_tail_kernel(const T* proj, int64_t row_stride, T* ring, const int32_t* cu,
                                                                const int32_t* slots, const int32_t* pos0, int channels, int taps) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.y;
  const int ch = blockIdx.x * kConvThreads + threadIdx.x;
  const int t0 = cu[b], n = cu[b + 1] - t0;
  if (ch >= channels) return;
  T* dst = ring + (int64_t)slots[b] * taps * channels + ch;
  for (int i = max(0, n - taps); i < n; ++i) dst[(int64_t)((pos0[b] + i) % taps) * channels] = proj[(int64_t)(t0 + i) * row_stride + ch];
}

template <typename T>
__global__ void __launch_bounds__(256) ssd_steps_kernel(const T* dt_in, int64_t row_stride, const float* dt_bias, const float* a_log,
                                                       float* dt, float* log_decay, int64_t total, int heads) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const int64_t t = i / heads;
  const int h = (int)(i - t * heads);
  const float d = softplus_f32(to_f32<T>(dt_in[t * row_stride + h]) + dt_bias[h]);
  dt[i] = d;
  log_decay[i] = -expf(a_log[h]) * d;
}

// One CTA per (request, head).  proj row: q [heads, dim], k [heads, dim], v [heads, vdim], gate [heads, vdim].
template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads) retention_step_kernel(const T* proj, int64_t row_stride, float* state,
                                                                     const int32_t* slots, const int32_t* pos0, const float* decay,
                                                                     const float2* freq, T* out, int heads, int dim, int vdim,
                                                                     int rot_dims, float k_scale, float eps) {
  extern __shared__ float sm[];
  float *q = sm, *k = q + dim, *v = k + dim, *o = v + vdim, *red = o + vdim;      // red: kStepThreads * 4
  __shared__ float wred[kStepThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x / heads, h = blockIdx.x - b * heads;
  const int pos = pos0[b];
  StateStep<V> step;
  step.prefetch(state + ((int64_t)slots[b] * heads + h) * dim * vdim, dim, vdim, pos == 0);
  const T* row = proj + (int64_t)b * row_stride;
  const T *qg = row + (int64_t)h * dim, *kg = row + (int64_t)(heads + h) * dim;
  const T* vg = row + (int64_t)2 * heads * dim + (int64_t)h * vdim;
  const T* gg = vg + (int64_t)heads * vdim;
  const int half = rot_dims / 2;
  for (int i = threadIdx.x; i < half; i += kStepThreads) {
    float s, c;
    turn(pos, freq[i].x, freq[i].y, &s, &c);
    const float qu = to_f32<T>(qg[i]), qv = to_f32<T>(qg[i + half]), ku = to_f32<T>(kg[i]), kv = to_f32<T>(kg[i + half]);
    q[i] = round_as<T>(qu * c - qv * s);
    q[i + half] = round_as<T>(qv * c + qu * s);
    k[i] = round_as<T>((ku * c - kv * s) * k_scale);
    k[i + half] = round_as<T>((kv * c + ku * s) * k_scale);
  }
  for (int i = rot_dims + threadIdx.x; i < dim; i += kStepThreads) {
    q[i] = to_f32<T>(qg[i]);
    k[i] = round_as<T>(to_f32<T>(kg[i]) * k_scale);
  }
  for (int i = threadIdx.x; i < vdim; i += kStepThreads) v[i] = to_f32<T>(vg[i]);
  __syncthreads();
  const float a = decay[h];
  step.run([a](int) { return a; }, k, q, v, o, red);
  float ss = 0.f;
  for (int i = threadIdx.x; i < vdim; i += kStepThreads) ss += o[i] * o[i];
  const float rstd = 1.0f / sqrtf(block_add<kStepThreads>(ss, wred) / (float)vdim + eps);
  T* dst = out + ((int64_t)b * heads + h) * vdim;
  for (int i = threadIdx.x; i < vdim; i += kStepThreads) dst[i] = from_f32<T>(o[i] * rstd * silu_act<T>(to_f32<T>(gg[i])));
}

// One CTA per (request, head).  proj row: z [inner], x [inner], B [groups, n], C [groups, n], dt [heads]; the ring holds
// the last `taps` inputs of x | B | C.  This step's inputs go to ring row pos mod taps, which holds an input that no
// longer counts, so heads of a group may read the other rows while one of them writes.
template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads, 4) ssd_step_kernel(const T* proj, int64_t row_stride, T* ring, float* state,
                                                               const int32_t* slots, const int32_t* pos0, const float* conv_w,
                                                               const float* conv_b, const float* dt_bias, const float* a_log,
                                                               const float* skip, T* out, int heads, int groups, int n, int vdim,
                                                               int taps) {
  extern __shared__ float sm[];
  float *q = sm, *k = q + n, *x = k + n, *v = x + vdim, *o = v + vdim, *red = o + vdim;
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x / heads, h = blockIdx.x - b * heads;
  const int hpg = heads / groups, g = h / hpg;
  const int pos = pos0[b], slot = slots[b], inner = heads * vdim, channels = inner + 2 * groups * n;
  StateStep<V> step;
  step.prefetch(state + ((int64_t)slot * heads + h) * n * vdim, n, vdim, pos == 0);
  const T* cur = proj + (int64_t)b * row_stride + inner;
  T* rg = ring + (int64_t)slot * taps * channels;
  const float dt = softplus_f32(to_f32<T>(cur[channels + h]) + dt_bias[h]);
  const float decay = expf(-expf(a_log[h]) * dt);
  const float sk = skip[h];
  // Two channels per thread and pass, every load requested before the first use.
  for (int base = threadIdx.x; base < vdim + 2 * n; base += 2 * kStepThreads) {
    float acc[2];
    T in[2];
    int chs[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = base + u * kStepThreads;
      if (i >= vdim + 2 * n) continue;
      const int ch = i < vdim ? h * vdim + i : (i < vdim + n ? inner + g * n + (i - vdim) : inner + (groups + g) * n + (i - vdim - n));
      chs[u] = ch;
      acc[u] = conv_b[ch];
      in[u] = cur[ch];
      if (taps == 4) {                                     // the usual number
        const float4 w = *reinterpret_cast<const float4*>(conv_w + (int64_t)ch * 4);
        const int r0 = pos & 3;
        const float x3 = pos >= 3 ? to_f32<T>(rg[(int64_t)((r0 + 1) & 3) * channels + ch]) : 0.f;
        const float x2 = pos >= 2 ? to_f32<T>(rg[(int64_t)((r0 + 2) & 3) * channels + ch]) : 0.f;
        const float x1 = pos >= 1 ? to_f32<T>(rg[(int64_t)((r0 + 3) & 3) * channels + ch]) : 0.f;
        acc[u] = fmaf(w.w, to_f32<T>(in[u]), fmaf(w.z, x1, fmaf(w.y, x2, fmaf(w.x, x3, acc[u]))));
      } else {
        for (int d = taps - 1; d > 0; --d)
          if (pos - d >= 0) acc[u] = fmaf(conv_w[(int64_t)ch * taps + taps - 1 - d], to_f32<T>(rg[(int64_t)((pos - d) % taps) * channels + ch]), acc[u]);
        acc[u] = fmaf(conv_w[(int64_t)ch * taps + taps - 1], to_f32<T>(in[u]), acc[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = base + u * kStepThreads;
      if (i >= vdim + 2 * n) continue;
      if (i < vdim || h == g * hpg) rg[(int64_t)(pos % taps) * channels + chs[u]] = in[u];
      const float y = round_as<T>(silu_act<T>(acc[u]));
      if (i < vdim) { x[i] = y; v[i] = dt * y; }
      else if (i < vdim + n) k[i - vdim] = y;
      else q[i - vdim - n] = y;
    }
  }
  __syncthreads();
  step.run([decay](int) { return decay; }, k, q, v, o, red);
  T* dst = out + (int64_t)b * inner + (int64_t)h * vdim;
  for (int i = threadIdx.x; i < vdim; i += kStepThreads) dst[i] = from_f32<T>(fmaf(sk, x[i], o[i]));
}

// ---------------------------------------------------------------------------------------------- scan, token by token
constexpr int kScanWarps = 8;

// One CTA per (request, head, 32 columns of v): lane = column, warps share the rows of the state.
template <typename T>
__global__ void __launch_bounds__(kScanWarps * 32) linrec_scan_kernel(LinrecParams a) {
  extern __shared__ float S[];                        // [n][32]
  __shared__ float red[2][kScanWarps][32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ptiles = (a.p + 31) / 32;
  const int pt = blockIdx.x % ptiles, bh = blockIdx.x / ptiles;
  const int b = bh / a.heads, h = bh - b * a.heads, g = h / (a.heads / a.groups);
  const int t0 = a.cu != nullptr ? a.cu[b] : b, t1 = a.cu != nullptr ? a.cu[b + 1] : b + 1;
  if (t1 <= t0) return;
  const int col = pt * 32 + lane;
  const bool ok = col < a.p;
  float* G = a.state + ((int64_t)a.slots[b] * a.heads + h) * a.n * a.p;
  const bool fresh = a.pos0[b] == 0;
  for (int r = warp; r < a.n; r += kScanWarps) S[r * 32 + lane] = (ok && !fresh) ? G[(int64_t)r * a.p + col] : 0.f;
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
  for (int t = t0; t < t1; ++t) {
    const int64_t th = (int64_t)t * a.heads + h;
    const float decay = a.log_decay != nullptr ? expf(a.log_decay[th]) : a.head_decay[h];
    const T* kt = (const T*)a.k + (int64_t)t * a.k_stride + (int64_t)g * a.n;
    const T* qt = (const T*)a.q + (int64_t)t * a.q_stride + (int64_t)g * a.n;
    const float x = ok ? to_f32<T>(((const T*)a.v)[(int64_t)t * a.v_stride + (int64_t)h * a.p + col]) : 0.f;
    const float v = a.v_scale != nullptr ? a.v_scale[th] * x : x;
    float acc = 0.f;
    for (int r = warp; r < a.n; r += kScanWarps) {
      const float s = fmaf(decay, S[r * 32 + lane], to_f32<T>(kt[r]) * v);
      S[r * 32 + lane] = s;
      acc = fmaf(to_f32<T>(qt[r]), s, acc);
    }
    const int par = t & 1;                             // two buffers: one barrier per token
    red[par][warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && ok) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kScanWarps; ++w) o += red[par][w][lane];
      ((T*)a.out)[(int64_t)t * a.heads * a.p + (int64_t)h * a.p + col] = from_f32<T>(fmaf(skip, x, o));
    }
  }
  for (int r = warp; r < a.n; r += kScanWarps)
    if (ok) G[(int64_t)r * a.p + col] = S[r * 32 + lane];
}

}  // namespace tkv

using namespace tkv;

#define TKV_CHECK_LAUNCH(call, name)                                                     \
  do {                                                                                   \
    cudaError_t e_ = (call);                                                             \
    if (e_ != cudaSuccess) return fail(TKV_ERR_LAUNCH, name ": %s", cudaGetErrorString(e_)); \
  } while (0)

extern "C" int tkv_rotate_qk(const void* proj, int64_t row_stride, void* out, const int32_t* cu_tokens, const int32_t* pos0,
                             int batch, int tokens, int heads, int dim, int rot_dims, const float* freq_hi_lo, float k_scale,
                             int dtype, tkv_stream_t stream) {
  if (!proj || !out || !pos0 || (rot_dims > 0 && !freq_hi_lo)) return fail(TKV_ERR_ARG, "tkv_rotate_qk: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_rotate_qk: dtype %d", dtype);
  if (batch < 0 || tokens < 0 || heads <= 0 || dim <= 0 || rot_dims < 0 || rot_dims > dim || rot_dims % 2 ||
      row_stride < (int64_t)2 * heads * dim)
    return fail(TKV_ERR_ARG, "tkv_rotate_qk: bad sizes");
  if (tokens == 0 || batch == 0) return TKV_OK;
  const int64_t es = elem_size(dtype);
  const bool vec = (rot_dims / 2) % 8 == 0 && dim % 8 == 0 && (row_stride * es) % 16 == 0 && aligned16(proj) && aligned16(out);
  const size_t smem = (size_t)(rot_dims > 0 ? rot_dims : 1) * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "tkv_rotate_qk: rot_dims=%d", rot_dims);
  TKV_WITH_TYPE(dtype, T, {
    if (vec) TKV_CHECK_LAUNCH(launch_pdl(rotate_qk_kernel<T, 8>, dim3(tokens), dim3(kRotThreads), smem, (cudaStream_t)stream, (const T*)proj,
                                         row_stride, (T*)out, cu_tokens, pos0, batch, heads, dim, rot_dims, (const float2*)freq_hi_lo, k_scale), "tkv_rotate_qk");
    else TKV_CHECK_LAUNCH(launch_pdl(rotate_qk_kernel<T, 1>, dim3(tokens), dim3(kRotThreads), smem, (cudaStream_t)stream, (const T*)proj,
                                     row_stride, (T*)out, cu_tokens, pos0, batch, heads, dim, rot_dims, (const float2*)freq_hi_lo, k_scale), "tkv_rotate_qk");
  });
  return check_launch("tkv_rotate_qk");
}

namespace tkv {
template <typename T, int V>
static cudaError_t launch_conv(dim3 grid, cudaStream_t st, const void* proj, int64_t row_stride, const void* ring, const float* w,
                               const float* bias, void* out, const int32_t* cu, const int32_t* slots, const int32_t* pos0,
                               int channels, int taps) {
  if (taps == 4)
    return launch_pdl(conv_silu_kernel<T, V, 4>, grid, dim3(kConvThreads), 0, st, (const T*)proj, row_stride, (const T*)ring, w, bias,
                      (T*)out, cu, slots, pos0, channels, taps);
  return launch_pdl(conv_silu_kernel<T, V, 0>, grid, dim3(kConvThreads), 0, st, (const T*)proj, row_stride, (const T*)ring, w, bias,
                    (T*)out, cu, slots, pos0, channels, taps);
}
}  // namespace tkv

extern "C" int tkv_conv_silu(const void* proj, int64_t row_stride, void* ring, const float* conv_w, const float* conv_b, void* out,
                             const int32_t* cu_tokens, const int32_t* slots, const int32_t* pos0, int batch, int max_tokens,
                             int channels, int taps, int dtype, tkv_stream_t stream) {
  if (!proj || !ring || !conv_w || !conv_b || !out || !cu_tokens || !slots || !pos0)
    return fail(TKV_ERR_ARG, "tkv_conv_silu: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_conv_silu: dtype %d", dtype);
  if (batch < 0 || max_tokens < 0 || channels <= 0 || taps <= 0 || row_stride < channels) return fail(TKV_ERR_ARG, "tkv_conv_silu: bad sizes");
  if (batch == 0 || max_tokens == 0) return TKV_OK;
  const int64_t strips = ((int64_t)max_tokens + kConvStrip - 1) / kConvStrip;
  if (batch > 65535 || strips > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_conv_silu: batch=%d max_tokens=%d (at most 65535 requests of 2097120 tokens)", batch, max_tokens);
  const int64_t es = elem_size(dtype);
  const bool vec = channels % 8 == 0 && (row_stride * es) % 16 == 0 && aligned16(proj) && aligned16(out) && aligned16(ring);
  const int per = kConvThreads * (vec ? 8 : 1);
  const dim3 grid((channels + per - 1) / per, (unsigned)strips, batch);
  TKV_WITH_TYPE(dtype, T, {
    TKV_CHECK_LAUNCH(vec ? (launch_conv<T, 8>(grid, (cudaStream_t)stream, proj, row_stride, ring, conv_w, conv_b, out, cu_tokens, slots, pos0, channels, taps))
                         : (launch_conv<T, 1>(grid, (cudaStream_t)stream, proj, row_stride, ring, conv_w, conv_b, out, cu_tokens, slots, pos0, channels, taps)),
                     "tkv_conv_silu");
    const dim3 tgrid((channels + kConvThreads - 1) / kConvThreads, batch);
    TKV_CHECK_LAUNCH(launch_pdl(conv_tail_kernel<T>, tgrid, dim3(kConvThreads), 0, (cudaStream_t)stream, (const T*)proj, row_stride, (T*)ring,
                                cu_tokens, slots, pos0, channels, taps), "tkv_conv_silu (tail)");
  });
  return check_launch("tkv_conv_silu");
}

extern "C" int tkv_ssd_steps(const void* dt_in, int64_t row_stride, const float* dt_bias, const float* a_log, float* dt,
                             float* log_decay, int tokens, int heads, int dtype, tkv_stream_t stream) {
  if (!dt_in || !dt_bias || !a_log || !dt || !log_decay) return fail(TKV_ERR_ARG, "tkv_ssd_steps: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_ssd_steps: dtype %d", dtype);
  if (tokens < 0 || heads <= 0 || row_stride < heads) return fail(TKV_ERR_ARG, "tkv_ssd_steps: bad sizes");
  const int64_t total = (int64_t)tokens * heads;
  if (total == 0) return TKV_OK;
  TKV_WITH_TYPE(dtype, T, {
    TKV_CHECK_LAUNCH(launch_pdl(ssd_steps_kernel<T>, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, (const T*)dt_in,
                                row_stride, dt_bias, a_log, dt, log_decay, total, heads), "tkv_ssd_steps");
  });
  return check_launch("tkv_ssd_steps");
}

extern "C" int tkv_retention_step(const void* proj, int64_t row_stride, float* state, const int32_t* slots, const int32_t* pos0,
                                  const float* head_decay, const float* freq_hi_lo, void* out, int batch, int heads, int dim,
                                  int vdim, int rot_dims, float k_scale, float eps, int dtype, tkv_stream_t stream) {
  if (!proj || !state || !slots || !pos0 || !head_decay || (rot_dims > 0 && !freq_hi_lo) || !out)
    return fail(TKV_ERR_ARG, "tkv_retention_step: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_retention_step: dtype %d", dtype);
  if (batch < 0 || heads <= 0 || dim <= 0 || vdim <= 0 || rot_dims < 0 || rot_dims > dim || rot_dims % 2 ||
      row_stride < (int64_t)2 * heads * (dim + vdim))
    return fail(TKV_ERR_ARG, "tkv_retention_step: bad sizes");
  if (batch == 0) return TKV_OK;
  const size_t smem = ((size_t)2 * dim + 2 * vdim + kStepThreads * 4) * sizeof(float);
  TKV_WITH_TYPE(dtype, T, {
    auto kern = vdim % 4 == 0 ? retention_step_kernel<T, 4> : retention_step_kernel<T, 1>;
    if (!allow_smem(kern, smem)) return fail(TKV_ERR_UNSUPPORTED, "tkv_retention_step: dim=%d vdim=%d", dim, vdim);
    TKV_CHECK_LAUNCH(launch_pdl(kern, dim3((unsigned)(batch * heads)), dim3(kStepThreads), smem, (cudaStream_t)stream,
                                (const T*)proj, row_stride, state, slots, pos0, head_decay, (const float2*)freq_hi_lo, (T*)out, heads, dim,
                                vdim, rot_dims, k_scale, eps), "tkv_retention_step");
  });
  return check_launch("tkv_retention_step");
}

extern "C" int tkv_ssd_step(const void* proj, int64_t row_stride, void* ring, float* state, const int32_t* slots,
                            const int32_t* pos0, const float* conv_w, const float* conv_b, const float* dt_bias,
                            const float* a_log, const float* skip, void* out, int batch, int heads, int groups, int n, int vdim,
                            int taps, int dtype, tkv_stream_t stream) {
  if (!proj || !ring || !state || !slots || !pos0 || !conv_w || !conv_b || !dt_bias || !a_log || !skip || !out)
    return fail(TKV_ERR_ARG, "tkv_ssd_step: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_ssd_step: dtype %d", dtype);
  if (batch < 0 || heads <= 0 || groups <= 0 || heads % groups || n <= 0 || vdim <= 0 || taps <= 0 ||
      row_stride < (int64_t)2 * heads * vdim + 2 * groups * n + heads)
    return fail(TKV_ERR_ARG, "tkv_ssd_step: bad sizes");
  if (batch == 0) return TKV_OK;
  const size_t smem = ((size_t)2 * n + 3 * vdim + kStepThreads * 4) * sizeof(float);
  TKV_WITH_TYPE(dtype, T, {
    auto kern = vdim % 4 == 0 ? ssd_step_kernel<T, 4> : ssd_step_kernel<T, 1>;
    if (!allow_smem(kern, smem)) return fail(TKV_ERR_UNSUPPORTED, "tkv_ssd_step: n=%d vdim=%d", n, vdim);
    TKV_CHECK_LAUNCH(launch_pdl(kern, dim3((unsigned)(batch * heads)), dim3(kStepThreads), smem, (cudaStream_t)stream,
                                (const T*)proj, row_stride, (T*)ring, state, slots, pos0, conv_w, conv_b, dt_bias, a_log, skip, (T*)out,
                                heads, groups, n, vdim, taps), "tkv_ssd_step");
  });
  return check_launch("tkv_ssd_step");
}

extern "C" int tkv_linrec_scan(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride,
                               const float* log_decay, const float* head_decay, const float* v_scale, const float* skip, void* out,
                               float* state, const int32_t* slots, const int32_t* cu_tokens, const int32_t* pos0, int batch,
                               int heads, int groups, int n, int vdim, int dtype, tkv_stream_t stream) {
  if (!q || !k || !v || (!log_decay && !head_decay) || !out || !state || !slots || !pos0)
    return fail(TKV_ERR_ARG, "tkv_linrec_scan: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_scan: dtype %d", dtype);
  if (batch < 0 || heads <= 0 || groups <= 0 || heads % groups || n <= 0 || vdim <= 0 || q_stride < (int64_t)groups * n ||
      k_stride < (int64_t)groups * n || v_stride < (int64_t)heads * vdim)
    return fail(TKV_ERR_ARG, "tkv_linrec_scan: bad sizes");
  if (batch == 0) return TKV_OK;
  LinrecParams a = {q, q_stride, k, k_stride, v, v_stride, log_decay, head_decay, nullptr, v_scale, skip, out, state, slots, cu_tokens,
                    pos0, batch, heads, groups, n, vdim};
  const size_t smem = (size_t)n * 32 * sizeof(float);
  const int64_t grid = (int64_t)batch * heads * ((vdim + 31) / 32);
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_scan: %lld blocks", (long long)grid);
  TKV_WITH_TYPE(dtype, T, {
    if (!allow_smem(linrec_scan_kernel<T>, smem)) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_scan: state rows n=%d", n);
    TKV_CHECK_LAUNCH(launch_pdl(linrec_scan_kernel<T>, dim3((unsigned)grid), dim3(kScanWarps * 32), smem, (cudaStream_t)stream, a), "tkv_linrec_scan");
  });
  return check_launch("tkv_linrec_scan");
}
