// Channel-decay recurrence (see tkv_chanrec.cuh), one token at a time:
//   chanrec_step_kernel : one token per request: gate, state update, read-out, RMS norm per head in one pass;
//   chanrec_scan_kernel : any number of tokens, every size and type, state in shared memory.
// A request whose start position is 0 starts from the zero state whatever its slot held before.
#include "tkv_chanrec.cuh"
#include "tkv_state_step.cuh"

namespace tkv {

// One CTA per (request, head).
template <typename T, int V>
__global__ void __launch_bounds__(kStepThreads) chanrec_step_kernel(ChanrecParams a, const float* norm_w, float eps) {
  extern __shared__ float sm[];
  float *q = sm, *f = q + a.n, *k = f + a.n, *v = k + a.n, *o = v + a.p, *red = o + a.p;      // red: kStepThreads * 4
  __shared__ float wred[kStepThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x / a.heads, h = blockIdx.x - b * a.heads;
  StateStep<V> step;
  step.prefetch(a.state + ((int64_t)a.slots[b] * a.heads + h) * a.n * a.p, a.n, a.p, a.pos0[b] == 0);
  const int64_t row = (int64_t)b * a.row_stride;
  const T *zq = (const T*)a.q + row + (int64_t)h * a.n, *zf = (const T*)a.f + row + (int64_t)h * a.n;
  const T* zv = (const T*)a.v + row + (int64_t)h * a.p;
  for (int i = threadIdx.x; i < a.n; i += kStepThreads) {
    q[i] = silu_f32(to_f32<T>(zq[i]));
    forget_gate(to_f32<T>(zf[i]) + a.f_bias[h * a.n + i], a.lower[h * a.n + i], &f[i], &k[i]);
  }
  for (int i = threadIdx.x; i < a.p; i += kStepThreads) v[i] = to_f32<T>(zv[i]);
  __syncthreads();
  step.run([f](int r) { return f[r]; }, k, q, v, o, red);
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.p; i += kStepThreads) ss += o[i] * o[i];
  const float rstd = 1.0f / sqrtf(block_add<kStepThreads>(ss, wred) / (float)a.p + eps);
  T* dst = (T*)a.out + ((int64_t)b * a.heads + h) * a.p;
  for (int i = threadIdx.x; i < a.p; i += kStepThreads) dst[i] = from_f32<T>(o[i] * rstd * norm_w[i]);
}

constexpr int kScanWarps = 8;

// One CTA per (request, head, 32 columns of v): lane = column, warps share the rows of the state.
template <typename T>
__global__ void __launch_bounds__(kScanWarps * 32) chanrec_scan_kernel(ChanrecParams a) {
  extern __shared__ float sm[];
  float *S = sm, *gate = S + (int64_t)a.n * 32;       // [n][32]; two buffers of q, f, k [n]
  __shared__ float red[2][kScanWarps][32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ptiles = (a.p + 31) / 32;
  const int pt = blockIdx.x % ptiles, bh = blockIdx.x / ptiles;
  const int b = bh / a.heads, h = bh - b * a.heads;
  const int t0 = a.cu != nullptr ? a.cu[b] : b, t1 = a.cu != nullptr ? a.cu[b + 1] : b + 1;
  if (t1 <= t0) return;
  const int col = pt * 32 + lane;
  const bool ok = col < a.p;
  float* G = a.state + ((int64_t)a.slots[b] * a.heads + h) * a.n * a.p;
  const bool fresh = a.pos0[b] == 0;
  for (int r = warp; r < a.n; r += kScanWarps) S[r * 32 + lane] = (ok && !fresh) ? G[(int64_t)r * a.p + col] : 0.f;
  const float *bias = a.f_bias + (int64_t)h * a.n, *lower = a.lower + (int64_t)h * a.n;
  auto gates = [&](int t) {
    float* g = gate + (t & 1) * 3 * a.n;
    const int64_t at = (int64_t)t * a.row_stride + (int64_t)h * a.n;
    for (int i = threadIdx.x; i < a.n; i += kScanWarps * 32) {
      g[i] = silu_f32(to_f32<T>(((const T*)a.q)[at + i]));
      forget_gate(to_f32<T>(((const T*)a.f)[at + i]) + bias[i], lower[i], &g[a.n + i], &g[2 * a.n + i]);
    }
  };
  gates(t0);
  __syncthreads();
  for (int t = t0; t < t1; ++t) {
    const float *q = gate + (t & 1) * 3 * a.n, *f = q + a.n, *k = f + a.n;
    const float v = ok ? to_f32<T>(((const T*)a.v)[(int64_t)t * a.row_stride + (int64_t)h * a.p + col]) : 0.f;
    float acc = 0.f;
    for (int r = warp; r < a.n; r += kScanWarps) {
      const float s = fmaf(f[r], S[r * 32 + lane], k[r] * v);
      S[r * 32 + lane] = s;
      acc = fmaf(q[r], s, acc);
    }
    const int par = t & 1;                             // two buffers: one barrier per token
    red[par][warp][lane] = acc;
    if (t + 1 < t1) gates(t + 1);
    __syncthreads();
    if (warp == 0 && ok) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kScanWarps; ++w) o += red[par][w][lane];
      ((T*)a.out)[(int64_t)t * a.heads * a.p + (int64_t)h * a.p + col] = from_f32<T>(o);
    }
  }
  for (int r = warp; r < a.n; r += kScanWarps)
    if (ok) G[(int64_t)r * a.p + col] = S[r * 32 + lane];
}

static int check_chanrec(const char* what, const void* q, const void* f, const void* v, int64_t row_stride, const float* f_bias,
                         const float* lower, const void* out, const float* state, const int32_t* slots, const int32_t* pos0,
                         int batch, int heads, int n, int vdim, int dtype) {
  if (!q || !f || !v || !f_bias || !lower || !out || !state || !slots || !pos0) return fail(TKV_ERR_ARG, "%s: NULL pointer argument", what);
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "%s: dtype %d", what, dtype);
  if (batch < 0 || heads <= 0 || n <= 0 || vdim <= 0 || row_stride < (int64_t)heads * n || row_stride < (int64_t)heads * vdim)
    return fail(TKV_ERR_ARG, "%s: bad sizes heads=%d n=%d vdim=%d", what, heads, n, vdim);
  return TKV_OK;
}

}  // namespace tkv

using namespace tkv;

extern "C" int tkv_chanrec_step(const void* q, const void* f, const void* v, int64_t row_stride, const float* f_bias,
                                const float* lower, const float* norm_w, float eps, void* out, float* state, const int32_t* slots,
                                const int32_t* pos0, int batch, int heads, int n, int vdim, int dtype, tkv_stream_t stream) {
  int rc = check_chanrec("tkv_chanrec_step", q, f, v, row_stride, f_bias, lower, out, state, slots, pos0, batch, heads, n, vdim, dtype);
  if (rc != TKV_OK) return rc;
  if (!norm_w) return fail(TKV_ERR_ARG, "tkv_chanrec_step: NULL pointer argument");
  if (batch == 0) return TKV_OK;
  if ((int64_t)batch * heads > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_step: %lld blocks", (long long)batch * heads);
  ChanrecParams a = {q, f, v, row_stride, f_bias, lower, out, state, slots, nullptr, pos0, batch, heads, n, vdim};
  const size_t smem = ((size_t)3 * n + 2 * vdim + kStepThreads * 4) * sizeof(float);
  TKV_WITH_TYPE(dtype, T, {
    auto kern = vdim % 4 == 0 && aligned16(state) ? chanrec_step_kernel<T, 4> : chanrec_step_kernel<T, 1>;
    if (!allow_smem(kern, smem)) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_step: n=%d vdim=%d", n, vdim);
    cudaError_t e = launch_pdl(kern, dim3((unsigned)(batch * heads)), dim3(kStepThreads), smem, (cudaStream_t)stream, a, norm_w, eps);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_step: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_chanrec_step");
}

extern "C" int tkv_chanrec_scan(const void* q, const void* f, const void* v, int64_t row_stride, const float* f_bias,
                                const float* lower, void* out, float* state, const int32_t* slots, const int32_t* cu_tokens,
                                const int32_t* pos0, int batch, int heads, int n, int vdim, int dtype, tkv_stream_t stream) {
  int rc = check_chanrec("tkv_chanrec_scan", q, f, v, row_stride, f_bias, lower, out, state, slots, pos0, batch, heads, n, vdim, dtype);
  if (rc != TKV_OK) return rc;
  if (batch == 0) return TKV_OK;
  ChanrecParams a = {q, f, v, row_stride, f_bias, lower, out, state, slots, cu_tokens, pos0, batch, heads, n, vdim};
  const size_t smem = (size_t)n * (32 + 6) * sizeof(float);
  const int64_t grid = (int64_t)batch * heads * ((vdim + 31) / 32);
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_scan: %lld blocks", (long long)grid);
  TKV_WITH_TYPE(dtype, T, {
    if (!allow_smem(chanrec_scan_kernel<T>, smem)) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_scan: state rows n=%d", n);
    cudaError_t e = launch_pdl(chanrec_scan_kernel<T>, dim3((unsigned)grid), dim3(kScanWarps * 32), smem, (cudaStream_t)stream, a);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_scan: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_chanrec_scan");
}
