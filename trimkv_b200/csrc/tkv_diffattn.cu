// Windowed differential attention: two softmax maps over the same values, combined and normed per head.
//
//   q rows [heads, 2, dim], k rows [kv_heads, 2, dim], v rows [kv_heads, vdim] of one projection; q and k are RMS-normed
//   per head and map; position i sees the `window` positions up to and including itself;
//   out_h = sigmoid(g_h) (1 - diff) rms(a1 - lambda a2).
//
// Storage.  Keys and values are held in rows padded with zeros to kp = 2 * dp and pp elements (dp, pp multiples of 64), so
// that the 16-bit kernels have one shape for every head size up to the padding:
//   ring   : k [slots, kv_heads, rows, 2, dp], v [slots, kv_heads, rows, pp]; position p lives in row p mod rows, and
//            rows >= min(window, tokens seen), so a decoding token sees exactly the rows that hold something;
//   linear : k [tokens, kv_heads, 2, dp], v [tokens, kv_heads, pp] of one step's tokens, each request's part preceded by
//            the positions before it that the window still reaches (fetched from the ring).
// Kernels here: diff_prep (norms, padding, ring and linear stores), ring_fetch, the split-KV decode kernel of the 16-bit
// type and its merge, and a kernel for every size in fp32 arithmetic.  The prompt kernel on tcgen05 is in
// tkv_diffattn_tc.cu.
#include "tkv_diffattn.cuh"
#include "tkv_ring.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kPrepThreads = 128;

// kVecLanes lanes per (token, vector): vectors are the 2 * heads query maps, the 2 * kv_heads key maps and the kv_heads
// values.  V: elements per access (8: dim, vdim and the row stride are multiples of 8).
constexpr int kVecLanes = 8;

template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) diff_prep_kernel(const T* proj, int64_t row_stride, const float* q_norm,
                                                                const float* k_norm, float eps, T* q_out, T* k_ring, T* v_ring,
                                                                int ring_rows, T* k_lin, T* v_lin, const int32_t* kv_start,
                                                                const int32_t* cu, const int32_t* slots, const int32_t* pos0,
                                                                int batch, int tokens, int heads, int kv_heads, int dim, int vdim,
                                                                int dp, int pp, int window) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = threadIdx.x & (kVecLanes - 1);
  const int vecs = 2 * heads + 3 * kv_heads;
  const int64_t items = (int64_t)tokens * vecs;
  const int64_t item_rt = (int64_t)blockIdx.x * (kPrepThreads / kVecLanes) + threadIdx.x / kVecLanes;
  const bool live = item_rt < items;                     // the rest of a warp takes part in its shuffles
  const int64_t item = live ? item_rt : items - 1;
  const int t = (int)(item / vecs), u = (int)(item - (int64_t)t * vecs);
  const bool is_q = u < 2 * heads, is_k = !is_q && u < 2 * (heads + kv_heads);
  const T* row = proj + (int64_t)t * row_stride;
  T *d0 = nullptr, *d1 = nullptr;                        // where the vector goes: q, or ring and linear buffer
  const T* src;
  if (is_q) {
    d0 = q_out + ((int64_t)t * 2 * heads + u) * dp;
    src = row + (int64_t)u * dim;
  } else {
    const int b = owner_of(cu, batch, t);
    const int i = cu != nullptr ? t - cu[b] : 0, n = cu != nullptr ? cu[b + 1] - cu[b] : 1;
    const int p0 = pos0[b], slot = slots[b], rr = (p0 + i) % ring_rows;
    const bool to_ring = i >= n - ring_rows;             // later tokens of the same step own the other rows
    const int64_t lin = k_lin != nullptr ? (int64_t)kv_start[b] + min(p0, window - 1) + i : 0;
    if (is_k) {
      const int km = u - 2 * heads, g = km >> 1, m = km & 1;
      if (to_ring) d0 = k_ring + ((((int64_t)slot * kv_heads + g) * ring_rows + rr) * 2 + m) * dp;
      if (k_lin != nullptr) d1 = k_lin + ((lin * kv_heads + g) * 2 + m) * dp;
      src = row + (int64_t)2 * heads * dim + (int64_t)km * dim;
    } else {
      const int g = u - 2 * (heads + kv_heads);
      if (to_ring) d0 = v_ring + (((int64_t)slot * kv_heads + g) * ring_rows + rr) * pp;
      if (v_lin != nullptr) d1 = v_lin + (lin * kv_heads + g) * pp;
      src = row + (int64_t)2 * (heads + kv_heads) * dim + (int64_t)g * vdim;
    }
  }
  const int len = is_q || is_k ? dim : vdim, padded = is_q || is_k ? dp : pp;
  const float* w = is_q ? q_norm : k_norm;
  float ss = 0.f;
  if (is_q || is_k)
    for (int i = lane * V; i < len; i += kVecLanes * V) {
      float x[V];
      load_vec<V>(src + i, x);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += x[e] * x[e];
    }
#pragma unroll
  for (int o = kVecLanes / 2; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!live) return;
  const float r = 1.0f / sqrtf(ss / (float)dim + eps);
  for (int i = lane * V; i < padded; i += kVecLanes * V) {
    float x[V];
    if (i < len) {
      load_vec<V>(src + i, x);
      if (is_q || is_k) {
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] *= r * w[i + e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] = 0.f;
    }
    if (d0 != nullptr) store_vec<V>(d0 + i, x);
    if (d1 != nullptr) store_vec<V>(d1 + i, x);
  }
}

// ------------------------------------------------------------------------------------------------ any size, fp32 arithmetic
constexpr int kAnyThreads = 128, kAnyCols = 4;            // vdim <= kAnyThreads * kAnyCols

// One CTA per (token, head).  Keys from the linear buffers (k_lin != nullptr) or from the ring (one token per request).
template <typename T>
__global__ void __launch_bounds__(kAnyThreads) diff_attn_any_kernel(DiffAttnParams p) {
  extern __shared__ float sm[];
  float* q = sm;                                          // [2][dim]
  float* w = q + 2 * p.dim;                               // [2][kAnyThreads]
  __shared__ float red[kAnyThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int t = blockIdx.x / p.heads, h = blockIdx.x - t * p.heads, g = h / (p.heads / p.kv_heads);
  const int b = owner_of(p.cu, p.batch, t), i = p.cu != nullptr ? t - p.cu[b] : 0;
  const int p0 = p.pos0[b], tid = threadIdx.x;
  int64_t k_row, v_row, k_step, v_step;
  const T *kb, *vb;
  int lo, hi;
  if (p.k_lin != nullptr) {
    const int hist = min(p0, p.window - 1);
    hi = hist + i + 1; lo = max(0, hi - p.window);
    kb = (const T*)p.k_lin; vb = (const T*)p.v_lin;
    k_row = ((int64_t)p.kv_start[b] * p.kv_heads + g) * 2 * p.dp; k_step = (int64_t)p.kv_heads * 2 * p.dp;
    v_row = ((int64_t)p.kv_start[b] * p.kv_heads + g) * p.pp; v_step = (int64_t)p.kv_heads * p.pp;
  } else {
    lo = 0; hi = min(p0 + 1, p.ring_rows);
    kb = (const T*)p.k_ring; vb = (const T*)p.v_ring;
    const int64_t r0 = ((int64_t)p.slots[b] * p.kv_heads + g) * p.ring_rows;
    k_row = r0 * 2 * p.dp; k_step = 2 * p.dp; v_row = r0 * p.pp; v_step = p.pp;
  }
  const T* qs = (const T*)p.q + ((int64_t)t * p.heads + h) * 2 * p.dp;
  for (int c = tid; c < 2 * p.dim; c += kAnyThreads) q[c] = to_f32<T>(qs[(c / p.dim) * p.dp + c % p.dim]);
  __syncthreads();
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, acc[2][kAnyCols] = {};
  for (int base = lo; base < hi; base += kAnyThreads) {
    const int j = base + tid, cnt = min(kAnyThreads, hi - base);
    float s[2] = {-INFINITY, -INFINITY};
    if (j < hi) {
      const T* kr = kb + k_row + (int64_t)j * k_step;
#pragma unroll
      for (int mp = 0; mp < 2; ++mp) {
        float a = 0.f;
        for (int c = 0; c < p.dim; ++c) a = fmaf(q[mp * p.dim + c], to_f32<T>(kr[mp * p.dp + c]), a);
        s[mp] = a * p.scale;
      }
    }
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float x = s[mp];
#pragma unroll
      for (int o = 16; o >= 1; o >>= 1) x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, o));
      if ((tid & 31) == 0) red[tid >> 5] = x;
      __syncthreads();
      float mx = m[mp];
#pragma unroll
      for (int k = 0; k < kAnyThreads / 32; ++k) mx = fmaxf(mx, red[k]);
      const float fix = expf(m[mp] - mx);                 // m = -inf before the first keys: 0
      m[mp] = mx;
      const float e = j < hi ? expf(s[mp] - mx) : 0.f;
      w[mp * kAnyThreads + tid] = e;
      l[mp] *= fix;
#pragma unroll
      for (int c = 0; c < kAnyCols; ++c) acc[mp][c] *= fix;
      __syncthreads();
    }
    for (int k = 0; k < cnt; ++k) {
      const float w0 = w[k], w1 = w[kAnyThreads + k];
      l[0] += w0; l[1] += w1;
      const T* vr = vb + v_row + (int64_t)(base + k) * v_step;
#pragma unroll
      for (int c = 0; c < kAnyCols; ++c) {
        const int col = tid + c * kAnyThreads;
        if (col < p.vdim) {
          const float x = to_f32<T>(vr[col]);
          acc[0][c] = fmaf(w0, x, acc[0][c]);
          acc[1][c] = fmaf(w1, x, acc[1][c]);
        }
      }
    }
    __syncthreads();
  }
  const float lam = *p.lambda;
  float o[kAnyCols], ss = 0.f;
#pragma unroll
  for (int c = 0; c < kAnyCols; ++c) {
    o[c] = tid + c * kAnyThreads < p.vdim ? acc[0][c] / l[0] - lam * (acc[1][c] / l[1]) : 0.f;
    ss += o[c] * o[c];
  }
  const float r = 1.0f / sqrtf(block_add<kAnyThreads>(ss, red) / (float)p.vdim + p.eps);
  const float gate = sigmoid_f32(to_f32<T>(((const T*)p.gate)[(int64_t)t * p.gate_stride + h])) * (1.0f - p.diff) * r;
  T* dst = (T*)p.out + ((int64_t)t * p.heads + h) * p.vdim;
#pragma unroll
  for (int c = 0; c < kAnyCols; ++c)
    if (tid + c * kAnyThreads < p.vdim) dst[tid + c * kAnyThreads] = from_f32<T>(o[c] * gate);
}

// ---------------------------------------------------------------------------------------------------- split-KV decode
// CTA = (a chunk of ring rows, (request, kv head), 8 query heads), four warps, each 16 rows at a time straight from global
// memory into mma.sync fragments (HBM-bound: no shared-memory staging).  MMA rows 0..7 are the first maps of up to eight
// query heads, rows 8..15 their second maps, so one P.V product serves both maps.  The contraction index of a product
// may be permuted as long as both operands agree, so a thread loads 16 contiguous bytes of a key (or of a value row) and
// uses its words as the fragments of two MMA steps.
constexpr int kDecWarps = 4;

// Ring rows per CTA: long chunks (their start and their merge cost what a few hundred rows do) as long as they fill the GPU.
static int dec_chunk(int64_t segments, int ring_rows) {
  for (int c = 1024; c > 256; c /= 2)
    if (segments * ((ring_rows + c - 1) / c) >= 148 * 6) return c;
  return 256;
}

__device__ __forceinline__ void mma16816(float* d, const uint32_t a0, const uint32_t a1, const uint32_t a2, const uint32_t a3,
                                         const uint32_t b0, const uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int KG /* dp / 32 */, int VG /* pp / 64 */>
__global__ void __launch_bounds__(kDecWarps * 32, KG == 2 ? 3 : 2) diff_decode_kernel(DiffAttnParams p) {
  constexpr int DP = KG * 32, PP = VG * 64;
  __shared__ float sm_o[kDecWarps][16][PP];
  __shared__ float sm_ml[kDecWarps][16][2];
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r = lane >> 2, c = lane & 3;
  const int chunk = blockIdx.x, seg = blockIdx.y, qg = blockIdx.z;
  const int b = seg / p.kv_heads, g = seg - b * p.kv_heads, hpg = p.heads / p.kv_heads;
  const int len = min(p.pos0[b] + 1, p.ring_rows);
  const int t0 = chunk * p.chunk, t1 = min(len, t0 + p.chunk);
  if (t0 >= len) return;
  const int nq = min(8, hpg - qg * 8);                    // query heads of this CTA
  const int64_t row0 = ((int64_t)p.slots[b] * p.kv_heads + g) * p.ring_rows;
  const __nv_bfloat16* K = (const __nv_bfloat16*)p.k_ring + row0 * 2 * DP;
  const __nv_bfloat16* V = (const __nv_bfloat16*)p.v_ring + row0 * PP;
  uint4 qf[2][KG];                                        // this thread's words of query head r, both maps
  {
    const __nv_bfloat16* q = (const __nv_bfloat16*)p.q + ((int64_t)b * p.heads + g * hpg + qg * 8 + r) * 2 * DP;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int d = 0; d < KG; ++d) qf[m][d] = r < nq ? ld16(q + m * DP + d * 32 + c * 8) : make_uint4(0, 0, 0, 0);
  }
  float o[VG][8][4] = {};
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  uint4 kf[2][2][KG];
  auto load_k = [&](int t) {
#pragma unroll
    for (int n8 = 0; n8 < 2; ++n8) {
      const int row = min(t + n8 * 8 + r, len - 1);       // rows beyond the end are masked below
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int d = 0; d < KG; ++d) kf[n8][m][d] = ld16_stream(K + ((int64_t)row * 2 + m) * DP + d * 32 + c * 8);
    }
  };
  for (int t = t0 + warp * 16; t < t1; t += kDecWarps * 16) {
    load_k(t);
    uint4 vf[4][VG];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int row = t + 2 * c + (k & 1) + (k >> 1) * 8;
#pragma unroll
      for (int v = 0; v < VG; ++v)
        vf[k][v] = row < len ? ld16_stream(V + (int64_t)row * PP + v * 64 + r * 8) : make_uint4(0, 0, 0, 0);
    }
    float s[2][4] = {};
#pragma unroll
    for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
      for (int d = 0; d < KG; ++d) {
        mma16816(s[n8], qf[0][d].x, 0u, qf[0][d].y, 0u, kf[n8][0][d].x, kf[n8][0][d].y);
        mma16816(s[n8], qf[0][d].z, 0u, qf[0][d].w, 0u, kf[n8][0][d].z, kf[n8][0][d].w);
        mma16816(s[n8], 0u, qf[1][d].x, 0u, qf[1][d].y, kf[n8][1][d].x, kf[n8][1][d].y);
        mma16816(s[n8], 0u, qf[1][d].z, 0u, qf[1][d].w, kf[n8][1][d].z, kf[n8][1][d].w);
      }
    float top[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const bool in = t + n8 * 8 + 2 * c + (e & 1) < len;
        s[n8][e] = in ? s[n8][e] * p.scale_log2 : -INFINITY;
        top[e >> 1] = fmaxf(top[e >> 1], s[n8][e]);
      }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      top[m] = fmaxf(top[m], __shfl_xor_sync(0xffffffffu, top[m], 1));
      top[m] = fmaxf(top[m], __shfl_xor_sync(0xffffffffu, top[m], 2));
      const float nm = fmaxf(mx[m], top[m]);              // finite: the first row of a step is always in range
      const float fix = exp2_weight(mx[m] - nm);
      mx[m] = nm;
      l[m] *= fix;
#pragma unroll
      for (int v = 0; v < VG; ++v)
#pragma unroll
        for (int j = 0; j < 8; ++j) { o[v][j][2 * m] *= fix; o[v][j][2 * m + 1] *= fix; }
#pragma unroll
      for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float w = exp2_weight(s[n8][2 * m + e] - nm);
          s[n8][2 * m + e] = w;
          l[m] += w;
        }
    }
    const uint32_t a0 = pack_bf16(s[0][0], s[0][1]), a1 = pack_bf16(s[0][2], s[0][3]);
    const uint32_t a2 = pack_bf16(s[1][0], s[1][1]), a3 = pack_bf16(s[1][2], s[1][3]);
#pragma unroll
    for (int v = 0; v < VG; ++v) {
      const uint32_t x[4][4] = {{vf[0][v].x, vf[0][v].y, vf[0][v].z, vf[0][v].w}, {vf[1][v].x, vf[1][v].y, vf[1][v].z, vf[1][v].w},
                                {vf[2][v].x, vf[2][v].y, vf[2][v].z, vf[2][v].w}, {vf[3][v].x, vf[3][v].y, vf[3][v].z, vf[3][v].w}};
#pragma unroll
      for (int j = 0; j < 8; ++j) {                       // n = r stands for dim v * 64 + r * 8 + j
        const uint32_t sel = (j & 1) ? 0x7632u : 0x5410u;
        mma16816(o[v][j], a0, a1, a2, a3, __byte_perm(x[0][j >> 1], x[1][j >> 1], sel), __byte_perm(x[2][j >> 1], x[3][j >> 1], sel));
      }
    }
  }
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 1);
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 2);
    if (c == 0) { sm_ml[warp][m * 8 + r][0] = mx[m]; sm_ml[warp][m * 8 + r][1] = l[m]; }
  }
  if (r < nq)
#pragma unroll
  for (int v = 0; v < VG; ++v)
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) sm_o[warp][(e >> 1) * 8 + r][v * 64 + (2 * c + (e & 1)) * 8 + j] = o[v][j][e];
  __syncthreads();
  const int64_t part = ((int64_t)seg * gridDim.z + qg) * gridDim.x + chunk;
  for (int i = threadIdx.x; i < 16 * PP; i += kDecWarps * 32) {
    const int row = i / PP, col = i - row * PP;
    if ((row & 7) >= nq) continue;
    float top = -INFINITY;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) top = fmaxf(top, sm_ml[w][row][0]);
    float a = 0.f, sum = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {                 // a warp without rows has -inf: weight 0
      const float f = exp2_weight(sm_ml[w][row][0] - top);
      a = fmaf(f, sm_o[w][row][col], a);
      sum = fmaf(f, sm_ml[w][row][1], sum);
    }
    p.part_o[(part * 16 + row) * PP + col] = a;
    if (col == 0) { p.part_ml[(part * 16 + row) * 2] = top; p.part_ml[(part * 16 + row) * 2 + 1] = sum; }
  }
}

// Merge of the chunks, combination of the maps, norm and gate.  One CTA per (request, query head).
template <typename T>
__global__ void __launch_bounds__(kAnyThreads) diff_merge_kernel(DiffAttnParams p, int nchunks, int qgroups) {
  __shared__ float red[kAnyThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x / p.heads, h = blockIdx.x - b * p.heads, hpg = p.heads / p.kv_heads, g = h / hpg, hh = h - g * hpg;
  const int len = min(p.pos0[b] + 1, p.ring_rows), used = (len + p.chunk - 1) / p.chunk;
  const int64_t part = (((int64_t)b * p.kv_heads + g) * qgroups + (hh >> 3)) * nchunks;
  const int tid = threadIdx.x;
  float a[2][2] = {}, sum[2] = {0.f, 0.f};
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const int row = m * 8 + (hh & 7);
    float top = -INFINITY;
    for (int k = 0; k < used; ++k) top = fmaxf(top, p.part_ml[((part + k) * 16 + row) * 2]);
    for (int k = 0; k < used; ++k) {
      const float f = exp2_weight(p.part_ml[((part + k) * 16 + row) * 2] - top);
      sum[m] = fmaf(f, p.part_ml[((part + k) * 16 + row) * 2 + 1], sum[m]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int col = tid + e * kAnyThreads;
        if (col < p.vdim) a[m][e] = fmaf(f, p.part_o[((part + k) * 16 + row) * p.pp + col], a[m][e]);
      }
    }
  }
  const float lam = *p.lambda;
  float o[2], ss = 0.f;
#pragma unroll
  for (int e = 0; e < 2; ++e) { o[e] = a[0][e] / sum[0] - lam * (a[1][e] / sum[1]); ss += o[e] * o[e]; }
  const float r = 1.0f / sqrtf(block_add<kAnyThreads>(ss, red) / (float)p.vdim + p.eps);
  const float gate = sigmoid_f32(to_f32<T>(((const T*)p.gate)[(int64_t)b * p.gate_stride + h])) * (1.0f - p.diff) * r;
  T* dst = (T*)p.out + ((int64_t)b * p.heads + h) * p.vdim;
#pragma unroll
  for (int e = 0; e < 2; ++e)
    if (tid + e * kAnyThreads < p.vdim) dst[tid + e * kAnyThreads] = from_f32<T>(o[e] * gate);
}

static bool fast_shape(int dp, int pp, int dtype) {
  return dtype == TKV_BF16 && (dp == 64 || dp == 128) && (pp == 64 || pp == 128);
}

static int check_diff_sizes(const char* what, int batch, int heads, int kv_heads, int dim, int vdim, int dp, int pp, int window,
                            int dtype) {
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "%s: dtype %d", what, dtype);
  if (batch < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || dp < dim || pp < vdim || dp % 64 ||
      pp % 64 || window <= 0)
    return fail(TKV_ERR_ARG, "%s: bad sizes heads=%d kv_heads=%d dim=%d vdim=%d dp=%d pp=%d window=%d", what, heads, kv_heads, dim, vdim,
                dp, pp, window);
  return TKV_OK;
}

}  // namespace tkv

using namespace tkv;

extern "C" int tkv_diff_prep(const void* proj, int64_t row_stride, const float* q_norm, const float* k_norm, float eps, void* q_out,
                             void* k_ring, void* v_ring, int ring_rows, void* k_lin, void* v_lin, const int32_t* kv_start,
                             const int32_t* cu_tokens, const int32_t* slots, const int32_t* pos0, int batch, int tokens,
                             int max_history, int heads, int kv_heads, int dim, int vdim, int dp, int pp, int window, int dtype,
                             tkv_stream_t stream) {
  if (!proj || !q_norm || !k_norm || !q_out || !k_ring || !v_ring || !slots || !pos0)
    return fail(TKV_ERR_ARG, "tkv_diff_prep: NULL pointer argument");
  if ((k_lin == nullptr) != (v_lin == nullptr) || (k_lin != nullptr && (!kv_start || !cu_tokens)))
    return fail(TKV_ERR_ARG, "tkv_diff_prep: the linear buffers come with kv_start and cu_tokens");
  int rc = check_diff_sizes("tkv_diff_prep", batch, heads, kv_heads, dim, vdim, dp, pp, window, dtype);
  if (rc != TKV_OK) return rc;
  if (tokens < 0 || ring_rows <= 0 || ring_rows > window || max_history < 0 ||
      row_stride < (int64_t)2 * (heads + kv_heads) * dim + (int64_t)kv_heads * vdim)
    return fail(TKV_ERR_ARG, "tkv_diff_prep: bad sizes");
  if (!aligned16(q_out) || !aligned16(k_ring) || !aligned16(v_ring) || (k_lin && (!aligned16(k_lin) || !aligned16(v_lin))))
    return fail(TKV_ERR_ARG, "tkv_diff_prep: pointers must be 16-byte aligned");
  if (batch == 0 || tokens == 0) return TKV_OK;
  if (batch > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_diff_prep: batch=%d", batch);
  const int64_t items = (int64_t)tokens * (2 * heads + 3 * kv_heads);
  const int64_t grid = (items + kPrepThreads / kVecLanes - 1) / (kPrepThreads / kVecLanes);
  const bool vec = dim % 8 == 0 && vdim % 8 == 0 && (row_stride * elem_size(dtype)) % 16 == 0 && aligned16(proj);
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_diff_prep: %lld blocks", (long long)grid);
  TKV_WITH_TYPE(dtype, T, {
    if (k_lin != nullptr && max_history > 0) {            // before the new tokens overwrite the ring rows it reads
      const int hist = max_history < window - 1 ? max_history : window - 1;
      const dim3 fgrid((unsigned)(((int64_t)hist * kv_heads + kFetchThreads / 32 - 1) / (kFetchThreads / 32)), batch);
      if (fgrid.x > 0) {
        cudaError_t e = launch_pdl(ring_fetch_kernel<T>, fgrid, dim3(kFetchThreads), 0, (cudaStream_t)stream, (const T*)k_ring, (const T*)v_ring,
                                   ring_rows, (T*)k_lin, (T*)v_lin, kv_start, slots, pos0, kv_heads, 2 * dp, pp, window);
        if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_diff_prep: %s", cudaGetErrorString(e));
      }
    }
    cudaError_t e = launch_pdl(vec ? diff_prep_kernel<T, 8> : diff_prep_kernel<T, 1>, dim3((unsigned)grid), dim3(kPrepThreads), 0, (cudaStream_t)stream, (const T*)proj, row_stride,
                               q_norm, k_norm, eps, (T*)q_out, (T*)k_ring, (T*)v_ring, ring_rows, (T*)k_lin, (T*)v_lin, kv_start, cu_tokens,
                               slots, pos0, batch, tokens, heads, kv_heads, dim, vdim, dp, pp, window);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_diff_prep: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_diff_prep");
}

extern "C" int64_t tkv_diff_decode_workspace_bytes(int batch, int heads, int kv_heads, int ring_rows, int dp, int pp, int dtype) {
  if (!fast_shape(dp, pp, dtype) || batch <= 0 || kv_heads <= 0 || heads < kv_heads || ring_rows <= 0) return 0;
  const int chunk = dec_chunk((int64_t)batch * kv_heads, ring_rows);
  const int64_t chunks = (ring_rows + chunk - 1) / chunk, qg = (heads / kv_heads + 7) / 8;
  return (int64_t)batch * kv_heads * qg * chunks * 16 * (pp + 2) * (int64_t)sizeof(float);
}

extern "C" int tkv_diff_decode(const void* q, const void* k_ring, const void* v_ring, int ring_rows, const int32_t* slots,
                               const int32_t* pos0, const float* lambda, float diff, float scale, float eps, const void* gate,
                               int64_t gate_stride, void* out, void* workspace, int64_t workspace_bytes, int batch, int heads,
                               int kv_heads, int dim, int vdim, int dp, int pp, int dtype, tkv_stream_t stream) {
  if (!q || !k_ring || !v_ring || !slots || !pos0 || !lambda || !gate || !out) return fail(TKV_ERR_ARG, "tkv_diff_decode: NULL pointer argument");
  int rc = check_diff_sizes("tkv_diff_decode", batch, heads, kv_heads, dim, vdim, dp, pp, ring_rows, dtype);
  if (rc != TKV_OK) return rc;
  if (gate_stride < heads) return fail(TKV_ERR_ARG, "tkv_diff_decode: gate_stride");
  if (batch == 0) return TKV_OK;
  DiffAttnParams p = {};
  p.q = q; p.k_ring = k_ring; p.v_ring = v_ring; p.ring_rows = ring_rows; p.slots = slots; p.pos0 = pos0; p.lambda = lambda;
  p.diff = diff; p.scale = scale; p.scale_log2 = scale * 1.4426950408889634f; p.eps = eps; p.gate = gate; p.gate_stride = gate_stride;
  p.out = out; p.batch = batch; p.tokens = batch; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.dp = dp; p.pp = pp;
  p.window = ring_rows;
  if (!fast_shape(dp, pp, dtype)) return launch_diff_any(p, dtype, (cudaStream_t)stream);
  if (!aligned16(q) || !aligned16(k_ring) || !aligned16(v_ring)) return fail(TKV_ERR_ARG, "tkv_diff_decode: pointers must be 16-byte aligned");
  const int64_t need = tkv_diff_decode_workspace_bytes(batch, heads, kv_heads, ring_rows, dp, pp, dtype);
  if (!workspace || workspace_bytes < need) return fail(TKV_ERR_ARG, "tkv_diff_decode: workspace of %lld bytes, %lld needed", (long long)workspace_bytes, (long long)need);
  p.chunk = dec_chunk((int64_t)batch * kv_heads, ring_rows);
  const int chunks = (ring_rows + p.chunk - 1) / p.chunk, qg = (heads / kv_heads + 7) / 8;
  if ((int64_t)batch * kv_heads > 65535 || qg > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_diff_decode: batch * kv_heads = %lld", (long long)batch * kv_heads);
  p.part_o = (float*)workspace;
  p.part_ml = p.part_o + (int64_t)batch * kv_heads * qg * chunks * 16 * pp;
  const dim3 grid(chunks, batch * kv_heads, qg), block(kDecWarps * 32);
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e = dp == 64 ? (pp == 64 ? launch_pdl(diff_decode_kernel<2, 1>, grid, block, 0, st, p) : launch_pdl(diff_decode_kernel<2, 2>, grid, block, 0, st, p))
                           : (pp == 64 ? launch_pdl(diff_decode_kernel<4, 1>, grid, block, 0, st, p) : launch_pdl(diff_decode_kernel<4, 2>, grid, block, 0, st, p));
  if (e == cudaSuccess) e = launch_pdl(diff_merge_kernel<__nv_bfloat16>, dim3(batch * heads), dim3(kAnyThreads), 0, st, p, chunks, qg);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_diff_decode: %s", cudaGetErrorString(e));
  return check_launch("tkv_diff_decode");
}

extern "C" int tkv_diff_prefill(const void* q, const void* k_lin, const void* v_lin, const int32_t* kv_start, int64_t kv_rows,
                                const int32_t* cu_tokens, const int32_t* pos0, const float* lambda, float diff, float scale, float eps,
                                const void* gate, int64_t gate_stride, void* out, int batch, int tokens, int max_tokens, int heads,
                                int kv_heads, int dim, int vdim, int dp, int pp, int window, int dtype, int32_t* status,
                                tkv_stream_t stream) {
  if (!q || !k_lin || !v_lin || !kv_start || !cu_tokens || !pos0 || !lambda || !gate || !out)
    return fail(TKV_ERR_ARG, "tkv_diff_prefill: NULL pointer argument");
  int rc = check_diff_sizes("tkv_diff_prefill", batch, heads, kv_heads, dim, vdim, dp, pp, window, dtype);
  if (rc != TKV_OK) return rc;
  if (tokens < 0 || max_tokens < 0 || max_tokens > tokens || kv_rows < tokens || gate_stride < heads)
    return fail(TKV_ERR_ARG, "tkv_diff_prefill: bad sizes");
  if (batch == 0 || tokens == 0) return TKV_OK;
  DiffAttnParams p = {};
  p.q = q; p.k_lin = k_lin; p.v_lin = v_lin; p.kv_start = kv_start; p.cu = cu_tokens; p.pos0 = pos0; p.lambda = lambda;
  p.diff = diff; p.scale = scale; p.scale_log2 = scale * 1.4426950408889634f; p.eps = eps; p.gate = gate; p.gate_stride = gate_stride;
  p.out = out; p.batch = batch; p.tokens = tokens; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.dp = dp; p.pp = pp;
  p.window = window; p.status = status;
  if (fast_shape(dp, pp, dtype) && scale > 0.f && kv_rows >= 128) return launch_diff_prefill_tc(p, kv_rows, max_tokens, (cudaStream_t)stream);
  return launch_diff_any(p, dtype, (cudaStream_t)stream);
}

namespace tkv {
int launch_diff_any(const DiffAttnParams& p, int dtype, cudaStream_t st) {
  if (p.vdim > kAnyThreads * kAnyCols) return fail(TKV_ERR_UNSUPPORTED, "differential attention: vdim=%d (at most %d)", p.vdim, kAnyThreads * kAnyCols);
  const size_t smem = ((size_t)2 * p.dim + 2 * kAnyThreads) * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "differential attention: dim=%d", p.dim);
  const int64_t grid = (int64_t)p.tokens * p.heads;
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "differential attention: %lld blocks", (long long)grid);
  cudaError_t e = dtype == TKV_BF16 ? launch_pdl(diff_attn_any_kernel<__nv_bfloat16>, dim3((unsigned)grid), dim3(kAnyThreads), smem, st, p)
                                    : launch_pdl(diff_attn_any_kernel<float>, dim3((unsigned)grid), dim3(kAnyThreads), smem, st, p);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "differential attention: %s", cudaGetErrorString(e));
  return check_launch("differential attention");
}
}  // namespace tkv
