// Latent attention (storage and score: tkv_latent.cuh):
//   latent_prep_kernel   : norm of the query latent; norm of the key/value latent, rotation of the shared key part, both into
//                          the ring and, for steps of several tokens, the linear buffer;
//   rotate_pairs_kernel  : rotary positions in place, dimension 2i with 2i + 1, on a part of every head;
//   two_part_any_kernel  : attention of every size and type;
//   latent_decode_kernel : one token per request in the latent space (queries absorbed into it): all heads share one key row
//                          of lw elements whose first cpad are also the value.  Split over the ring, merged by
//                          latent_merge_kernel.
// The prompt kernel on tcgen05 is in tkv_latent_tc.cu.
#include "tkv_latent.cuh"
#include "tkv_ring.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kLpThreads = 128;

struct LatentPrep {
  const void* u; int64_t u_stride;                       // row: [q_rank | kv_rank | rot_dim | ...]
  const float* q_norm; const float* kv_norm; float eps;
  const float2* freq;
  void* cq;                                              // [tokens, q_rank]
  void* ring; int ring_rows; void* lin; const int32_t* kv_start;
  const int32_t* cu; const int32_t* slots; const int32_t* pos0;
  int batch, q_rank, kv_rank, rot_dim, rot_dims, cpad, lw, window;
};

// One CTA per token.  V = 8: the ranks and the row stride are multiples of 8.
template <typename T, int V>
__global__ void __launch_bounds__(kLpThreads) latent_prep_kernel(LatentPrep p) {
  __shared__ float red[2][kLpThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x;
  const int b = owner_of(p.cu, p.batch, t);
  const int i = p.cu != nullptr ? t - p.cu[b] : 0, n = p.cu != nullptr ? p.cu[b + 1] - p.cu[b] : 1;
  const int p0 = p.pos0[b], pos = p0 + i;
  const T* uq = (const T*)p.u + (int64_t)t * p.u_stride;
  const T *uc = uq + p.q_rank, *ur = uc + p.kv_rank;
  float sq = 0.f, sc = 0.f;
  for (int c = tid * V; c < p.q_rank; c += kLpThreads * V) {
    float x[V];
    load_vec<V>(uq + c, x);
#pragma unroll
    for (int e = 0; e < V; ++e) sq += x[e] * x[e];
  }
  for (int c = tid * V; c < p.kv_rank; c += kLpThreads * V) {
    float x[V];
    load_vec<V>(uc + c, x);
#pragma unroll
    for (int e = 0; e < V; ++e) sc += x[e] * x[e];
  }
  const float rq = 1.0f / sqrtf(block_add<kLpThreads>(sq, red[0]) / (float)p.q_rank + p.eps);
  const float rc = 1.0f / sqrtf(block_add<kLpThreads>(sc, red[1]) / (float)p.kv_rank + p.eps);
  T* cq = (T*)p.cq + (int64_t)t * p.q_rank;
  for (int c = tid * V; c < p.q_rank; c += kLpThreads * V) {
    float x[V], w[V];
    load_vec<V>(uq + c, x);
    load_vec<V>(p.q_norm + c, w);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] *= rq * w[e];
    store_vec<V>(cq + c, x);
  }
  // later tokens of the same step own the ring rows of tokens that are more than the ring behind
  T* d0 = i >= n - p.ring_rows ? (T*)p.ring + ((int64_t)p.slots[b] * p.ring_rows + pos % p.ring_rows) * p.lw : nullptr;
  T* d1 = p.lin != nullptr ? (T*)p.lin + ((int64_t)p.kv_start[b] + min(p0, p.window - 1) + i) * p.lw : nullptr;
  for (int c = tid * V; c < p.cpad; c += kLpThreads * V) {
    float x[V];
    if (c < p.kv_rank) {
      float w[V];
      load_vec<V>(uc + c, x);
      load_vec<V>(p.kv_norm + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] *= rc * w[e];
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] = 0.f;
    }
    if (d0 != nullptr) store_vec<V>(d0 + c, x);
    if (d1 != nullptr) store_vec<V>(d1 + c, x);
  }
  for (int c = 2 * tid; c < p.lw - p.cpad; c += 2 * kLpThreads) {
    float x = c < p.rot_dim ? to_f32<T>(ur[c]) : 0.f, y = c + 1 < p.rot_dim ? to_f32<T>(ur[c + 1]) : 0.f;
    if (c < p.rot_dims) {
      float s, co;
      const float2 f = p.freq[c / 2];
      turn(pos, f.x, f.y, &s, &co);
      const float a = x * co - y * s;
      y = y * co + x * s;
      x = a;
    }
    if (d0 != nullptr) { d0[p.cpad + c] = from_f32<T>(x); d0[p.cpad + c + 1] = from_f32<T>(y); }
    if (d1 != nullptr) { d1[p.cpad + c] = from_f32<T>(x); d1[p.cpad + c + 1] = from_f32<T>(y); }
  }
}

// One CTA per token: elements [offset, offset + rot_dims) of every head of head_len elements.  V: 8 or 2 elements per access
// (V = 2 moves single elements).
template <typename T, int V>
__global__ void __launch_bounds__(kLpThreads) rotate_pairs_kernel(T* x, int64_t row_stride, const int32_t* cu, const int32_t* pos0,
                                                                 int batch, int heads, int head_len, int offset, int rot_dims,
                                                                 const float2* freq) {
  extern __shared__ float tab[];                         // sin [half], cos [half]
  grid_dependency_wait();
  grid_launch_dependents();
  const int t = blockIdx.x, half = rot_dims / 2;
  const int b = owner_of(cu, batch, t);
  const int pos = pos0[b] + (cu != nullptr ? t - cu[b] : 0);
  for (int i = threadIdx.x; i < half; i += kLpThreads) turn(pos, freq[i].x, freq[i].y, &tab[i], &tab[half + i]);
  __syncthreads();
  const int per = rot_dims / V;
  T* row = x + (int64_t)t * row_stride + offset;
  for (int i = threadIdx.x; i < heads * per; i += kLpThreads) {
    const int h = i / per, c = (i - h * per) * V;
    T* at = row + (int64_t)h * head_len + c;
    float v[V];
    if constexpr (V == 8) load_vec<8>(at, v);
    else { v[0] = to_f32<T>(at[0]); v[1] = to_f32<T>(at[1]); }
#pragma unroll
    for (int e = 0; e < V; e += 2) {
      const float s = tab[(c + e) / 2], co = tab[half + (c + e) / 2];
      const float a = v[e] * co - v[e + 1] * s;
      v[e + 1] = v[e + 1] * co + v[e] * s;
      v[e] = a;
    }
    if constexpr (V == 8) store_vec<8>(at, v);
    else { at[0] = from_f32<T>(v[0]); at[1] = from_f32<T>(v[1]); }
  }
}

// ------------------------------------------------------------------------------------------------ any size, fp32 arithmetic
constexpr int kTpThreads = 128, kTpCols = 8;              // vdim <= kTpThreads * kTpCols

// One CTA per (token, head).
template <typename T>
__global__ void __launch_bounds__(kTpThreads) two_part_any_kernel(TwoPartAttn p) {
  extern __shared__ float sm[];
  float *q1 = sm, *q2 = q1 + p.d1, *w = q2 + p.d2;        // w [kTpThreads]
  __shared__ float red[kTpThreads / 32];
  grid_dependency_wait();
  grid_launch_dependents();
  const int t = blockIdx.x / p.heads, h = blockIdx.x - t * p.heads;
  const int b = owner_of(p.cu, p.batch, t), i = p.cu != nullptr ? t - p.cu[b] : 0;
  const int p0 = p.pos0[b], tid = threadIdx.x;
  int64_t row0;
  int lo, hi;
  if (p.ring_rows > 0) {
    row0 = (int64_t)p.slots[b] * p.ring_rows;
    lo = 0; hi = min(p0 + 1, p.ring_rows);
  } else {
    row0 = p.kv_start[b];
    hi = min(p0, p.window - 1) + i + 1; lo = max(0, hi - p.window);
  }
  const T* a1 = (const T*)p.q1 + (int64_t)t * p.q1_token + (int64_t)h * p.q1_head;
  const T* a2 = (const T*)p.q2 + (int64_t)t * p.q2_token + (int64_t)h * p.q2_head;
  for (int c = tid; c < p.d1; c += kTpThreads) q1[c] = to_f32<T>(a1[c]);
  for (int c = tid; c < p.d2; c += kTpThreads) q2[c] = to_f32<T>(a2[c]);
  __syncthreads();
  float m = -INFINITY, l = 0.f, acc[kTpCols] = {};
  for (int base = lo; base < hi; base += kTpThreads) {
    const int j = base + tid, cnt = min(kTpThreads, hi - base);
    float s = -INFINITY;
    if (j < hi) {
      const T* k1 = (const T*)p.k1 + (row0 + j) * p.k1_row + (int64_t)h * p.k1_head;
      const T* k2 = (const T*)p.k2 + (row0 + j) * p.k2_row;
      float a = 0.f;
      for (int c = 0; c < p.d1; ++c) a = fmaf(q1[c], to_f32<T>(k1[c]), a);
      for (int c = 0; c < p.d2; ++c) a = fmaf(q2[c], to_f32<T>(k2[c]), a);
      s = a * p.scale;
    }
    float x = s;
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, o));
    if ((tid & 31) == 0) red[tid >> 5] = x;
    __syncthreads();
    float mx = m;
#pragma unroll
    for (int k = 0; k < kTpThreads / 32; ++k) mx = fmaxf(mx, red[k]);
    const float fix = expf(m - mx);                       // m = -inf before the first keys: 0
    m = mx;
    w[tid] = j < hi ? expf(s - mx) : 0.f;
    l *= fix;
#pragma unroll
    for (int c = 0; c < kTpCols; ++c) acc[c] *= fix;
    __syncthreads();
    for (int k = 0; k < cnt; ++k) {
      const float wk = w[k];
      l += wk;
      const T* vr = (const T*)p.v + (row0 + base + k) * p.v_row + (int64_t)h * p.v_head;
#pragma unroll
      for (int c = 0; c < kTpCols; ++c) {
        const int col = tid + c * kTpThreads;
        if (col < p.vdim) acc[c] = fmaf(wk, to_f32<T>(vr[col]), acc[c]);
      }
    }
    __syncthreads();
  }
  T* dst = (T*)p.out + (int64_t)t * p.out_token + (int64_t)h * p.out_head;
#pragma unroll
  for (int c = 0; c < kTpCols; ++c)
    if (tid + c * kTpThreads < p.vdim) dst[tid + c * kTpThreads] = from_f32<T>(acc[c] / l);
}

int launch_two_part_any(const char* what, const TwoPartAttn& p, int dtype, cudaStream_t st) {
  if (p.vdim > kTpThreads * kTpCols) return fail(TKV_ERR_UNSUPPORTED, "%s: values of %d elements (at most %d)", what, p.vdim, kTpThreads * kTpCols);
  const size_t smem = ((size_t)p.d1 + p.d2 + kTpThreads) * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "%s: keys of %d + %d elements", what, p.d1, p.d2);
  const int64_t grid = (int64_t)p.tokens * p.heads;
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "%s: %lld blocks", what, (long long)grid);
  cudaError_t e = dtype == TKV_BF16 ? launch_pdl(two_part_any_kernel<__nv_bfloat16>, dim3((unsigned)grid), dim3(kTpThreads), smem, st, p)
                                    : launch_pdl(two_part_any_kernel<float>, dim3((unsigned)grid), dim3(kTpThreads), smem, st, p);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "%s: %s", what, cudaGetErrorString(e));
  return check_launch(what);
}

// ---------------------------------------------------------------------------------------------------- split-KV decode
// CTA = (a chunk of ring rows, request, HG groups of 16 query heads), eight warps per group, 16 warps per SM, tiles of 32 rows
// through a ring of shared-memory stages (16-byte pieces XOR-swizzled by row) that the groups share.  Scores: a warp takes 16
// rows of the tile and a quarter of the contraction, its part of the queries stays in registers; softmax: a warp adds the
// quarters up and takes two heads; weighted sum: a warp takes cpad / 8 = 8 * NT value dims for the group's heads.  CTAs of the
// same rows and other heads are neighbours in the grid, so that the rows come from HBM once.
constexpr int kLdThreads = 256, kLdTile = 32, kLdHeads = 16;

struct LatentDecode {
  const void* q_abs; int64_t qa_token, qa_head;           // queries in the latent space, [.., cdim]
  const void* q_rot; int64_t qr_token, qr_head;           // rotary part before rotation, [.., rot_dim]
  const float2* freq; int rot_dim, rot_dims;
  const void* ring; int ring_rows, cdim, cpad, lw;
  const int32_t* slots; const int32_t* pos0;
  float scale_log2;
  int batch, heads, groups, chunk;
  float* part_o; float* part_ml;                          // [batch, groups, chunks, 16, cpad], [.., 2]
  void* out; int64_t out_token, out_head;
};

__device__ __forceinline__ void ld_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ld_x4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_x4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

template <int NT, int HG> struct LatentTile {
  static constexpr int R = kLdHeads, LW = 64 * (NT + 1), QS = LW + 8, SS = kLdTile + 8, PS = kLdTile + 8;
  static constexpr int kStageBytes = kLdTile * LW * 2, kStages = (NT >= 6 ? 2 : NT >= 4 ? 3 : NT >= 2 ? 4 : 6) * HG;
  static constexpr int kQBytes = R * QS * 2, kSBytes = 4 * R * SS * 4;           // the queries' place is taken by the scores
  static constexpr int kUnion = kQBytes > kSBytes ? kQBytes : kSBytes;
  static constexpr int kGroupBytes = kUnion + R * PS * 2 + R * 4;
  static constexpr int kBytes = kStages * kStageBytes + HG * kGroupBytes;
};

template <int NT, int HG>
__global__ void __launch_bounds__(kLdThreads * HG, 2 / HG) latent_decode_kernel(LatentDecode p) {
  using L = LatentTile<NT, HG>;
  constexpr int R = L::R, LW = L::LW, QS = L::QS, SS = L::SS, PS = L::PS, S = L::kStages, kPieces = LW / 8, KS = LW / 64;
  extern __shared__ __align__(128) uint8_t raw[];
  const int group = HG > 1 ? threadIdx.x / kLdThreads : 0, tid = threadIdx.x - group * kLdThreads;
  uint8_t* tiles = raw;                                                          // [S][32][LW] swizzled
  uint8_t* mine = raw + S * L::kStageBytes + group * L::kGroupBytes;
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(mine);                   // [R][QS], then
  float* s_s = reinterpret_cast<float*>(q_s);                                    // [4][R][SS]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(mine + L::kUnion);       // [R][PS]
  float* fix_s = reinterpret_cast<float*>(p_s + R * PS);                         // [R]
  auto group_sync = [&]() {
    if constexpr (HG == 1) __syncthreads();
    else asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "n"(kLdThreads) : "memory");
  };
  grid_dependency_wait();
  grid_launch_dependents();
  const int lane = tid & 31, warp = tid >> 5, gr = lane >> 2, gc = lane & 3;
  const int cgroups = (p.groups + HG - 1) / HG, chunk = blockIdx.x / cgroups, grp = (blockIdx.x - chunk * cgroups) * HG + group;
  const int b = blockIdx.y, h0 = grp * R, nh = max(0, min(R, p.heads - h0));      // a last CTA may have a group without heads
  const int pos = p.pos0[b], len = min(pos + 1, p.ring_rows);
  const int t0 = chunk * p.chunk, t1 = min(len, t0 + p.chunk);
  if (t0 >= len) return;
  const __nv_bfloat16* K = (const __nv_bfloat16*)p.ring + (int64_t)p.slots[b] * p.ring_rows * LW;
  auto fetch = [&](int t, int st) {                       // a group per tile, empty beyond the end
    const uint32_t dst = smem_u32(tiles) + st * L::kStageBytes;
    if (t < t1)
#pragma unroll
      for (int j = 0; j < (kLdTile * kPieces + kLdThreads * HG - 1) / (kLdThreads * HG); ++j) {
        const int i = threadIdx.x + j * kLdThreads * HG, r = i / kPieces, c = i - r * kPieces;
        if (kLdTile * kPieces % (kLdThreads * HG) != 0 && r >= kLdTile) break;
        const bool live = t + r < t1;                     // the rest reads as zeros
        const int bytes = live ? 16 : 0;
        const void* src = K + (live ? (int64_t)(t + r) * LW + c * 8 : 0);
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + (r * kPieces + (c ^ (r & 7))) * 16), "l"(src), "r"(bytes) : "memory");
      }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < S - 1; ++i) fetch(t0 + i * kLdTile, i);
  // ---- queries: absorbed part as it is, rotary part turned to this position
  for (int i = tid; i < R * NT * 64; i += kLdThreads) {
    const int r = i / (NT * 64), c = i - r * (NT * 64);
    q_s[r * QS + c] = r < nh && c < p.cdim ? ((const __nv_bfloat16*)p.q_abs)[(int64_t)b * p.qa_token + (int64_t)(h0 + r) * p.qa_head + c]
                                           : __float2bfloat16_rn(0.f);
  }
  {
    const int i = tid & 31, c = 2 * i;                    // pair i of heads warp, warp + 8, ..
    float s = 0.f, co = 1.f;
    if (c < p.rot_dims) turn(pos, p.freq[i].x, p.freq[i].y, &s, &co);
    for (int r = warp; r < R; r += kLdThreads / 32) {
      float x = 0.f, y = 0.f;
      if (r < nh && c < p.rot_dim) {
        const __nv_bfloat16* src = (const __nv_bfloat16*)p.q_rot + (int64_t)b * p.qr_token + (int64_t)(h0 + r) * p.qr_head + c;
        x = __bfloat162float(src[0]);
        if (c + 1 < p.rot_dim) y = __bfloat162float(src[1]);
      }
      q_s[r * QS + NT * 64 + c] = __float2bfloat16_rn(x * co - y * s);
      q_s[r * QS + NT * 64 + c + 1] = __float2bfloat16_rn(y * co + x * s);
    }
  }
  group_sync();
  const int rg = warp & 1, kq = warp >> 1;                // 16 rows of a tile, quarter of the contraction
  uint32_t qf[KS][4];
#pragma unroll
  for (int k = 0; k < KS; ++k)
    ld_x4(qf[k], smem_u32(q_s) + (uint32_t)((lane & 15) * QS + (kq * KS + k) * 16 + (lane >> 4) * 8) * 2);
  float o[NT][4] = {};
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const uint32_t p_addr = smem_u32(p_s);
  int st = 0;
  for (int t = t0; t < t1; t += kLdTile, st = st + 1 == S ? 0 : st + 1) {
    asm volatile("cp.async.wait_group %0;" ::"n"(S - 2) : "memory");
    __syncthreads();                                      // this tile is here; everyone is done with the last one
    fetch(t + (S - 1) * kLdTile, st == 0 ? S - 1 : st - 1);
    const uint32_t tile = smem_u32(tiles) + st * L::kStageBytes;
    // ---- scores
    {
      float acc[2][4] = {};
      const int row = rg * 16 + (lane & 7) + ((lane >> 4) & 1) * 8;
      const uint32_t krow = tile + (uint32_t)row * LW * 2;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t kf[4];
        ld_x4(kf, krow + (uint32_t)((((kq * KS + k) * 2 + ((lane >> 3) & 1)) ^ (row & 7)) * 16));
        ld_mma(acc[0], qf[k], kf[0], kf[1]);
        ld_mma(acc[1], qf[k], kf[2], kf[3]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2)
          *reinterpret_cast<float2*>(s_s + (kq * R + gr + (e >> 1) * 8) * SS + rg * 16 + n * 8 + 2 * gc) = make_float2(acc[n][e], acc[n][e + 1]);
    }
    group_sync();
    // ---- softmax of heads 2 warp, 2 warp + 1
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = warp * 2 + i;
      float x = 0.f;
#pragma unroll
      for (int q = 0; q < 4; ++q) x += s_s[(q * R + r) * SS + lane];
      x = t + lane < t1 ? x * p.scale_log2 : -INFINITY;
      float top = x;
#pragma unroll
      for (int d = 16; d >= 1; d >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, d));
      top = fmaxf(top, mx[i]);                            // finite: the first row of a tile is always in range
      const float fix = exp2_weight(mx[i] - top), w = exp2_weight(x - top);
      mx[i] = top;
      l[i] = fmaf(l[i], fix, w);                          // this lane's part of the sum
      p_s[r * PS + lane] = __float2bfloat16_rn(w);
      if (lane == 0) fix_s[r] = fix;
    }
    group_sync();
    // ---- weighted sum of the latents
    const float f0 = fix_s[gr], f1 = fix_s[gr + 8];
#pragma unroll
    for (int n = 0; n < NT; ++n) { o[n][0] *= f0; o[n][1] *= f0; o[n][2] *= f1; o[n][3] *= f1; }
#pragma unroll
    for (int k = 0; k < kLdTile / 16; ++k) {
      uint32_t pf[4];
      ld_x4(pf, p_addr + (uint32_t)((lane & 15) * PS + k * 16 + (lane >> 4) * 8) * 2);
      const int row = k * 16 + (lane & 15);
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t vf[4];
        const int c = warp * NT + min(n + (lane >> 4), NT - 1);
        ld_x4t(vf, tile + (uint32_t)row * LW * 2 + (uint32_t)((c ^ (row & 7)) * 16));
        ld_mma(o[n], pf, vf[0], vf[1]);
        if (n + 1 < NT) ld_mma(o[n + 1], pf, vf[2], vf[3]);
      }
    }
  }
  if (nh == 0) return;
  const int64_t part = (((int64_t)b * p.groups + grp) * (gridDim.x / cgroups) + chunk) * R;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float sum = warp_add(l[i]);
    const int r = warp * 2 + i;
    if (lane == 0) { p.part_ml[(part + r) * 2] = mx[i]; p.part_ml[(part + r) * 2 + 1] = sum; }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int r = gr + (e >> 1) * 8;
      if (r < nh) *reinterpret_cast<float2*>(p.part_o + (part + r) * p.cpad + (warp * NT + n) * 8 + 2 * gc) = make_float2(o[n][e], o[n][e + 1]);
    }
}

// Merge of the chunks.  One CTA per (request, head).
__global__ void __launch_bounds__(kLpThreads) latent_merge_kernel(LatentDecode p, int nchunks) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int b = blockIdx.x / p.heads, h = blockIdx.x - b * p.heads, grp = h / kLdHeads, r = h - grp * kLdHeads;
  const int len = min(p.pos0[b] + 1, p.ring_rows), used = (len + p.chunk - 1) / p.chunk;
  const int64_t part = ((int64_t)b * p.groups + grp) * nchunks;
  float top = -INFINITY, sum = 0.f;
  for (int k = 0; k < used; ++k) top = fmaxf(top, p.part_ml[((part + k) * kLdHeads + r) * 2]);
  for (int k = 0; k < used; ++k) {
    const float* ml = p.part_ml + ((part + k) * kLdHeads + r) * 2;
    sum = fmaf(exp2_weight(ml[0] - top), ml[1], sum);
  }
  __nv_bfloat16* dst = (__nv_bfloat16*)p.out + (int64_t)b * p.out_token + (int64_t)h * p.out_head;
  for (int c = threadIdx.x; c < p.cdim; c += kLpThreads) {
    float a = 0.f;
    for (int k = 0; k < used; ++k) {
      const int64_t at = (part + k) * kLdHeads + r;
      a = fmaf(exp2_weight(p.part_ml[at * 2] - top), p.part_o[at * p.cpad + c], a);
    }
    dst[c] = __float2bfloat16_rn(a / sum);
  }
}

static bool latent_decode_shape(int cdim, int rot_dim, int dtype) { return dtype == TKV_BF16 && cdim <= 512 && rot_dim >= 1 && rot_dim <= 64; }

// Rows of the ring per CTA: the smallest time under a simple cost (waves of CTAs, each its rows and a fixed start and merge).
static int latent_chunk(int batch, int groups, int ring_rows) {
  const int64_t segments = (int64_t)batch * (groups > 1 ? (groups + 1) / 2 : 1), width = 148 * (groups > 1 ? 1 : 2);
  int best = kLdTile;
  int64_t best_cost = -1;
  for (int c = kLdTile; c < ring_rows + kLdTile; c += kLdTile) {
    const int64_t ctas = segments * ((ring_rows + c - 1) / c), waves = (ctas + width - 1) / width;
    const int64_t cost = waves * (c + 128);
    if (best_cost < 0 || cost < best_cost) { best = c; best_cost = cost; }
  }
  return best;
}

}  // namespace tkv

using namespace tkv;

static int pad64(int n) { return (n + 63) / 64 * 64; }

extern "C" int tkv_latent_prep(const void* u, int64_t u_stride, const float* q_norm, const float* kv_norm, float eps, int q_rank,
                               int kv_rank, int rot_dim, int rot_dims, const float* freq_hi_lo, void* cq, void* ring, int ring_rows,
                               void* lin, const int32_t* kv_start, const int32_t* cu_tokens, const int32_t* slots,
                               const int32_t* pos0, int batch, int tokens, int max_history, int window, int dtype,
                               tkv_stream_t stream) {
  if (!u || !q_norm || !kv_norm || !cq || !ring || !slots || !pos0 || (rot_dims > 0 && !freq_hi_lo))
    return fail(TKV_ERR_ARG, "tkv_latent_prep: NULL pointer argument");
  if (lin != nullptr && (!kv_start || !cu_tokens)) return fail(TKV_ERR_ARG, "tkv_latent_prep: the linear buffer comes with kv_start and cu_tokens");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_prep: dtype %d", dtype);
  if (batch < 0 || tokens < 0 || q_rank <= 0 || kv_rank <= 0 || rot_dim < 0 || rot_dims < 0 || rot_dims > rot_dim || rot_dims % 2 ||
      ring_rows <= 0 || window <= 0 || ring_rows > window || max_history < 0 || u_stride < (int64_t)q_rank + kv_rank + rot_dim)
    return fail(TKV_ERR_ARG, "tkv_latent_prep: bad sizes q_rank=%d kv_rank=%d rot_dim=%d rot_dims=%d window=%d", q_rank, kv_rank, rot_dim, rot_dims, window);
  if (!aligned16(ring) || (lin && !aligned16(lin))) return fail(TKV_ERR_ARG, "tkv_latent_prep: pointers must be 16-byte aligned");
  if (batch == 0 || tokens == 0) return TKV_OK;
  if (batch > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_prep: batch=%d", batch);
  const int cpad = pad64(kv_rank), lw = cpad + pad64(rot_dim);
  LatentPrep p = {u, u_stride, q_norm, kv_norm, eps, (const float2*)freq_hi_lo, cq, ring, ring_rows, lin, kv_start, cu_tokens, slots, pos0,
                  batch, q_rank, kv_rank, rot_dim, rot_dims, cpad, lw, window};
  const bool vec = q_rank % 8 == 0 && kv_rank % 8 == 0 && (u_stride * elem_size(dtype)) % 16 == 0 && aligned16(u) && aligned16(cq) &&
                   aligned16(q_norm) && aligned16(kv_norm);
  cudaStream_t st = (cudaStream_t)stream;
  TKV_WITH_TYPE(dtype, T, {
    cudaError_t e = cudaSuccess;
    if (lin != nullptr && max_history > 0 && window > 1) {  // before the new tokens overwrite the ring rows it reads
      const int hist = max_history < window - 1 ? max_history : window - 1;
      e = launch_pdl(ring_fetch_kernel<T>, dim3((hist + kFetchThreads / 32 - 1) / (kFetchThreads / 32), batch), dim3(kFetchThreads), 0, st,
                     (const T*)ring, (const T*)nullptr, ring_rows, (T*)lin, (T*)nullptr, kv_start, slots, pos0, 1, lw, 0, window);
      if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_prep: %s", cudaGetErrorString(e));
    }
    e = launch_pdl(vec ? latent_prep_kernel<T, 8> : latent_prep_kernel<T, 1>, dim3(tokens), dim3(kLpThreads), 0, st, p);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_prep: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_latent_prep");
}

extern "C" int tkv_rotate_pairs(void* x, int64_t row_stride, const int32_t* cu_tokens, const int32_t* pos0, int batch, int tokens,
                                int heads, int head_len, int offset, int rot_dims, const float* freq_hi_lo, int dtype,
                                tkv_stream_t stream) {
  if (!x || !pos0 || !freq_hi_lo) return fail(TKV_ERR_ARG, "tkv_rotate_pairs: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_rotate_pairs: dtype %d", dtype);
  if (batch < 0 || tokens < 0 || heads <= 0 || head_len <= 0 || offset < 0 || rot_dims < 0 || rot_dims % 2 || offset + rot_dims > head_len ||
      row_stride < (int64_t)heads * head_len)
    return fail(TKV_ERR_ARG, "tkv_rotate_pairs: bad sizes");
  if (tokens == 0 || batch == 0 || rot_dims == 0) return TKV_OK;
  const size_t smem = (size_t)rot_dims * sizeof(float);
  if (smem > 48 * 1024) return fail(TKV_ERR_UNSUPPORTED, "tkv_rotate_pairs: rot_dims=%d", rot_dims);
  const bool vec = head_len % 8 == 0 && offset % 8 == 0 && rot_dims % 8 == 0 && (row_stride * elem_size(dtype)) % 16 == 0 && aligned16(x);
  TKV_WITH_TYPE(dtype, T, {
    cudaError_t e = launch_pdl(vec ? rotate_pairs_kernel<T, 8> : rotate_pairs_kernel<T, 2>, dim3(tokens), dim3(kLpThreads), smem,
                               (cudaStream_t)stream, (T*)x, row_stride, cu_tokens, pos0, batch, heads, head_len, offset, rot_dims,
                               (const float2*)freq_hi_lo);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_rotate_pairs: %s", cudaGetErrorString(e));
  });
  return check_launch("tkv_rotate_pairs");
}

extern "C" int tkv_latent_prefill(const void* q, int64_t q_stride, const void* kv, int64_t kv_stride, const void* lin,
                                  const int32_t* kv_start, int64_t kv_rows, const int32_t* cu_tokens, const int32_t* pos0, float scale,
                                  void* out, int batch, int tokens, int max_tokens, int heads, int dim, int rot_dim, int vdim,
                                  int kv_rank, int window, int dtype, int32_t* status, tkv_stream_t stream) {
  if (!q || !kv || !lin || !kv_start || !cu_tokens || !pos0 || !out) return fail(TKV_ERR_ARG, "tkv_latent_prefill: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_prefill: dtype %d", dtype);
  if (batch < 0 || tokens < 0 || max_tokens < 0 || max_tokens > tokens || kv_rows < tokens || heads <= 0 || dim <= 0 || rot_dim < 0 ||
      vdim <= 0 || kv_rank <= 0 || window <= 0 || q_stride < (int64_t)heads * (dim + rot_dim) || kv_stride < (int64_t)heads * (dim + vdim))
    return fail(TKV_ERR_ARG, "tkv_latent_prefill: bad sizes heads=%d dim=%d rot_dim=%d vdim=%d window=%d", heads, dim, rot_dim, vdim, window);
  if (batch == 0 || tokens == 0) return TKV_OK;
  const int64_t es = elem_size(dtype);
  const int cpad = pad64(kv_rank), lw = cpad + pad64(rot_dim);
  TwoPartAttn p = {};
  p.q1 = q; p.q1_token = q_stride; p.q1_head = dim + rot_dim; p.d1 = dim;
  p.q2 = (const char*)q + dim * es; p.q2_token = q_stride; p.q2_head = dim + rot_dim; p.d2 = rot_dim;
  p.k1 = kv; p.k1_row = kv_stride; p.k1_head = dim;
  p.k2 = (const char*)lin + cpad * es; p.k2_row = lw;
  p.v = (const char*)kv + (int64_t)heads * dim * es; p.v_row = kv_stride; p.v_head = vdim; p.vdim = vdim;
  p.out = out; p.out_token = (int64_t)heads * vdim; p.out_head = vdim;
  p.kv_start = kv_start; p.cu = cu_tokens; p.pos0 = pos0; p.batch = batch; p.tokens = tokens; p.heads = heads; p.window = window;
  p.scale = scale; p.status = status;
  if (two_part_tc_shape(p, dtype)) return launch_two_part_tc(p, kv_rows, max_tokens, (cudaStream_t)stream);
  return launch_two_part_any("tkv_latent_prefill", p, dtype, (cudaStream_t)stream);
}

extern "C" int64_t tkv_latent_decode_workspace_bytes(int batch, int heads, int kv_rank, int rot_dim, int ring_rows, int dtype) {
  if (batch <= 0 || heads <= 0 || kv_rank <= 0 || rot_dim < 0 || ring_rows <= 0) return 0;
  if (!latent_decode_shape(kv_rank, rot_dim, dtype)) return -1;
  const int groups = (heads + kLdHeads - 1) / kLdHeads, cpad = pad64(kv_rank);
  const int chunk = latent_chunk(batch, groups, ring_rows);
  return (int64_t)batch * groups * ((ring_rows + chunk - 1) / chunk) * kLdHeads * (cpad + 2) * (int64_t)sizeof(float);
}

namespace tkv {
template <int NT, int HG>
static int launch_latent_decode(const LatentDecode& p, int chunks, cudaStream_t st) {
  constexpr int kBytes = LatentTile<NT, HG>::kBytes;
  const dim3 grid(chunks * ((p.groups + HG - 1) / HG), p.batch);
  static_assert(kBytes <= 232448, "shared memory of the kernel");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NT, HG>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_decode: %s", cudaGetErrorString(e));
    configured = true;
  }
  cudaError_t e = launch_pdl(latent_decode_kernel<NT, HG>, grid, dim3(kLdThreads * HG), (size_t)kBytes, st, p);
  if (e == cudaSuccess) e = launch_pdl(latent_merge_kernel, dim3((unsigned)(p.batch * p.heads)), dim3(kLpThreads), 0, st, p, chunks);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_decode: %s", cudaGetErrorString(e));
  return check_launch("tkv_latent_decode");
}
template <int HG>
static int launch_latent_decode_nt(const LatentDecode& p, int chunks, cudaStream_t st) {
  switch (p.cpad / 64) {
    case 1: return launch_latent_decode<1, HG>(p, chunks, st);
    case 2: return launch_latent_decode<2, HG>(p, chunks, st);
    case 3: return launch_latent_decode<3, HG>(p, chunks, st);
    case 4: return launch_latent_decode<4, HG>(p, chunks, st);
    case 5: return launch_latent_decode<5, HG>(p, chunks, st);
    case 6: return launch_latent_decode<6, HG>(p, chunks, st);
    case 7: return launch_latent_decode<7, HG>(p, chunks, st);
    default: return launch_latent_decode<8, HG>(p, chunks, st);
  }
}
}  // namespace tkv

extern "C" int tkv_latent_decode(const void* q_abs, int64_t qa_token, int64_t qa_head, const void* q_rot, int64_t qr_token,
                                 int64_t qr_head, const float* freq_hi_lo, const void* ring, int ring_rows, const int32_t* slots,
                                 const int32_t* pos0, float scale, void* out, int64_t out_token, int64_t out_head, void* workspace,
                                 int64_t workspace_bytes, int batch, int heads, int kv_rank, int rot_dim, int rot_dims, int dtype,
                                 tkv_stream_t stream) {
  if (!q_abs || !q_rot || !ring || !slots || !pos0 || !out || (rot_dims > 0 && !freq_hi_lo))
    return fail(TKV_ERR_ARG, "tkv_latent_decode: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_decode: dtype %d", dtype);
  if (batch < 0 || heads <= 0 || kv_rank <= 0 || rot_dim < 0 || rot_dims < 0 || rot_dims > rot_dim || rot_dims % 2 || ring_rows <= 0 || !aligned16(ring))
    return fail(TKV_ERR_ARG, "tkv_latent_decode: bad sizes heads=%d kv_rank=%d rot_dim=%d rot_dims=%d", heads, kv_rank, rot_dim, rot_dims);
  if (batch == 0) return TKV_OK;
  const int cpad = pad64(kv_rank), lw = cpad + pad64(rot_dim);
  const int64_t es = elem_size(dtype);
  if (!latent_decode_shape(kv_rank, rot_dim, dtype)) {    // q_rot already rotated by the caller (tkv_rotate_pairs)
    TwoPartAttn p = {};
    p.q1 = q_abs; p.q1_token = qa_token; p.q1_head = qa_head; p.d1 = kv_rank;
    p.q2 = q_rot; p.q2_token = qr_token; p.q2_head = qr_head; p.d2 = rot_dim;
    p.k1 = ring; p.k1_row = lw; p.k2 = (const char*)ring + cpad * es; p.k2_row = lw;
    p.v = ring; p.v_row = lw; p.vdim = kv_rank;
    p.out = out; p.out_token = out_token; p.out_head = out_head;
    p.slots = slots; p.ring_rows = ring_rows; p.pos0 = pos0; p.batch = batch; p.tokens = batch; p.heads = heads; p.window = ring_rows;
    p.scale = scale;
    return launch_two_part_any("tkv_latent_decode", p, dtype, (cudaStream_t)stream);
  }
  const int64_t need = tkv_latent_decode_workspace_bytes(batch, heads, kv_rank, rot_dim, ring_rows, dtype);
  if (!workspace || workspace_bytes < need)
    return fail(TKV_ERR_ARG, "tkv_latent_decode: workspace of %lld bytes, %lld needed", (long long)workspace_bytes, (long long)need);
  if (batch > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_decode: batch=%d", batch);
  const int groups = (heads + kLdHeads - 1) / kLdHeads;
  LatentDecode p = {q_abs, qa_token, qa_head, q_rot, qr_token, qr_head, (const float2*)freq_hi_lo, rot_dim, rot_dims, ring, ring_rows, kv_rank,
                    cpad, lw, slots, pos0, scale * 1.4426950408889634f, batch, heads, groups, latent_chunk(batch, groups, ring_rows),
                    nullptr, nullptr, out, out_token, out_head};
  const int chunks = (ring_rows + p.chunk - 1) / p.chunk;
  p.part_o = (float*)workspace;
  p.part_ml = p.part_o + (int64_t)batch * groups * chunks * kLdHeads * cpad;
  return groups > 1 ? launch_latent_decode_nt<2>(p, chunks, (cudaStream_t)stream) : launch_latent_decode_nt<1>(p, chunks, (cudaStream_t)stream);
}
