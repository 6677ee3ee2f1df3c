// Routing of a mixture of experts, and the grouped product for every size and type:
//   moe_route_kernel : softmax scores, choice among the experts of the best groups, weights, and each choice's rank among the
//                      choices of its expert; with one CTA (few tokens) also the places;
//   moe_place_kernel : first row of every expert, row of every choice, token of every row;
//   moe_any_kernel   : grouped product on the CUDA cores.
// The last `identity` experts return their input: they own no rows, their choices get place -1.
#include "tkv_moe.cuh"

namespace tkv {

constexpr int kRouteThreads = 1024, kRouteWarps = kRouteThreads / 32, kRoutePerWarp = 4;
constexpr int kRouteTokens = kRouteWarps * kRoutePerWarp;  // tokens of a CTA
constexpr int kMaxExperts = 1024, kMaxTop = 64;

struct MoeRoute {
  const float* logits; int64_t stride;                    // [tokens, experts]
  const float* correction;                                // [experts]
  int tokens, experts, identity, top, groups, keep;       // experts: all of them, the identity ones last
  float scale;
  float* weight;                                          // [tokens, top]
  int32_t* choice;                                        // [tokens, top]
  int32_t* place;                                         // [tokens, top]: row, -1 for an identity expert (multi-CTA: rank until placed)
  int32_t* src;                                           // [tokens * top]: token of every row
  int32_t* counts;                                        // [experts], zero on entry (multi-CTA only)
  int32_t* offsets;                                       // [experts - identity + 1]
};

// Exclusive sums of the counts of the experts that own rows, by one warp; off[n] = total.
__device__ __forceinline__ void warp_offsets(const int32_t* counts, int n, int32_t* off) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int e0 = 0; e0 < n; e0 += 32) {
    const int c = e0 + lane < n ? counts[e0 + lane] : 0;
    int x = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    if (e0 + lane < n) off[e0 + lane] = base + x - c;
    base += __shfl_sync(0xffffffffu, x, 31);
  }
  if (lane == 0) off[n] = base;
}

// One warp per token, kRoutePerWarp tokens in turn; lane l holds experts l, l + 32, .. (kPer of them).  A choice is the largest
// order-preserving integer image of the choice scores over the warp, the lowest expert on a tie.
template <int kPer>
__global__ void __launch_bounds__(kRouteThreads) moe_route_kernel(MoeRoute p) {
  extern __shared__ float sm[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = p.experts, real = E - p.identity;
  float* cs = sm + (size_t)warp * (E + p.groups);         // choice scores of the warp's token, then the groups' best
  float* gs = cs + E;
  int32_t* hist = reinterpret_cast<int32_t*>(sm + (size_t)kRouteWarps * (E + p.groups));   // [E]
  int32_t* base = hist + E;                               // [E + 1]
  grid_dependency_wait();
  grid_launch_dependents();
  for (int e = threadIdx.x; e < E; e += kRouteThreads) hist[e] = 0;
  __syncthreads();
  const int size = E / p.groups;
  const bool all_open = p.keep >= p.groups;
  float corr[kPer];
  int group[kPer];
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int e = lane + 32 * i;
    corr[i] = e < E ? p.correction[e] : 0.f;
    group[i] = e < E ? e / size : 0;
  }
  const int tok0 = blockIdx.x * kRouteTokens;
  for (int it = 0; it < kRoutePerWarp; ++it) {
    const int t = tok0 + it * kRouteWarps + warp;
    if (t >= p.tokens) break;
    const float* z = p.logits + (int64_t)t * p.stride;
    float s[kPer], top = -INFINITY, sum = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      s[i] = lane + 32 * i < E ? z[lane + 32 * i] : -INFINITY;
      top = fmaxf(top, s[i]);
    }
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      s[i] = lane + 32 * i < E ? expf(s[i] - top) : 0.f;
      sum += s[i];
    }
    const float inv = 1.0f / warp_add(sum);
    uint32_t key[kPer];                                   // 0: not open
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      s[i] *= inv;
      key[i] = lane + 32 * i < E ? max(score_key(s[i] + corr[i]), 1u) : 0u;
    }
    if (!all_open) {
#pragma unroll
      for (int i = 0; i < kPer; ++i)
        if (lane + 32 * i < E) cs[lane + 32 * i] = s[i] + corr[i];
      __syncwarp();
      for (int g = lane; g < p.groups; g += 32) {
        float m = -INFINITY;
        for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, cs[e]);
        gs[g] = m;
      }
      __syncwarp();
      int last = -1;                                      // a group is kept if fewer than `keep` groups come before it
      bool open = false;
#pragma unroll
      for (int i = 0; i < kPer; ++i) {
        if (lane + 32 * i >= E) continue;
        if (group[i] != last) {
          last = group[i];
          const float mine = gs[last];
          int before = 0;
          for (int g = 0; g < p.groups; ++g) before += gs[g] > mine || (gs[g] == mine && g < last);
          open = before < p.keep;
        }
        if (!open) key[i] = 0u;
      }
      __syncwarp();
    }
    float picked = 0.f;                                   // lane c (and c + 32): choice c
    int mine[2] = {-1, -1};
    float mine_w[2] = {0.f, 0.f};
    for (int c = 0; c < p.top; ++c) {
      uint32_t best = 0u;
      int at = 0;
      float w = 0.f;
#pragma unroll
      for (int i = 0; i < kPer; ++i)
        if (key[i] > best) { best = key[i]; at = lane + 32 * i; w = s[i]; }
      const uint32_t top_key = __reduce_max_sync(0xffffffffu, best);
      const int winner = (int)__reduce_min_sync(0xffffffffu, best == top_key && best != 0u ? (uint32_t)at : 0x7fffffffu);
      // (fewer open experts than choices: the host refuses such sizes)
      const int e = min(winner, E - 1);
      w = __shfl_sync(0xffffffffu, w, e & 31);
#pragma unroll
      for (int i = 0; i < kPer; ++i)
        if (lane + 32 * i == e) key[i] = 0u;
      picked += w;
      if (lane == (c & 31)) { mine[c >> 5] = e; mine_w[c >> 5] = w; }
    }
    const float norm = p.scale / (picked + 1e-20f);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int c = lane + 32 * k;
      if (c < p.top) {
        const int64_t o = (int64_t)t * p.top + c;
        const bool owns = mine[k] < real;
        p.weight[o] = mine_w[k] * norm;
        p.choice[o] = mine[k];
        p.place[o] = owns ? atomicAdd(&hist[mine[k]], 1) : -1;           // rank within the CTA
      }
    }
    __syncwarp();
  }
  __syncthreads();
  const bool single = gridDim.x == 1;
  if (single) {
    if (warp == 0) {
      warp_offsets(hist, real, base);
      __syncwarp();
      for (int e = lane; e <= real; e += 32) p.offsets[e] = base[e];
    }
  } else {
    for (int e = threadIdx.x; e < real; e += kRouteThreads) base[e] = hist[e] > 0 ? atomicAdd(&p.counts[e], hist[e]) : 0;
  }
  __syncthreads();
  const int n = min(kRouteTokens, p.tokens - tok0) * p.top;
  for (int i = threadIdx.x; i < n; i += kRouteThreads) {
    const int64_t o = (int64_t)tok0 * p.top + i;
    if (p.place[o] < 0) continue;
    const int at = p.place[o] + base[p.choice[o]];        // single: the row; else: the rank among all tokens
    p.place[o] = at;
    if (single) p.src[at] = tok0 + i / p.top;
  }
}

constexpr int kPlaceThreads = 256;

__global__ void __launch_bounds__(kPlaceThreads) moe_place_kernel(MoeRoute p) {
  extern __shared__ int32_t off[];                        // [real + 1]
  grid_dependency_wait();
  grid_launch_dependents();
  const int real = p.experts - p.identity;
  if (threadIdx.x < 32) {
    warp_offsets(p.counts, real, off);
    __syncwarp();
    if (blockIdx.x == 0)
      for (int e = threadIdx.x; e <= real; e += 32) p.offsets[e] = off[e];
  }
  __syncthreads();
  const int64_t n = (int64_t)p.tokens * p.top;
  for (int64_t i = (int64_t)blockIdx.x * kPlaceThreads + threadIdx.x; i < n; i += (int64_t)gridDim.x * kPlaceThreads) {
    const int rank = p.place[i];
    if (rank < 0) continue;
    const int at = off[p.choice[i]] + rank;
    p.place[i] = at;
    p.src[at] = (int32_t)(i / p.top);
  }
}

// ------------------------------------------------------------------------------------------------ any size, fp32 arithmetic
constexpr int kAnyM = 32, kAnyN = 64, kAnyK = 16, kAnyThreads = 256;

// One CTA per (row tile, column tile): 32 x 64 results, eight per thread.
template <typename T>
__global__ void __launch_bounds__(kAnyThreads) moe_any_kernel(GroupedGemm p) {
  __shared__ float sa[kAnyK][kAnyM + 1], sw[kAnyK][kAnyN + 1];
  grid_dependency_wait();
  grid_launch_dependents();
  int e, r0;
  if (!find_tile(p.offsets, p.experts, kAnyM, blockIdx.y, &e, &r0)) return;
  const int rows = min(kAnyM, p.offsets[e + 1] - r0), n0 = blockIdx.x * kAnyN;
  const T* W = (const T*)p.w + (int64_t)e * p.n * p.k;
  const int tr = threadIdx.x / 16, tc = threadIdx.x % 16;  // rows tr, tr + 16; columns tc + 16 i
  float acc[2][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kAnyK) {
    for (int i = threadIdx.x; i < kAnyM * kAnyK; i += kAnyThreads) {
      const int r = i / kAnyK, k = i - r * kAnyK;
      float x = 0.f;
      if (r < rows && k0 + k < p.k) {
        const int64_t row = p.src != nullptr ? p.src[r0 + r] : r0 + r;
        x = to_f32<T>(((const T*)p.a)[row * p.a_stride + k0 + k]);
      }
      sa[k][r] = x;
    }
    for (int i = threadIdx.x; i < kAnyN * kAnyK; i += kAnyThreads) {
      const int c = i / kAnyK, k = i - c * kAnyK;
      sw[k][c] = n0 + c < p.n && k0 + k < p.k ? to_f32<T>(W[(int64_t)(n0 + c) * p.k + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kAnyK; ++k) {
      const float a0 = sa[k][tr], a1 = sa[k][tr + 16];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float w = sw[k][tc + 16 * i];
        acc[0][i] = fmaf(a0, w, acc[0][i]);
        acc[1][i] = fmaf(a1, w, acc[1][i]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int r = tr + 16 * j;
    if (r >= rows) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = n0 + tc + 16 * i;
      if (c < p.n) ((T*)p.out)[(int64_t)(r0 + r) * p.n + c] = from_f32<T>(p.act == 1 ? gelu_erf(acc[j][i]) : acc[j][i]);
    }
  }
}

}  // namespace tkv

using namespace tkv;

extern "C" int tkv_moe_route(const float* logits, int64_t logit_stride, const float* correction, int tokens, int experts,
                             int identity, int top, int groups, int keep, float scale, float* weight, int32_t* choice,
                             int32_t* place, int32_t* src, int32_t* counts, int32_t* offsets, tkv_stream_t stream) {
  if (!logits || !correction || !weight || !choice || !place || !src || !offsets) return fail(TKV_ERR_ARG, "tkv_moe_route: NULL pointer argument");
  if (tokens < 0 || experts <= 0 || identity < 0 || identity >= experts || top <= 0 || groups <= 0 || experts % groups || keep <= 0 ||
      keep > groups || top > keep * (experts / groups) || logit_stride < experts)
    return fail(TKV_ERR_ARG, "tkv_moe_route: experts=%d identity=%d top=%d groups=%d keep=%d", experts, identity, top, groups, keep);
  if (experts > kMaxExperts || top > kMaxTop) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_route: experts=%d (at most %d), top=%d (at most %d)", experts, kMaxExperts, top, kMaxTop);
  if ((int64_t)tokens * top > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_route: %lld choices", (long long)tokens * top);
  cudaStream_t st = (cudaStream_t)stream;
  MoeRoute p = {logits, logit_stride, correction, tokens, experts, identity, top, groups, keep, scale, weight, choice, place, src, counts, offsets};
  const int ctas = (tokens + kRouteTokens - 1) / kRouteTokens;
  if (ctas > 1 && !counts) return fail(TKV_ERR_ARG, "tkv_moe_route: counts is needed for more than %d tokens", kRouteTokens);
  if (tokens == 0) return TKV_OK;
  const size_t smem = ((size_t)kRouteWarps * (experts + groups) + 2 * experts + 1) * sizeof(float);
  if (smem > 220 * 1024) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_route: experts=%d groups=%d", experts, groups);
  auto kern = experts <= 32 ? moe_route_kernel<1> : experts <= 64 ? moe_route_kernel<2> : experts <= 128 ? moe_route_kernel<4>
              : experts <= 256 ? moe_route_kernel<8> : moe_route_kernel<32>;
  cudaError_t e = smem > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
  if (e == cudaSuccess) e = launch_pdl(kern, dim3(ctas), dim3(kRouteThreads), smem, st, p);
  if (e == cudaSuccess && ctas > 1) {
    const int64_t blocks = ((int64_t)tokens * top + kPlaceThreads * 4 - 1) / (kPlaceThreads * 4);
    e = launch_pdl(moe_place_kernel, dim3((unsigned)blocks), dim3(kPlaceThreads), (size_t)(experts + 1) * sizeof(int32_t), st, p);
  }
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_moe_route: %s", cudaGetErrorString(e));
  return check_launch("tkv_moe_route");
}

extern "C" int tkv_moe_gemm(const void* a, int64_t a_stride, int64_t a_rows, const int32_t* src, const void* w,
                            const int32_t* offsets, void* out, int64_t max_rows, int experts, int n, int k, int act, int dtype,
                            int32_t* status, tkv_stream_t stream) {
  if (!a || !w || !offsets || !out) return fail(TKV_ERR_ARG, "tkv_moe_gemm: NULL pointer argument");
  if (!is_model_dtype(dtype)) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_gemm: dtype %d", dtype);
  if (max_rows < 0 || a_rows < 0 || experts <= 0 || n <= 0 || k <= 0 || a_stride < k || act < 0 || act > 1 || (!src && a_rows < max_rows))
    return fail(TKV_ERR_ARG, "tkv_moe_gemm: bad sizes experts=%d n=%d k=%d act=%d", experts, n, k, act);
  if (max_rows == 0) return TKV_OK;
  if (max_rows > INT32_MAX || a_rows > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_gemm: %lld rows", (long long)max_rows);
  GroupedGemm p = {a, a_stride, a_rows, src, w, offsets, out, experts, n, k, act, max_rows, status};
  cudaStream_t st = (cudaStream_t)stream;
  if (moe_tc_shape(p, dtype)) return launch_moe_tc(p, st);
  const int64_t tiles = max_rows / kAnyM + (experts < max_rows ? experts : max_rows);
  if (tiles > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_gemm: %lld row tiles", (long long)tiles);
  const dim3 grid((n + kAnyN - 1) / kAnyN, (unsigned)tiles);
  cudaError_t e = dtype == TKV_BF16 ? launch_pdl(moe_any_kernel<__nv_bfloat16>, grid, dim3(kAnyThreads), 0, st, p)
                                    : launch_pdl(moe_any_kernel<float>, grid, dim3(kAnyThreads), 0, st, p);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_moe_gemm: %s", cudaGetErrorString(e));
  return check_launch("tkv_moe_gemm");
}
