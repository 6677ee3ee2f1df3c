// Windowed attention with keys in two parts over many query tokens (prompts and portions of prompts) on tcgen05 + TMEM.
//
// One CTA = (request, head, block of 128 query tokens), key tiles of 128:
//   S[128 x 128]  = Q . K(tile)^T   two TMEM buffers (columns 0, 128); the key tile is fetched as 64-column pieces, the first
//                                   part from the head's keys, the second from the row that all heads share
//   online softmax (two threads per row), P in the 16-bit type through shared memory
//   O[128 x VH*64] += P . V(tile)   TMEM columns 256 ..
// Scores of tile j + 1 are computed while tile j is in the softmax.  Pieces beyond a part's width are zero-filled by the copy.
// A row sees the columns [lo, hi) of the request's linear keys; tiles before the first row's window are never loaded.  Waits
// are bounded; on expiry the CTA records TKV_DEV_TIMEOUT, drains its copies and frees its TMEM.
#include <cuda.h>
#include "tkv_attn_block.cuh"
#include "tkv_latent.cuh"

namespace tkv {

struct TpSmem {
  uint64_t bar_k[2], bar_v, bar_s[2], bar_o, bar_p, bar_x;
  uint32_t tmem_base;
  int abort_flag;
  float red[2][2][kDaTile];
};
template <int KH, int VH> constexpr int tp_smem_bytes() { return (3 * KH + VH + 2) * kDaHalf + (int)sizeof(TpSmem); }

// K1, K2: 64-element pieces of the two key parts; VH: of a value.
template <int K1, int K2, int VH>
__global__ void __launch_bounds__(kDaThreads, 1)
two_part_prefill_kernel(const __grid_constant__ CUtensorMap map_k1, const __grid_constant__ CUtensorMap map_k2,
                        const __grid_constant__ CUtensorMap map_v, TwoPartAttn p, int nblocks) {
  extern __shared__ __align__(1024) uint8_t base[];
  constexpr int KH = K1 + K2, kTileK = KH * kDaHalf, kTileV = VH * kDaHalf;
  constexpr int OD = VH * 32;                              // value elements per thread
  grid_dependency_wait();
  grid_launch_dependents();
  const int seg = (int)(blockIdx.x / (unsigned)nblocks);
  const int blk = nblocks - 1 - (int)(blockIdx.x % (unsigned)nblocks);
  const int tid = threadIdx.x, warp = tid >> 5;
  const bool is_ctrl = warp == 8;
  const int row = tid & (kDaTile - 1), half = (tid >> 7) & 1;
  const int b = seg / p.heads, head = seg - b * p.heads;
  const int tok0 = p.cu[b], n = p.cu[b + 1] - tok0;
  if (blk * kDaTile >= n) return;
  if ((smem_u32(base) & 1023u) != 0) {                     // the swizzled tiles need it; the launch gives it
    if (tid == 0) report(p.status, TKV_DEV_TIMEOUT);
    return;
  }
  const int hist = min(p.pos0[b], p.window - 1);
  const int len = hist + n;                                // linear rows of the request
  const bool row_valid = !is_ctrl && blk * kDaTile + row < n;
  const int token = row_valid ? blk * kDaTile + row : 0;
  const int hi_row = row_valid ? hist + token + 1 : 0, lo_row = max(0, hi_row - p.window);
  const int hi_max = hist + min(blk * kDaTile + kDaTile, n);
  const int lo_min = max(0, hist + blk * kDaTile + 1 - p.window);
  const int tile0 = lo_min / kDaTile, steps = (hi_max + kDaTile - 1) / kDaTile - tile0;
  const float scale_log2 = p.scale * 1.4426950408889634f;

  uint8_t* q_s = base;
  uint8_t* p_s = q_s + kTileK;
  uint8_t* k_s = p_s + 2 * kDaHalf;                        // two stages
  uint8_t* v_s = k_s + 2 * kTileK;
  TpSmem* sm = reinterpret_cast<TpSmem*>(v_s + kTileV);
  volatile int* abort_flag = &sm->abort_flag;
  const int kv0 = p.kv_start[b] + tile0 * kDaTile;

  int k_issued = 0, v_issued = 0;
  auto load_k = [&](int s) {
    const int st = s & 1;
    mbar_expect_tx(&sm->bar_k[st], kTileK);
#pragma unroll
    for (int hh = 0; hh < K1; ++hh) tma_load_3d(k_s + st * kTileK + hh * kDaHalf, &map_k1, &sm->bar_k[st], hh * 64, head, kv0 + s * kDaTile);
#pragma unroll
    for (int hh = 0; hh < K2; ++hh) tma_load_3d(k_s + st * kTileK + (K1 + hh) * kDaHalf, &map_k2, &sm->bar_k[st], hh * 64, 0, kv0 + s * kDaTile);
    ++k_issued;
  };
  auto load_v = [&](int s) {
    mbar_expect_tx(&sm->bar_v, kTileV);
#pragma unroll
    for (int hh = 0; hh < VH; ++hh) tma_load_3d(v_s + hh * kDaHalf, &map_v, &sm->bar_v, hh * 64, head, kv0 + s * kDaTile);
    ++v_issued;
  };
  if (tid == kDaSoftmaxThreads) {
    for (int i = 0; i < 2; ++i) { mbar_init(&sm->bar_k[i], 1); mbar_init(&sm->bar_s[i], 1); }
    mbar_init(&sm->bar_v, 1);
    mbar_init(&sm->bar_o, 1);
    mbar_init(&sm->bar_p, kDaSoftmaxThreads);
    mbar_init(&sm->bar_x, kDaSoftmaxThreads);
    sm->abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    load_k(0);                                             // steps >= 1
    if (steps > 1) load_k(1);
    load_v(0);
  }
  __syncwarp();
  if (is_ctrl) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kDaTmemCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  } else {
    const __nv_bfloat16* q1 = (const __nv_bfloat16*)p.q1 + (int64_t)(tok0 + token) * p.q1_token + (int64_t)head * p.q1_head;
    const __nv_bfloat16* q2 = (const __nv_bfloat16*)p.q2 + (int64_t)(tok0 + token) * p.q2_token + (int64_t)head * p.q2_head;
#pragma unroll
    for (int c = 0; c < KH * 4; ++c) {
      const int cc = half * (KH * 4) + c;
      const bool first = cc < K1 * 8;
      const int e = (first ? cc : cc - K1 * 8) * 8;
      const bool live = row_valid && e < (first ? p.d1 : p.d2);
      st16(q_s + da_swz(row, cc), live ? ld16((first ? q1 : q2) + e) : make_uint4(0, 0, 0, 0));
    }
  }
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;

  if (is_ctrl) {
    if (tid == kDaSoftmaxThreads) {
      const uint32_t idesc_s = da_idesc(128, 0), idesc_pv = da_idesc(VH * 64, 1);
      const uint32_t p_addr = smem_u32(p_s), q_addr = smem_u32(q_s), v_addr = smem_u32(v_s);
      auto issue_s = [&](int s) -> bool {
        if (!mbar_wait_or_abort(&sm->bar_k[s & 1], (s >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(k_s + (s & 1) * kTileK);
#pragma unroll
        for (int k = 0; k < KH * 4; ++k) {
          const uint32_t off = (k >> 2) * kDaHalf + (k & 3) * 32;
          umma(tmem + 128 * (s & 1), make_desc(q_addr + off, 16, 1024, 2), make_desc(k_addr + off, 16, 1024, 2), idesc_s, k > 0);
        }
        umma_commit(&sm->bar_s[s & 1]);
        return true;
      };
      bool ok = issue_s(0);
      for (int s = 0; s < steps && ok; ++s) {
        // the S buffer and the K stage of step s + 1 were last used by step s - 1, whose P has been waited for
        if (s + 1 < steps) ok = issue_s(s + 1);
        if (ok && s + 2 < steps) {                         // K two steps ahead goes where K of this step is
          ok = mbar_wait_or_abort(&sm->bar_s[s & 1], (s >> 1) & 1, abort_flag);
          if (ok) load_k(s + 2);
        }
        if (ok && s > 0) {                                 // V of this step goes where V of the last one was
          ok = mbar_wait_or_abort(&sm->bar_o, (s - 1) & 1, abort_flag);
          if (ok) load_v(s);
        }
        if (ok) ok = mbar_wait_or_abort(&sm->bar_p, s & 1, abort_flag);
        if (ok) ok = mbar_wait_or_abort(&sm->bar_v, s & 1, abort_flag);
        if (ok) {
          tc_fence_after();
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint64_t ad = make_desc(p_addr + (k >> 2) * kDaHalf + (k & 3) * 32, 16, 1024, 2);
            const uint64_t bd = make_desc(v_addr + k * 2048, kDaHalf, 1024, 2);
            umma(tmem + 256, ad, bd, idesc_pv, (s > 0 || k > 0));
          }
          umma_commit(&sm->bar_o);
        }
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
    }
    __syncwarp();
  } else {
    const uint32_t lane_base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    float m_ref = -INFINITY, l_sum = 0.f;
    bool alive = true;
    for (int s = 0; s < steps && alive; ++s) {
      const int t0 = (tile0 + s) * kDaTile;
      const int lo = lo_row - t0 - half * 64, hi = hi_row - t0 - half * 64;   // visible columns of this thread's half
      bool ok = mbar_wait_or_abort(&sm->bar_s[s & 1], (s >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) { alive = false; break; }
      tc_fence_after();
      const uint32_t s_addr = lane_base + 128 * (s & 1) + 64 * half;
      uint32_t sv[64];
      da_ld32_nowait(s_addr, sv);
      da_ld32_nowait(s_addr + 32, sv + 32);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      const bool full = lo <= 0 && hi >= 64;
      float m_part = -INFINITY;
      if (full) {
        float mr[4] = {__uint_as_float(sv[0]), __uint_as_float(sv[1]), __uint_as_float(sv[2]), __uint_as_float(sv[3])};
#pragma unroll
        for (int i = 4; i < 64; i += 4) {
          mr[0] = fmaxf(mr[0], __uint_as_float(sv[i])); mr[1] = fmaxf(mr[1], __uint_as_float(sv[i + 1]));
          mr[2] = fmaxf(mr[2], __uint_as_float(sv[i + 2])); mr[3] = fmaxf(mr[3], __uint_as_float(sv[i + 3]));
        }
        m_part = fmaxf(fmaxf(mr[0], mr[1]), fmaxf(mr[2], mr[3])) * scale_log2;
      } else {
#pragma unroll
        for (int i = 0; i < 64; ++i)
          if (i >= lo && i < hi) m_part = fmaxf(m_part, __uint_as_float(sv[i]) * scale_log2);
      }
      sm->red[s & 1][half][row] = m_part;
      da_arrive(&sm->bar_x);
      ok = mbar_wait_or_abort(&sm->bar_x, s & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) { alive = false; break; }
      const float m_tile = fmaxf(m_part, sm->red[s & 1][half ^ 1][row]);
      const bool grow = m_tile > m_ref + kDaRescaleGap || (m_ref == -INFINITY && m_tile > -INFINITY);
      const bool rescale = __any_sync(0xffffffffu, grow);
      if (s > 0) {                                         // P.V of the previous step: the P buffer is free, O is readable
        ok = mbar_wait_or_abort(&sm->bar_o, (s - 1) & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) { alive = false; break; }
        tc_fence_after();
      }
      if (rescale) {
        const float m_new = fmaxf(m_ref, m_tile);
        if (s > 0) {
          const float alpha = (m_ref == -INFINITY) ? 1.0f : exp2_weight(m_ref - m_new);
#pragma unroll
          for (int c2 = 0; c2 < OD / 32; ++c2) {
            float o[32];
            const uint32_t at = lane_base + 256 + OD * half + c2 * 32;
            tmem_ld32(at, o);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] *= alpha;
            da_st32(at, o);
          }
          l_sum *= alpha;
        }
        m_ref = m_new;
      }
      const float neg_m = m_ref == -INFINITY ? 0.f : -m_ref;   // a row that has seen no key yet: weights 0
      float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        uint32_t w[16];
        if (full) {
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float a = exp2_weight(fmaf(__uint_as_float(sv[c2 * 32 + i]), scale_log2, neg_m));
            const float bb = exp2_weight(fmaf(__uint_as_float(sv[c2 * 32 + i + 1]), scale_log2, neg_m));
            ls[(i >> 1) & 3] += a + bb;
            w[i >> 1] = da_pack2(a, bb);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const int col = c2 * 32 + i;
            const float a = (col >= lo && col < hi) ? exp2_weight(fmaf(__uint_as_float(sv[col]), scale_log2, neg_m)) : 0.f;
            const float bb = (col + 1 >= lo && col + 1 < hi) ? exp2_weight(fmaf(__uint_as_float(sv[col + 1]), scale_log2, neg_m)) : 0.f;
            ls[(i >> 1) & 3] += a + bb;
            w[i >> 1] = da_pack2(a, bb);
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c)
          st16(p_s + da_swz(row, half * 8 + c2 * 4 + c), make_uint4(w[4 * c], w[4 * c + 1], w[4 * c + 2], w[4 * c + 3]));
      }
      l_sum += (ls[0] + ls[1]) + (ls[2] + ls[3]);
      // Rows of the V tile beyond the request's own hold another request's values: weight zero, but 0 x NaN must not
      // poison the product.
      if (t0 + kDaTile > len) {
        ok = mbar_wait_or_abort(&sm->bar_v, s & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) { alive = false; break; }
        if (t0 + row >= len && half < VH) {
          uint8_t* vt = v_s + half * kDaHalf + row * 128;
#pragma unroll
          for (int c = 0; c < 8; ++c) st16(vt + c * 16, make_uint4(0, 0, 0, 0));
        }
      }
      fence_async_smem();
      tc_fence_before();
      da_arrive(&sm->bar_p);
    }
    // ---- epilogue: the sum of both halves of a row, O over it
    if (alive) {
      bool ok = mbar_wait_or_abort(&sm->bar_o, (steps - 1) & 1, abort_flag);
      alive = __all_sync(0xffffffffu, ok);
    }
    if (alive) {
      tc_fence_after();
      sm->red[0][half][row] = l_sum;
      da_arrive(&sm->bar_x);
      bool ok = mbar_wait_or_abort(&sm->bar_x, steps & 1, abort_flag);
      alive = __all_sync(0xffffffffu, ok);
    }
    if (alive) {
      const float l = l_sum + sm->red[0][half ^ 1][row];
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      __nv_bfloat16* dst = (__nv_bfloat16*)p.out + (int64_t)(tok0 + token) * p.out_token + (int64_t)head * p.out_head + half * OD;
      const int live = min(OD, p.vdim - half * OD);        // elements of this thread that exist
#pragma unroll
      for (int c2 = 0; c2 < OD / 32; ++c2) {
        float o[32];
        tmem_ld32(lane_base + 256 + OD * half + c2 * 32, o);
        if (row_valid)
#pragma unroll
          for (int i = 0; i < 32; i += 8)
            if (c2 * 32 + i < live)
              st16(dst + c2 * 32 + i, make_uint4(da_pack2(o[i] * inv, o[i + 1] * inv), da_pack2(o[i + 2] * inv, o[i + 3] * inv),
                                                 da_pack2(o[i + 4] * inv, o[i + 5] * inv), da_pack2(o[i + 6] * inv, o[i + 7] * inv)));
      }
    }
    if (!alive && (tid & 31) == 0 && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
  }
  tc_fence_before();
  __syncthreads();
  if (tid == kDaSoftmaxThreads && *abort_flag != 0) {
    for (int i = max(0, k_issued - 2); i < k_issued; ++i) mbar_wait(&sm->bar_k[i & 1], (i >> 1) & 1);
    for (int i = max(0, v_issued - 1); i < v_issued; ++i) mbar_wait(&sm->bar_v, i & 1);
  }
  __syncthreads();
  if (is_ctrl) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kDaTmemCols));
}

// Parts of whole 16-byte pieces: every row, head and part starts on a 16-byte boundary.
bool two_part_tc_shape(const TwoPartAttn& p, int dtype) {
  if (dtype != TKV_BF16 || p.ring_rows > 0 || p.scale <= 0.f) return false;
  if (p.d1 > 128 || p.d2 <= 0 || p.d2 > 64 || p.vdim > 128 || p.d1 % 8 || p.d2 % 8 || p.vdim % 8) return false;
  if (p.q1_token % 8 || p.q2_token % 8 || p.k1_row % 8 || p.k2_row % 8 || p.v_row % 8 || p.out_token % 8) return false;
  return aligned16(p.q1) && aligned16(p.q2) && aligned16(p.k1) && aligned16(p.k2) && aligned16(p.v) && aligned16(p.out);
}

template <int K1, int VH>
static int launch_tp(const CUtensorMap& m1, const CUtensorMap& m2, const CUtensorMap& mv, const TwoPartAttn& p, int64_t grid, int nblocks,
                     cudaStream_t st) {
  static bool configured = false;
  constexpr int kBytes = tp_smem_bytes<K1 + 1, VH>();
  static_assert(kBytes <= 232448, "shared memory of the kernel");
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(two_part_prefill_kernel<K1, 1, VH>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_prefill: %s", cudaGetErrorString(e));
    configured = true;
  }
  cudaError_t e = launch_pdl(two_part_prefill_kernel<K1, 1, VH>, dim3((unsigned)grid), dim3(kDaThreads), (size_t)kBytes, st, m1, m2, mv, p, nblocks);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_latent_prefill: %s", cudaGetErrorString(e));
  return check_launch("tkv_latent_prefill");
}

int launch_two_part_tc(const TwoPartAttn& p, int64_t kv_rows, int max_tokens, cudaStream_t st) {
  const int64_t nblocks = ((int64_t)max_tokens + kDaTile - 1) / kDaTile, grid = (int64_t)p.batch * p.heads * nblocks;
  if (grid > INT32_MAX || kv_rows + kDaTile > INT32_MAX)
    return fail(TKV_ERR_UNSUPPORTED, "tkv_latent_prefill: %lld query blocks, %lld key rows", (long long)grid, (long long)kv_rows);
  CUtensorMap m1, m2, mv;
  int rc = make_map_3d_bf16(&m1, p.k1, p.d1, p.heads, kv_rows, p.k1_row, 64, 128);
  if (rc == TKV_OK) rc = make_map_3d_bf16(&m2, p.k2, 64, 1, kv_rows, p.k2_row, 64, 128);
  if (rc == TKV_OK) rc = make_map_3d_bf16(&mv, p.v, p.vdim, p.heads, kv_rows, p.v_row, 64, 128);
  if (rc != TKV_OK) return rc;
  if (p.d1 <= 64) return p.vdim <= 64 ? launch_tp<1, 1>(m1, m2, mv, p, grid, (int)nblocks, st) : launch_tp<1, 2>(m1, m2, mv, p, grid, (int)nblocks, st);
  return p.vdim <= 64 ? launch_tp<2, 1>(m1, m2, mv, p, grid, (int)nblocks, st) : launch_tp<2, 2>(m1, m2, mv, p, grid, (int)nblocks, st);
}

}  // namespace tkv
