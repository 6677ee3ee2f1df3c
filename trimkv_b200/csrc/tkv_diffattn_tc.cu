// Windowed differential attention over many query tokens (prompts and portions of prompts) on tcgen05 + TMEM.
//
// The schedule is that of the query-resident kernel (tkv_attn_prefill.cu) walked twice per tile: step 2j + m is map m of
// key tile j.  One CTA = (request, kv head, block of 128 query rows), row = token * heads_per_kv + head:
//   S[128 x 128]   = Q_m . K_m(tile)^T     two TMEM buffers (columns 0, 128), one per map
//   online softmax per map (two threads per row), P in the 16-bit type through shared memory
//   O_m[128 x pp] += P . V(tile)           TMEM columns 256 + 128 m; the V tile is loaded once for both maps
// and the epilogue combines the maps, norms the head and applies the gate in fp32 registers: nothing of a map's output
// goes to memory.  A row sees the columns [lo, hi) of the request's linear keys; tiles before the first row's window are
// never loaded.  Waits are bounded; on expiry the CTA records TKV_DEV_TIMEOUT, drains its copies and frees its TMEM.
#include <cuda.h>
#include "tkv_attn_block.cuh"
#include "tkv_diffattn.cuh"

namespace tkv {

struct DaSmem {
  uint64_t bar_k[2], bar_v[2], bar_s[2], bar_o, bar_p, bar_x;
  uint32_t tmem_base;
  int abort_flag;
  float red[2][2][kDaTile];
};
template <int KH, int VH> constexpr int da_smem_bytes() { return (4 * KH + 2 * VH + 2) * kDaHalf + (int)sizeof(DaSmem); }

// KH = dp / 64, VH = pp / 64.  Warps 0-7: softmax (row r is shared by threads r and 128 + r); warp 8 issues copies and MMAs.
template <int KH, int VH>
__global__ void __launch_bounds__(kDaThreads, 1)
diff_prefill_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, DiffAttnParams p, int nblocks) {
  extern __shared__ __align__(1024) uint8_t base[];
  constexpr int kTileK = KH * kDaHalf, kTileV = VH * kDaHalf;
  constexpr int DP = KH * 64, PP = VH * 64;
  constexpr int OD = PP / 2;                               // dims of O per thread: 32 or 64
  grid_dependency_wait();
  grid_launch_dependents();
  const int seg = (int)(blockIdx.x / (unsigned)nblocks);
  const int blk = nblocks - 1 - (int)(blockIdx.x % (unsigned)nblocks);
  const int tid = threadIdx.x, warp = tid >> 5;
  const bool is_ctrl = warp == 8;
  const int row = tid & (kDaTile - 1), half = (tid >> 7) & 1;
  const int hpg = p.heads / p.kv_heads;
  const int b = seg / p.kv_heads, g = seg - b * p.kv_heads;
  const int tok0 = p.cu[b], n = p.cu[b + 1] - tok0;
  const int rows = n * hpg;
  if (blk * kDaTile >= rows) return;
  if ((smem_u32(base) & 1023u) != 0) {                     // the swizzled tiles need it; the launch gives it
    if (tid == 0) report(p.status, TKV_DEV_TIMEOUT);
    return;
  }
  const int hist = min(p.pos0[b], p.window - 1);
  const int len = hist + n;                                // linear rows of the request
  const int R = blk * kDaTile + row;
  const bool row_valid = !is_ctrl && R < rows;
  const int token = row_valid ? R / hpg : 0, head = g * hpg + (row_valid ? R - token * hpg : 0);
  const int hi_row = row_valid ? hist + token + 1 : 0, lo_row = max(0, hi_row - p.window);
  const int hi_max = hist + (min(blk * kDaTile + kDaTile, rows) - 1) / hpg + 1;
  const int lo_min = max(0, hist + (blk * kDaTile) / hpg + 1 - p.window);
  const int tile0 = lo_min / kDaTile, ntiles = (hi_max + kDaTile - 1) / kDaTile - tile0, steps = 2 * ntiles;

  uint8_t* q_s = base;                                     // [map]
  uint8_t* p_s = q_s + 2 * kTileK;
  uint8_t* k_s = p_s + 2 * kDaHalf;                        // [map]
  uint8_t* v_s = k_s + 2 * kTileK;                         // two stages
  DaSmem* sm = reinterpret_cast<DaSmem*>(v_s + 2 * kTileV);
  volatile int* abort_flag = &sm->abort_flag;
  const int kv0 = p.kv_start[b] + tile0 * kDaTile;

  int k_issued = 0, v_issued = 0;
  auto load_k = [&](int s) {                               // keys of step s (tile s / 2, map s & 1)
    const int st = s & 1;
    mbar_expect_tx(&sm->bar_k[st], kTileK);
#pragma unroll
    for (int hh = 0; hh < KH; ++hh)
      tma_load_2d(k_s + st * kTileK + hh * kDaHalf, &map_k, &sm->bar_k[st], (g * 2 + st) * DP + hh * 64, kv0 + (s >> 1) * kDaTile);
    ++k_issued;
  };
  auto load_v = [&](int j) {
    const int st = j & 1;
    mbar_expect_tx(&sm->bar_v[st], kTileV);
#pragma unroll
    for (int hh = 0; hh < VH; ++hh)
      tma_load_2d(v_s + st * kTileV + hh * kDaHalf, &map_v, &sm->bar_v[st], g * PP + hh * 64, kv0 + j * kDaTile);
    ++v_issued;
  };
  if (tid == kDaSoftmaxThreads) {
    for (int i = 0; i < 2; ++i) { mbar_init(&sm->bar_k[i], 1); mbar_init(&sm->bar_v[i], 1); mbar_init(&sm->bar_s[i], 1); }
    mbar_init(&sm->bar_o, 1);
    mbar_init(&sm->bar_p, kDaSoftmaxThreads);
    mbar_init(&sm->bar_x, kDaSoftmaxThreads);
    sm->abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    load_k(0); load_k(1);                                  // ntiles >= 1: both maps of the first tile
    load_v(0);
  }
  __syncwarp();
  if (is_ctrl) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kDaTmemCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  } else {
    const __nv_bfloat16* qp = (const __nv_bfloat16*)p.q + ((int64_t)(tok0 + token) * p.heads + head) * 2 * DP;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int c = 0; c < DP / 16; ++c) {
        const int cc = half * (DP / 16) + c;
        st16(q_s + m * kTileK + da_swz(row, cc), row_valid ? ld16(qp + m * DP + cc * 8) : make_uint4(0, 0, 0, 0));
      }
  }
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;

  if (is_ctrl) {
    if (tid == kDaSoftmaxThreads) {
      const uint32_t idesc_s = da_idesc(128, 0), idesc_pv = da_idesc(PP, 1);
      const uint32_t p_addr = smem_u32(p_s);
      auto issue_s = [&](int s) -> bool {
        if (!mbar_wait_or_abort(&sm->bar_k[s & 1], (s >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t q_addr = smem_u32(q_s + (s & 1) * kTileK), k_addr = smem_u32(k_s + (s & 1) * kTileK);
#pragma unroll
        for (int k = 0; k < DP / 16; ++k) {
          const uint32_t off = (k >> 2) * kDaHalf + (k & 3) * 32;
          umma(tmem + 128 * (s & 1), make_desc(q_addr + off, 16, 1024, 2), make_desc(k_addr + off, 16, 1024, 2), idesc_s, k > 0);
        }
        umma_commit(&sm->bar_s[s & 1]);
        return true;
      };
      bool ok = issue_s(0);
      for (int s = 0; s < steps && ok; ++s) {
        const int j = s >> 1;
        // the S buffer and the K stage of step s + 1 were last used by step s - 1, whose P has been waited for
        if (s + 1 < steps) ok = issue_s(s + 1);
        // V of the next tile goes where V of tile j - 1 was: free once both P.V of that tile have completed
        if (ok && (s & 1) == 0 && j + 1 < ntiles) {
          if (s > 0) ok = mbar_wait_or_abort(&sm->bar_o, (s - 1) & 1, abort_flag);
          if (ok) load_v(j + 1);
        }
        if (ok && s + 2 < steps) {                         // K two steps ahead goes where K of this step is
          ok = mbar_wait_or_abort(&sm->bar_s[s & 1], (s >> 1) & 1, abort_flag);
          if (ok) load_k(s + 2);
        }
        if (ok) ok = mbar_wait_or_abort(&sm->bar_p, s & 1, abort_flag);
        if (ok) ok = mbar_wait_or_abort(&sm->bar_v[j & 1], (j >> 1) & 1, abort_flag);
        if (ok) {
          tc_fence_after();
          const uint32_t v_addr = smem_u32(v_s + (j & 1) * kTileV);
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const uint64_t ad = make_desc(p_addr + (k >> 2) * kDaHalf + (k & 3) * 32, 16, 1024, 2);
            const uint64_t bd = make_desc(v_addr + k * 2048, kDaHalf, 1024, 2);
            umma(tmem + 256 + 128 * (s & 1), ad, bd, idesc_pv, (s > 1 || k > 0));
          }
          umma_commit(&sm->bar_o);
        }
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
    }
    __syncwarp();
  } else {
    const uint32_t lane_base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    float m_ref[2] = {-INFINITY, -INFINITY}, l_sum[2] = {0.f, 0.f};
    bool alive = true;
    for (int j = 0; j < ntiles && alive; ++j) {
      const int t0 = (tile0 + j) * kDaTile;
      const int lo = lo_row - t0 - half * 64, hi = hi_row - t0 - half * 64;   // visible columns of this thread's half
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (!alive) break;
        const int s = 2 * j + m;
        bool ok = mbar_wait_or_abort(&sm->bar_s[m], j & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) { alive = false; break; }
        tc_fence_after();
        const uint32_t s_addr = lane_base + 128 * m + 64 * half;
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
          m_part = fmaxf(fmaxf(mr[0], mr[1]), fmaxf(mr[2], mr[3])) * p.scale_log2;
        } else {
#pragma unroll
          for (int i = 0; i < 64; ++i)
            if (i >= lo && i < hi) m_part = fmaxf(m_part, __uint_as_float(sv[i]) * p.scale_log2);
        }
        sm->red[m][half][row] = m_part;
        da_arrive(&sm->bar_x);
        ok = mbar_wait_or_abort(&sm->bar_x, s & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) { alive = false; break; }
        const float m_tile = fmaxf(m_part, sm->red[m][half ^ 1][row]);
        const bool grow = m_tile > m_ref[m] + kDaRescaleGap || (m_ref[m] == -INFINITY && m_tile > -INFINITY);
        const bool rescale = __any_sync(0xffffffffu, grow);
        if (s > 0) {                                       // P.V of the previous step: the P buffer is free, O is readable
          ok = mbar_wait_or_abort(&sm->bar_o, (s - 1) & 1, abort_flag);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) { alive = false; break; }
          tc_fence_after();
        }
        if (rescale) {
          const float m_new = fmaxf(m_ref[m], m_tile);
          if (j > 0) {
            const float alpha = (m_ref[m] == -INFINITY) ? 1.0f : exp2_weight(m_ref[m] - m_new);
#pragma unroll
            for (int c2 = 0; c2 < OD / 32; ++c2) {
              float o[32];
              const uint32_t at = lane_base + 256 + 128 * m + OD * half + c2 * 32;
              tmem_ld32(at, o);
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] *= alpha;
              da_st32(at, o);
            }
            l_sum[m] *= alpha;
          }
          m_ref[m] = m_new;
        }
        const float neg_m = -m_ref[m];
        float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int c2 = 0; c2 < 2; ++c2) {
          uint32_t w[16];
          if (full) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const float a = exp2_weight(fmaf(__uint_as_float(sv[c2 * 32 + i]), p.scale_log2, neg_m));
              const float bb = exp2_weight(fmaf(__uint_as_float(sv[c2 * 32 + i + 1]), p.scale_log2, neg_m));
              ls[(i >> 1) & 3] += a + bb;
              w[i >> 1] = da_pack2(a, bb);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const int col = c2 * 32 + i;
              const float a = (col >= lo && col < hi) ? exp2_weight(fmaf(__uint_as_float(sv[col]), p.scale_log2, neg_m)) : 0.f;
              const float bb = (col + 1 >= lo && col + 1 < hi) ? exp2_weight(fmaf(__uint_as_float(sv[col + 1]), p.scale_log2, neg_m)) : 0.f;
              ls[(i >> 1) & 3] += a + bb;
              w[i >> 1] = da_pack2(a, bb);
            }
          }
#pragma unroll
          for (int c = 0; c < 4; ++c)
            st16(p_s + da_swz(row, half * 8 + c2 * 4 + c), make_uint4(w[4 * c], w[4 * c + 1], w[4 * c + 2], w[4 * c + 3]));
        }
        l_sum[m] += (ls[0] + ls[1]) + (ls[2] + ls[3]);
        // Rows of the V tile beyond the request's own hold another request's values: weight zero, but 0 x NaN must not
        // poison the product.
        if (m == 0 && t0 + kDaTile > len) {
          ok = mbar_wait_or_abort(&sm->bar_v[j & 1], (j >> 1) & 1, abort_flag);
          ok = __all_sync(0xffffffffu, ok);
          if (!ok) { alive = false; break; }
          if (t0 + row >= len && half < VH) {
            uint8_t* vt = v_s + (j & 1) * kTileV + half * kDaHalf + row * 128;
#pragma unroll
            for (int c = 0; c < 8; ++c) st16(vt + c * 16, make_uint4(0, 0, 0, 0));
          }
        }
        fence_async_smem();
        tc_fence_before();
        da_arrive(&sm->bar_p);
      }
    }
    // ---- epilogue: both maps / their sums, combination, norm over the head (two threads per row), gate
    auto meet = [&](int phase) {
      da_arrive(&sm->bar_x);
      const bool ok = mbar_wait_or_abort(&sm->bar_x, phase & 1, abort_flag);
      return (bool)__all_sync(0xffffffffu, ok);
    };
    if (alive) {
      bool ok = mbar_wait_or_abort(&sm->bar_o, (steps - 1) & 1, abort_flag);
      alive = __all_sync(0xffffffffu, ok);
    }
    if (alive) {
      tc_fence_after();
      sm->red[0][half][row] = l_sum[0];
      sm->red[1][half][row] = l_sum[1];
      alive = meet(steps);
    }
    if (alive) {
      const float l0 = l_sum[0] + sm->red[0][half ^ 1][row], l1 = l_sum[1] + sm->red[1][half ^ 1][row];
      const float i0 = l0 > 0.f ? 1.0f / l0 : 0.f, i1 = l1 > 0.f ? *p.lambda / l1 : 0.f;
      float o[OD], ss = 0.f;
#pragma unroll
      for (int c2 = 0; c2 < OD / 32; ++c2) {
        float x[32];
        tmem_ld32(lane_base + 256 + OD * half + c2 * 32, o + c2 * 32);
        tmem_ld32(lane_base + 384 + OD * half + c2 * 32, x);
#pragma unroll
        for (int i = 0; i < 32; ++i) {                     // padded dims are zero in both maps
          o[c2 * 32 + i] = o[c2 * 32 + i] * i0 - x[i] * i1;
          ss += o[c2 * 32 + i] * o[c2 * 32 + i];
        }
      }
      float* xch = reinterpret_cast<float*>(q_s);          // every product that read Q has completed
      xch[half * kDaTile + row] = ss;
      alive = meet(steps + 1);
      if (alive && row_valid) {
        const float rr = 1.0f / sqrtf((ss + xch[(half ^ 1) * kDaTile + row]) / (float)p.vdim + p.eps);
        const float gate = rr * (1.0f - p.diff) *
                           sigmoid_f32(__bfloat162float(((const __nv_bfloat16*)p.gate)[(int64_t)(tok0 + token) * p.gate_stride + head]));
        __nv_bfloat16* dst = (__nv_bfloat16*)p.out + ((int64_t)(tok0 + token) * p.heads + head) * p.vdim + half * OD;
        const int live = min(OD, p.vdim - half * OD);      // dims of this thread that exist
        if (p.vdim % 8 == 0) {
#pragma unroll
          for (int i = 0; i < OD; i += 8)
            if (i < live)
              st16(dst + i, make_uint4(da_pack2(o[i] * gate, o[i + 1] * gate), da_pack2(o[i + 2] * gate, o[i + 3] * gate),
                                       da_pack2(o[i + 4] * gate, o[i + 5] * gate), da_pack2(o[i + 6] * gate, o[i + 7] * gate)));
        } else {
#pragma unroll
          for (int i = 0; i < OD; ++i)
            if (i < live) dst[i] = __float2bfloat16_rn(o[i] * gate);
        }
      }
    }
    if (!alive && (tid & 31) == 0 && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
  }
  tc_fence_before();
  __syncthreads();
  if (tid == kDaSoftmaxThreads && *abort_flag != 0) {
    for (int i = max(0, k_issued - 2); i < k_issued; ++i) mbar_wait(&sm->bar_k[i & 1], (i >> 1) & 1);
    for (int i = max(0, v_issued - 2); i < v_issued; ++i) mbar_wait(&sm->bar_v[i & 1], (i >> 1) & 1);
  }
  __syncthreads();
  if (is_ctrl) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kDaTmemCols));
}

template <int KH, int VH>
static int launch_da(const CUtensorMap& mk, const CUtensorMap& mv, const DiffAttnParams& p, int64_t grid, int nblocks, cudaStream_t st) {
  static bool configured = false;
  constexpr int kBytes = da_smem_bytes<KH, VH>();
  static_assert(kBytes <= 232448, "shared memory of the kernel");
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(diff_prefill_kernel<KH, VH>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_diff_prefill: %s", cudaGetErrorString(e));
    configured = true;
  }
  cudaError_t e = launch_pdl(diff_prefill_kernel<KH, VH>, dim3((unsigned)grid), dim3(kDaThreads), (size_t)kBytes, st, mk, mv, p, nblocks);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_diff_prefill: %s", cudaGetErrorString(e));
  return check_launch("tkv_diff_prefill");
}

int launch_diff_prefill_tc(const DiffAttnParams& p, int64_t kv_rows, int max_tokens, cudaStream_t st) {
  const int64_t rows = (int64_t)max_tokens * (p.heads / p.kv_heads), nblocks = (rows + kDaTile - 1) / kDaTile;
  const int64_t grid = (int64_t)p.batch * p.kv_heads * nblocks;
  if (grid > INT32_MAX || rows > INT32_MAX - kDaTile || kv_rows + kDaTile > INT32_MAX)
    return fail(TKV_ERR_UNSUPPORTED, "tkv_diff_prefill: %lld query blocks, %lld key rows", (long long)grid, (long long)kv_rows);
  if (!aligned16(p.q) || !aligned16(p.k_lin) || !aligned16(p.v_lin) || !aligned16(p.out))
    return fail(TKV_ERR_ARG, "tkv_diff_prefill: pointers must be 16-byte aligned");
  CUtensorMap mk, mv;
  int rc = make_map_2d(&mk, p.k_lin, (int64_t)p.kv_heads * 2 * p.dp, kv_rows, 64, 128, TKV_BF16);
  if (rc != TKV_OK) return rc;
  rc = make_map_2d(&mv, p.v_lin, (int64_t)p.kv_heads * p.pp, kv_rows, 64, 128, TKV_BF16);
  if (rc != TKV_OK) return rc;
  if (p.dp == 64) return p.pp == 64 ? launch_da<1, 1>(mk, mv, p, grid, (int)nblocks, st) : launch_da<1, 2>(mk, mv, p, grid, (int)nblocks, st);
  return p.pp == 64 ? launch_da<2, 1>(mk, mv, p, grid, (int)nblocks, st) : launch_da<2, 2>(mk, mv, p, grid, (int)nblocks, st);
}

}  // namespace tkv
