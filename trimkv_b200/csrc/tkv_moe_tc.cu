// Grouped product of a mixture of experts on tcgen05 + TMEM, for prompts and for decoding:
//   out[r, :] = act(a[src[r], :] . w[e]^T)   for the rows r of expert e.
//
// One persistent CTA per SM walks tiles of 128 rows x BN columns, expert by expert.  Per 64 columns of k the weight rows are one
// TMA box; the rows of A are TMA boxes of 32 where they are consecutive, and are gathered by four warps with cp.async where they
// are not (TMA's own gather moves four rows per instruction and was the limit).  Rows a tile does not have are not fetched, so
// few rows per expert cost little more than the weights.  A ring of stages feeds the MMAs; two TMEM accumulators let the
// epilogue of a tile (activation, rounding, stores) overlap the next tile.
// A weight tile that reaches beyond an expert's n rows holds rows of the next expert: those columns are not stored.
// Every wait is bounded; on expiry the CTA records TKV_DEV_TIMEOUT, drains its copies and frees its TMEM.
#include <cuda.h>
#include "tkv_moe.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kMgGather = 128, kMgLag = 2;                // gathering threads; stages they run ahead of what they hand over
constexpr int kMgThreads = 192;                           // warp 0: copies, warp 1: products, warps 2-5: epilogue (6-9: gathering)
constexpr int kMgM = 128, kMgK = 64, kMgBoxRows = 32;
constexpr int kMgABytes = kMgM * kMgK * 2;
template <int BN> struct MgRing {
  static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 6 : 8, kStageBytes = kMgABytes + BN * kMgK * 2;
};

struct MgSmem {
  uint64_t full[8], empty[8], acc_full[2], acc_empty[2];
  uint64_t full_a[8];                                     // gathered rows of a stage are there
  uint32_t tmem_base;
  int abort_flag;
};
template <int BN> constexpr int mg_smem_bytes(int experts) {
  return MgRing<BN>::kStages * MgRing<BN>::kStageBytes + (int)sizeof(MgSmem) + (2 * experts + 1) * 4;
}

// Walks this CTA's tiles in order; every role keeps its own.
struct MgTiles {
  const int32_t* off; const int32_t* tile_end;            // shared memory: [experts + 1], [experts]
  int experts, ncols, e, tile, step;
  int row0, rows, col;                                    // of the current tile
  __device__ __forceinline__ bool next() {
    tile += step;
    const int m = tile / ncols;
    while (e < experts && tile_end[e] <= m) ++e;
    if (e >= experts) return false;
    const int first = e > 0 ? tile_end[e - 1] : 0;
    row0 = off[e] + (m - first) * kMgM;
    rows = min(kMgM, off[e + 1] - row0);
    col = tile - m * ncols;
    return true;
  }
};

template <int BN, bool kGather>
__global__ void __launch_bounds__(kMgThreads + (kGather ? kMgGather : 0), 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, GroupedGemm p) {
  extern __shared__ __align__(1024) uint8_t base[];
  constexpr int S = MgRing<BN>::kStages, kStage = MgRing<BN>::kStageBytes;
  constexpr int kTmemCols = 2 * BN;
  MgSmem* sm = reinterpret_cast<MgSmem*>(base + S * kStage);
  int32_t* off = reinterpret_cast<int32_t*>(sm + 1);      // [experts + 1]
  int32_t* tile_end = off + p.experts + 1;                // [experts]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  volatile int* abort_flag = &sm->abort_flag;
  if (tid == 0) {
    for (int s = 0; s < S; ++s) { mbar_init(&sm->full[s], 1); mbar_init(&sm->empty[s], 1); mbar_init(&sm->full_a[s], kMgGather); }
    for (int s = 0; s < 2; ++s) { mbar_init(&sm->acc_full[s], 1); mbar_init(&sm->acc_empty[s], 4); }
    sm->abort_flag = (smem_u32(base) & 1023u) != 0;       // the swizzled tiles need the alignment; the launch gives it
    if (sm->abort_flag) report(p.status, TKV_DEV_TIMEOUT);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kTmemCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  grid_dependency_wait();
  grid_launch_dependents();
  for (int e = tid; e <= p.experts; e += blockDim.x) off[e] = p.offsets[e];
  __syncthreads();
  if (warp == 0) {                                        // running number of row tiles
    int sum = 0;
    for (int e0 = 0; e0 < p.experts; e0 += 32) {
      const int e = e0 + lane;
      int x = e < p.experts ? (off[e + 1] - off[e] + kMgM - 1) / kMgM : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x += y;
      }
      if (e < p.experts) tile_end[e] = sum + x;
      sum += __shfl_sync(0xffffffffu, x, 31);
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;
  const int ksteps = (p.k + kMgK - 1) / kMgK, ncols = (p.n + BN - 1) / BN;
  int mg_copies = 0;                                      // stages whose TMA copies thread 0 has started
  MgTiles t = {off, tile_end, p.experts, ncols, 0, (int)blockIdx.x - (int)gridDim.x, (int)gridDim.x, 0, 0, 0};

  if (warp == 0) {
    // ---- weights, and consecutive rows
    if (lane == 0) {
      int it = 0;
      bool ok = *abort_flag == 0;
      while (ok && t.next()) {
        const int boxes = kGather ? 0 : (t.rows + kMgBoxRows - 1) / kMgBoxRows;
        const uint32_t bytes = (uint32_t)boxes * kMgBoxRows * 128 + BN * kMgK * 2;
        const int wrow = t.e * p.n + t.col * BN;
        for (int k = 0; k < ksteps; ++k, ++it) {
          const int s = it % S;
          ok = mbar_wait_or_abort(&sm->empty[s], ((it / S) & 1) ^ 1, abort_flag);
          if (!ok) break;
          uint8_t* st = base + s * kStage;
          mbar_expect_tx(&sm->full[s], bytes);
          tma_load_2d(st + kMgABytes, &map_w, &sm->full[s], k * kMgK, wrow);
          for (int i = 0; i < boxes; ++i)
            tma_load_2d(st + i * kMgBoxRows * 128, &map_a, &sm->full[s], k * kMgK, t.row0 + i * kMgBoxRows);
        }
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
      mg_copies = it;
    }
    __syncwarp();
  } else if (kGather && warp >= kMgThreads / 32) {
    // ---- gathered rows: thread g fetches the 16-byte piece g % 8 of rows g / 8 + 16 i
    const int g = tid - kMgThreads, piece = g & 7, r0 = g >> 3;
    const uint32_t swz = (uint32_t)((piece ^ (r0 & 7)) << 4);        // rows 16 apart share it
    auto hand_over = [&](int i) {
      fence_async_smem();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&sm->full_a[i % S])) : "memory");
    };
    int it = 0;
    bool ok = *abort_flag == 0;
    while (ok && t.next()) {
      const __nv_bfloat16* row[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = r0 + 16 * i;
        row[i] = r < t.rows ? (const __nv_bfloat16*)p.a + (int64_t)p.src[t.row0 + r] * p.a_stride + piece * 8 : nullptr;
      }
      for (int k = 0; k < ksteps; ++k, ++it) {
        const int s = it % S;
        ok = mbar_wait_or_abort(&sm->empty[s], ((it / S) & 1) ^ 1, abort_flag);
        if (!ok) break;
        const uint32_t dst = smem_u32(base + s * kStage) + (uint32_t)r0 * 128 + swz;
        const int bytes = k * kMgK + piece * 8 < p.k ? 16 : 0;       // the rest of the last piece of k reads as zeros
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (row[i] != nullptr)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + i * 16 * 128), "l"(bytes ? row[i] + k * kMgK : row[i] - piece * 8), "r"(bytes) : "memory");
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (it >= kMgLag) {
          asm volatile("cp.async.wait_group %0;" ::"n"(kMgLag) : "memory");
          hand_over(it - kMgLag);
        }
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    for (int i = max(0, it - kMgLag); i < it; ++i) hand_over(i);
    if (!ok && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
  } else if (warp == 1) {
    // ---- products
    if (lane == 0) {
      const uint32_t idesc = make_idesc(1, 0, BN);
      int it = 0, n = 0;
      bool ok = *abort_flag == 0;
      while (ok && t.next()) {
        const int buf = n & 1;
        ok = mbar_wait_or_abort(&sm->acc_empty[buf], ((n >> 1) & 1) ^ 1, abort_flag);
        tc_fence_after();
        for (int k = 0; k < ksteps && ok; ++k, ++it) {
          const int s = it % S;
          ok = mbar_wait_or_abort(&sm->full[s], (it / S) & 1, abort_flag);
          if (ok && kGather) ok = mbar_wait_or_abort(&sm->full_a[s], (it / S) & 1, abort_flag);
          if (!ok) break;
          tc_fence_after();
          const uint32_t a = smem_u32(base + s * kStage), w = a + kMgABytes;
#pragma unroll
          for (int q = 0; q < 4; ++q)
            umma(tmem + buf * BN, make_desc(a + q * 32, 16, 1024, 2), make_desc(w + q * 32, 16, 1024, 2), idesc, (k > 0 || q > 0));
          umma_commit(&sm->empty[s]);
        }
        if (ok) umma_commit(&sm->acc_full[buf]);
        ++n;
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
    }
    __syncwarp();
  } else {
    // ---- epilogue: thread = row of the tile
    const int quarter = warp & 3, row = quarter * 32 + lane;
    int n = 0;
    bool ok = *abort_flag == 0;
    while (ok && t.next()) {
      const int buf = n & 1;
      ok = mbar_wait_or_abort(&sm->acc_full[buf], (n >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      __nv_bfloat16* dst = (__nv_bfloat16*)p.out + (int64_t)(t.row0 + row) * p.n + t.col * BN;
      const int cols = p.n - t.col * BN;                  // of this tile that exist (a multiple of 8)
      if (quarter * 32 < t.rows)                          // else: a warp without rows has nothing to read
        for (int c = 0; c < BN / 32 && c * 32 < cols; ++c) {
          float v[32];
          tmem_ld32(tmem + ((uint32_t)(quarter * 32) << 16) + buf * BN + c * 32, v);
          if (row < t.rows) {
            if (p.act == 1) {
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = gelu_erf(v[i]);
            }
#pragma unroll
            for (int i = 0; i < 32; i += 8)
              if (c * 32 + i < cols) store_vec<8>(dst + c * 32 + i, v + i);
          }
          __syncwarp();
        }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&sm->acc_empty[buf])) : "memory");
      ++n;
    }
    if (!ok && lane == 0 && *abort_flag == 0) { *abort_flag = 1; report(p.status, TKV_DEV_TIMEOUT); }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (tid == 0 && *abort_flag != 0)                       // copies in flight land before the shared memory is released
    for (int i = max(0, mg_copies - S); i < mg_copies; ++i) mbar_wait(&sm->full[i % S], (i / S) & 1);
  if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemCols));
}

bool moe_tc_shape(const GroupedGemm& p, int dtype) {
  return dtype == TKV_BF16 && p.n % 8 == 0 && p.k % 8 == 0 && p.a_stride % 8 == 0 && aligned16(p.a) && aligned16(p.w) && aligned16(p.out) &&
         p.experts <= 1024 && (int64_t)p.experts * p.n + 256 <= INT32_MAX && p.a_rows > 0;
}

template <int BN, bool kGather>
static int launch_mg(const GroupedGemm& p, int64_t tiles, cudaStream_t st) {
  CUtensorMap ma, mw;
  int rc = make_map_rows(&ma, p.a, p.k, p.a_rows, p.a_stride, kMgK, kMgBoxRows);
  if (rc == TKV_OK) rc = make_map_2d(&mw, p.w, p.k, (int64_t)p.experts * p.n, kMgK, BN, TKV_BF16);
  if (rc != TKV_OK) return rc;
  const int bytes = mg_smem_bytes<BN>(p.experts);
  static int allowed = 0;
  if (bytes > allowed) {
    if (bytes > 232448) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_gemm: experts=%d", p.experts);
    cudaError_t e = cudaFuncSetAttribute(moe_tc_kernel<BN, kGather>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_moe_gemm: %s", cudaGetErrorString(e));
    allowed = bytes;
  }
  cudaError_t e = launch_pdl(moe_tc_kernel<BN, kGather>, dim3((unsigned)(tiles < 148 ? tiles : 148)), dim3(kMgThreads + (kGather ? kMgGather : 0)),
                             (size_t)bytes, st, ma, mw, p);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_moe_gemm: %s", cudaGetErrorString(e));
  return check_launch("tkv_moe_gemm");
}
template <int BN>
static int launch_mg(const GroupedGemm& p, int64_t tiles, cudaStream_t st) {
  return p.src != nullptr ? launch_mg<BN, true>(p, tiles, st) : launch_mg<BN, false>(p, tiles, st);
}

int launch_moe_tc(const GroupedGemm& p, cudaStream_t st) {
  // the widest column tile that still gives every SM a few tiles (row tiles: about one per expert beyond whole ones)
  const int64_t row_tiles = p.max_rows / kMgM + (p.experts < p.max_rows ? p.experts : p.max_rows);
  auto tiles = [&](int bn) { return row_tiles * ((p.n + bn - 1) / bn); };
  if (tiles(256) > INT32_MAX / 2) return fail(TKV_ERR_UNSUPPORTED, "tkv_moe_gemm: %lld tiles", (long long)tiles(256));
  if (tiles(256) >= 148 * 6) return launch_mg<256>(p, tiles(256), st);
  if (tiles(128) >= 148 * 2) return launch_mg<128>(p, tiles(128), st);
  return launch_mg<64>(p, tiles(64), st);
}

}  // namespace tkv
