// Chunked scalar-decay linear recurrence on tcgen05 + TMEM (the mathematics: tkv_linrec_chunk.cu), for state rows n up to
// 128 (padded to the MMA's 128), 64 value columns per CTA, chunks of 128 tokens.
//
// One CTA walks the chunks of one (request, head, 64 columns of v, segment).  Per chunk, D in TMEM:
//   S  [128 tok x 128 tok] = Q . K^T                     A = Q, B = K as TMA wrote them (K-major)
//   O1 [128 tok x 2 x 64]  = Q . [S_prev high | low]     B = the state before the chunk as two bf16 parts (MN-major)
//   O2 [128 tok x 64]      = P . V                       A = P, the weighted scores, high and low part; B = V (MN-major)
//   ST [128 n x 2 x 64]    = e^{L_end} ST + K^T . [w V high | low]   A = K read MN-major, B = weighted values as two parts
// A product with few columns costs what reading its 128 rows costs, so the two parts of a B operand go side by side into one
// product of 128 columns and are added when they are read.  The state stays in TMEM as the accumulator of its own update; once per chunk its rows pass through registers to be scaled
// and to be written as the operand of O1.  fp32 factors of a product enter as two bf16 parts, so nothing that recurs is
// rounded to 16 bits.
//
// Roles: warps 0-7 hold rows (TMEM lane = token, or state row; two threads per row, one per column half); warp 8 issues TMA
// copies and MMAs (one lane); warp 9 computes the running log decays of the next chunk.  Q and K are refetched as soon as
// the products that read them have completed, under the weighting of the scores; V has two stages.  Every wait is bounded;
// on expiry the CTA records TKV_DEV_TIMEOUT, drains its copies, frees its TMEM and returns.
#include <cuda.h>
#include "tkv_linrec.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kLtC = 128, kLtP = 64;                       // tokens per chunk, value columns per CTA
constexpr int kLtRows = 256, kLtThreads = kLtRows + 64;
constexpr int kLtHalf = 16384;                             // 128 rows x 64 bf16
constexpr int kLtS = 0, kLtO1 = 128, kLtO2 = 256, kLtST = 320, kLtCols = 512;   // O1, ST: high | low

struct LtSmem {
  float2 lv[2][kLtC];                                      // running log2 decay and value scale; by chunk parity
  uint64_t bar_qk, bar_v[2], bar_l[2], bar_s, bar_sp, bar_o1, bar_wv, bar_st, bar_p, bar_o2, bar_clr;
  uint32_t tmem_base;
  int abort_flag;
};
constexpr int kLtSmemBytes = 14 * kLtHalf + (int)sizeof(LtSmem);
static_assert(kLtSmemBytes <= 232448, "shared memory of the kernel");

__device__ __forceinline__ uint32_t lt_idesc(int n, int a_mn, int b_mn) {   // bf16 operands, fp32 D, M = 128
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)b_mn << 16) | ((uint32_t)(n >> 3) << 17) | ((128u >> 4) << 24);
}
__device__ __forceinline__ uint32_t lt_swz(int r, int c) {  // 16-byte chunk c (0..7) of row r of a 64-column tile
  return (uint32_t)(r * 128 + ((c ^ (r & 7)) << 4));
}
__device__ __forceinline__ void lt_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void lt_ld32_nowait(uint32_t taddr, uint32_t* r) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
      "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
__device__ __forceinline__ void lt_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void lt_st32(uint32_t taddr, const float* v) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
      "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
      ::"r"(taddr), "r"(__float_as_uint(v[0])), "r"(__float_as_uint(v[1])), "r"(__float_as_uint(v[2])),
        "r"(__float_as_uint(v[3])), "r"(__float_as_uint(v[4])), "r"(__float_as_uint(v[5])), "r"(__float_as_uint(v[6])),
        "r"(__float_as_uint(v[7])), "r"(__float_as_uint(v[8])), "r"(__float_as_uint(v[9])), "r"(__float_as_uint(v[10])),
        "r"(__float_as_uint(v[11])), "r"(__float_as_uint(v[12])), "r"(__float_as_uint(v[13])), "r"(__float_as_uint(v[14])),
        "r"(__float_as_uint(v[15])), "r"(__float_as_uint(v[16])), "r"(__float_as_uint(v[17])), "r"(__float_as_uint(v[18])),
        "r"(__float_as_uint(v[19])), "r"(__float_as_uint(v[20])), "r"(__float_as_uint(v[21])), "r"(__float_as_uint(v[22])),
        "r"(__float_as_uint(v[23])), "r"(__float_as_uint(v[24])), "r"(__float_as_uint(v[25])), "r"(__float_as_uint(v[26])),
        "r"(__float_as_uint(v[27])), "r"(__float_as_uint(v[28])), "r"(__float_as_uint(v[29])), "r"(__float_as_uint(v[30])),
        "r"(__float_as_uint(v[31]))
      : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}
// x = hi + lo in bf16, two values at a time.
__device__ __forceinline__ void lt_split(float a, float b, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(*hi << 16), b - __uint_as_float(*hi & 0xffff0000u));
  *lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <bool kStateOnly>
__global__ void __launch_bounds__(kLtThreads, 1)
linrec_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                 LinrecParams a, LinrecSegs sg, int32_t* status) {
  extern __shared__ __align__(1024) uint8_t base[];
  grid_dependency_wait();
  grid_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ptiles = (a.p + kLtP - 1) / kLtP, per_seg = a.batch * a.heads * ptiles;
  const int seg = blockIdx.x / per_seg, item = blockIdx.x - seg * per_seg;
  const int pt = item % ptiles, bh = item / ptiles, b = bh / a.heads, h = bh - b * a.heads, g = h / (a.heads / a.groups);
  const int tok0 = a.cu[b], ntok = a.cu[b + 1] - tok0;
  const int t_first = seg * sg.tokens, t_end = min(ntok, t_first + sg.tokens);
  if (t_first >= t_end) return;
  if (kStateOnly && t_end == ntok) return;                 // nobody starts from the end of the last segment
  if ((smem_u32(base) & 1023u) != 0) {                     // the swizzled tiles need it; the launch gives it
    if (tid == 0) report(status, TKV_DEV_TIMEOUT);
    return;
  }
  const int nchunks = (t_end - t_first + kLtC - 1) / kLtC;
  const int last_rows = t_end - t_first - (nchunks - 1) * kLtC;    // live tokens of the last chunk
  const int pbase = pt * kLtP;

  uint8_t* q_s = base;                                     // two 64-column halves
  uint8_t* k_s = q_s + 2 * kLtHalf;
  uint8_t* v_s = k_s + 2 * kLtHalf;                        // two stages
  uint8_t* wv_s = v_s + 2 * kLtHalf;                       // high, low
  uint8_t* sp_s = wv_s + 2 * kLtHalf;                      // high, low
  uint8_t* p_s = sp_s + 2 * kLtHalf;                       // high (two halves), low (two halves)
  LtSmem* sm = reinterpret_cast<LtSmem*>(p_s + 4 * kLtHalf);
  volatile int* abort_flag = &sm->abort_flag;

  int qk_issued = 0, v_issued = 0;
  auto load_qk = [&](int i) {
    mbar_expect_tx(&sm->bar_qk, (kStateOnly ? 2 : 4) * kLtHalf);
    const int row = tok0 + t_first + i * kLtC;
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      if (!kStateOnly) tma_load_3d(q_s + hh * kLtHalf, &map_q, &sm->bar_qk, hh * 64, g, row);
      tma_load_3d(k_s + hh * kLtHalf, &map_k, &sm->bar_qk, hh * 64, g, row);
    }
    ++qk_issued;
  };
  auto load_v = [&](int i) {
    mbar_expect_tx(&sm->bar_v[i & 1], kLtHalf);
    tma_load_3d(v_s + (i & 1) * kLtHalf, &map_v, &sm->bar_v[i & 1], pbase, h, tok0 + t_first + i * kLtC);
    ++v_issued;
  };
  if (tid == kLtRows) {
    mbar_init(&sm->bar_qk, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&sm->bar_v[i], 1); mbar_init(&sm->bar_l[i], 32); }
    mbar_init(&sm->bar_s, 1); mbar_init(&sm->bar_o1, 1); mbar_init(&sm->bar_st, 1); mbar_init(&sm->bar_o2, 1);
    mbar_init(&sm->bar_sp, kLtRows); mbar_init(&sm->bar_wv, kLtRows); mbar_init(&sm->bar_p, kLtRows); mbar_init(&sm->bar_clr, kLtRows);
    sm->abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    load_qk(0);
    load_v(0);
  }
  __syncwarp();
  if (warp == 8) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kLtCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;
  const int64_t np = (int64_t)a.n * a.p;
  float* const final_state = a.state + ((int64_t)a.slots[b] * a.heads + h) * np;

  if (warp == 8) {
    // ------------------------------------------------------------------------------------ TMA + MMA issue (one lane)
    if (lane == 0) {
      const uint32_t id_s = lt_idesc(128, 0, 0), id_o1 = lt_idesc(2 * kLtP, 0, 1), id_o2 = lt_idesc(kLtP, 0, 1), id_st = lt_idesc(2 * kLtP, 1, 1);
      const uint32_t qa = smem_u32(q_s), ka = smem_u32(k_s);
      // K-major operand: step k covers 16 columns; MN-major operand of 128 rows: step k covers 16 rows.
      auto kmaj = [&](uint32_t at, int k) { return make_desc(at + (k >> 2) * kLtHalf + (k & 3) * 32, 16, 1024, 2); };
      auto mnmaj = [&](uint32_t at, int k) { return make_desc(at + k * 2048, kLtHalf, 1024, 2); };
      bool ok = true;
      for (int i = 0; i < nchunks && ok; ++i) {
        const int ph = i & 1;
        ok = mbar_wait_or_abort(&sm->bar_qk, ph, abort_flag);
        if (ok && i == nchunks - 1 && last_rows < kLtC) ok = mbar_wait_or_abort(&sm->bar_clr, 0, abort_flag);
        if (!ok) break;
        tc_fence_after();
        if (!kStateOnly) {
#pragma unroll
          for (int k = 0; k < 8; ++k) umma(tmem + kLtS, kmaj(qa, k), kmaj(ka, k), id_s, k > 0);
          umma_commit(&sm->bar_s);
        }
        ok = mbar_wait_or_abort(&sm->bar_sp, ph, abort_flag);      // the state is scaled, its operand written, chunk i - 1 finished
        if (!ok) break;
        tc_fence_after();
        if (i + 1 < nchunks) load_v(i + 1);
        if (!kStateOnly) {
          const uint32_t sp = smem_u32(sp_s);
#pragma unroll
          for (int k = 0; k < 8; ++k) umma(tmem + kLtO1, kmaj(qa, k), mnmaj(sp, k), id_o1, k > 0);
          umma_commit(&sm->bar_o1);
        }
        ok = mbar_wait_or_abort(&sm->bar_wv, ph, abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint32_t wv = smem_u32(wv_s);
#pragma unroll
        for (int k = 0; k < 8; ++k) umma(tmem + kLtST, mnmaj(ka, k), mnmaj(wv, k), id_st, 1);
        umma_commit(&sm->bar_st);
        if (i + 1 < nchunks) {                             // Q and K are free once these products have completed
          ok = mbar_wait_or_abort(&sm->bar_st, ph, abort_flag);
          if (ok && !kStateOnly) ok = mbar_wait_or_abort(&sm->bar_o1, ph, abort_flag);
          if (ok) load_qk(i + 1);
        }
        if (!kStateOnly && ok) {
          ok = mbar_wait_or_abort(&sm->bar_p, ph, abort_flag);
          if (!ok) break;
          tc_fence_after();
          const uint32_t pa = smem_u32(p_s), va = smem_u32(v_s + (i & 1) * kLtHalf);   // V has arrived: wV was made of it
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int k = 0; k < 8; ++k) umma(tmem + kLtO2, kmaj(pa + part * 2 * kLtHalf, k), mnmaj(va, k), id_o2, part > 0 || k > 0);
          umma_commit(&sm->bar_o2);
        }
      }
      if (!ok && *abort_flag == 0) { *abort_flag = 1; report(status, TKV_DEV_TIMEOUT); }
    }
    __syncwarp();
  } else if (warp == 9) {
    // ------------------------------------------------------------------------------------ running log decays, 4 tokens a lane
    float d[4], s[4], seg_log = 0.f;
    auto fetch = [&](int i) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = t_first + i * kLtC + 4 * lane + e;
        const int64_t th = (int64_t)(tok0 + t) * a.heads + h;
        const bool live = t < t_end;
        d[e] = live ? (a.log_decay != nullptr ? a.log_decay[th] : a.head_log_decay[h]) : 0.f;
        s[e] = live ? (a.v_scale != nullptr ? a.v_scale[th] : 1.f) : 0.f;
      }
    };
    fetch(0);
    bool ok = true;
    for (int i = 0; i < nchunks && ok; ++i) {
      d[1] += d[0]; d[2] += d[1]; d[3] += d[2];
      float sum = d[3];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += y;
      }
      const float before = sum - d[3];
      if (i >= 1) {                                        // chunk i - 2, which used this buffer last, is finished
        ok = mbar_wait_or_abort(&sm->bar_sp, (i - 1) & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
      }
      constexpr float kLog2e = 1.4426950408889634f;
#pragma unroll
      for (int e = 0; e < 4; ++e) sm->lv[i & 1][4 * lane + e] = make_float2((before + d[e]) * kLog2e, s[e]);
      seg_log += __shfl_sync(0xffffffffu, sum, 31) * kLog2e;
      lt_arrive(&sm->bar_l[i & 1]);
      if (i + 1 < nchunks) fetch(i + 1);
    }
    if (!ok && lane == 0 && *abort_flag == 0) { *abort_flag = 1; report(status, TKV_DEV_TIMEOUT); }
    if (kStateOnly && ok && lane == 0 && pt == 0) sg.log_sum[(int64_t)bh * sg.count + seg] = seg_log;
  } else {
    // ------------------------------------------------------------------------------------ rows
    const int row = tid & 127, half = tid >> 7;
    const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t st_at = lanes + kLtST + half * 32;
    auto sync_on = [&](uint64_t* bar, int parity) {
      const bool ok = mbar_wait_or_abort(bar, parity & 1, abort_flag);
      return (bool)__all_sync(0xffffffffu, ok);
    };
    {                                                      // the state before the first chunk
      const float* S = kStateOnly ? nullptr : sg.count > 1 ? sg.start + ((int64_t)bh * sg.count + seg) * np : a.pos0[b] == 0 ? nullptr : final_state;
      float s[32];
#pragma unroll
      for (int c = 0; c < 32; c += 4) {
        const int p = pbase + half * 32 + c;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (S != nullptr && row < a.n && p < a.p) x = *reinterpret_cast<const float4*>(S + (int64_t)row * a.p + p);
        s[c] = x.x; s[c + 1] = x.y; s[c + 2] = x.z; s[c + 3] = x.w;
      }
      lt_st32(st_at, s);
#pragma unroll
      for (int c = 0; c < 32; ++c) s[c] = 0.f;
      lt_st32(st_at + kLtP, s);
    }
    const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
    bool alive = true;
    for (int i = 0; i < nchunks; ++i) {
      const int ph = i & 1;
      const float2* lv = sm->lv[ph];
      uint8_t* v_t = v_s + (i & 1) * kLtHalf;
      // ---- tokens beyond the request's end belong to another request: their keys and values read as zeros
      if (i == nchunks - 1 && last_rows < kLtC) {
        alive = sync_on(&sm->bar_qk, ph) && sync_on(&sm->bar_v[i & 1], i >> 1);
        if (!alive) break;
        if (row >= last_rows) {
#pragma unroll
          for (int c = 0; c < 8; ++c) st16(k_s + half * kLtHalf + row * 128 + c * 16, make_uint4(0, 0, 0, 0));
#pragma unroll
          for (int c = 0; c < 4; ++c) st16(v_t + row * 128 + half * 64 + c * 16, make_uint4(0, 0, 0, 0));
        }
        fence_async_smem();
        lt_arrive(&sm->bar_clr);
      }
      // ---- the state before this chunk: operand of the read-out, then scaled for its update
      alive = sync_on(&sm->bar_l[i & 1], i >> 1);
      if (alive && i > 0) alive = sync_on(&sm->bar_st, i - 1);
      if (!alive) break;
      tc_fence_after();
      const float lend = lv[kLtC - 1].x;
      {
        float s[32];
        {
          uint32_t x[32], y[32];
          lt_ld32_nowait(st_at, x);
          lt_ld32_nowait(st_at + kLtP, y);
          lt_wait_ld();
#pragma unroll
          for (int c = 0; c < 32; ++c) s[c] = __uint_as_float(x[c]) + __uint_as_float(y[c]);
        }
        if (!kStateOnly) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) lt_split(s[c * 8 + 2 * e], s[c * 8 + 2 * e + 1], &hi[e], &lo[e]);
            const uint32_t at = lt_swz(row, half * 4 + c);
            st16(sp_s + at, make_uint4(hi[0], hi[1], hi[2], hi[3]));
            st16(sp_s + kLtHalf + at, make_uint4(lo[0], lo[1], lo[2], lo[3]));
          }
        }
        const float ec = exp2_weight(lend);
#pragma unroll
        for (int c = 0; c < 32; ++c) s[c] *= ec;
        lt_st32(st_at, s);
#pragma unroll
        for (int c = 0; c < 32; ++c) s[c] = 0.f;
        lt_st32(st_at + kLtP, s);
      }
      fence_async_smem();
      tc_fence_before();
      lt_arrive(&sm->bar_sp);
      // ---- weighted values
      alive = sync_on(&sm->bar_v[i & 1], i >> 1);
      if (!alive) break;
      const float l_row = lv[row].x, w_row = exp2_weight(lend - l_row) * lv[row].y;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const uint32_t at = lt_swz(row, half * 4 + c);
        const uint4 x = ld16(v_t + at);
        const uint32_t xs[4] = {x.x, x.y, x.z, x.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) lt_split(__uint_as_float(xs[e] << 16) * w_row, __uint_as_float(xs[e] & 0xffff0000u) * w_row, &hi[e], &lo[e]);
        st16(wv_s + at, make_uint4(hi[0], hi[1], hi[2], hi[3]));
        st16(wv_s + kLtHalf + at, make_uint4(lo[0], lo[1], lo[2], lo[3]));
      }
      fence_async_smem();
      lt_arrive(&sm->bar_wv);
      if (kStateOnly) continue;
      // ---- weighted scores: this thread's 64 columns of its row
      alive = sync_on(&sm->bar_s, ph);
      if (!alive) break;
      tc_fence_after();
      const int j0 = half * 64, r0 = row & ~31;            // rows r0 .. r0 + 31 of this warp
      uint8_t* p_hi = p_s + half * kLtHalf;
      uint8_t* p_lo = p_hi + 2 * kLtHalf;
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        const int jb = j0 + c2 * 32;
        if (jb > r0 + 31) {                                // all of it in the future (warp-uniform)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const uint32_t at = lt_swz(row, c2 * 4 + c);
            st16(p_hi + at, make_uint4(0, 0, 0, 0));
            st16(p_lo + at, make_uint4(0, 0, 0, 0));
          }
          continue;
        }
        uint32_t sv[32];
        lt_ld32_nowait(lanes + kLtS + jb, sv);
        lt_wait_ld();
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int j = jb + c * 8 + 2 * e;
            const float4 w = *reinterpret_cast<const float4*>(&lv[j]);     // two tokens: log decay, scale
            const float x = j <= row ? __uint_as_float(sv[c * 8 + 2 * e]) * exp2_weight(l_row - w.x) * w.y : 0.f;
            const float y = j + 1 <= row ? __uint_as_float(sv[c * 8 + 2 * e + 1]) * exp2_weight(l_row - w.z) * w.w : 0.f;
            lt_split(x, y, &hi[e], &lo[e]);
          }
          const uint32_t at = lt_swz(row, c2 * 4 + c);
          st16(p_hi + at, make_uint4(hi[0], hi[1], hi[2], hi[3]));
          st16(p_lo + at, make_uint4(lo[0], lo[1], lo[2], lo[3]));
        }
      }
      fence_async_smem();
      tc_fence_before();
      lt_arrive(&sm->bar_p);
      // ---- output
      alive = sync_on(&sm->bar_o1, ph) && sync_on(&sm->bar_o2, ph);
      if (!alive) break;
      tc_fence_after();
      {
        uint32_t o1[32], o2[32], o3[32];
        lt_ld32_nowait(lanes + kLtO1 + half * 32, o1);
        lt_ld32_nowait(lanes + kLtO1 + kLtP + half * 32, o3);
        lt_ld32_nowait(lanes + kLtO2 + half * 32, o2);
        lt_wait_ld();
        const float er = exp2_weight(l_row);
        const int t = t_first + i * kLtC + row;
        __nv_bfloat16* dst = (__nv_bfloat16*)a.out + ((int64_t)(tok0 + t) * a.heads + h) * a.p + pbase + half * 32;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const uint4 x = ld16(v_t + lt_swz(row, half * 4 + c));
          const uint32_t xs[4] = {x.x, x.y, x.z, x.w};
          uint32_t w[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int at = c * 8 + 2 * e;
            const float u = fmaf(er, __uint_as_float(o1[at]) + __uint_as_float(o3[at]), __uint_as_float(o2[at])) + skip * __uint_as_float(xs[e] << 16);
            const float v = fmaf(er, __uint_as_float(o1[at + 1]) + __uint_as_float(o3[at + 1]), __uint_as_float(o2[at + 1])) + skip * __uint_as_float(xs[e] & 0xffff0000u);
            const __nv_bfloat162 pr = __floats2bfloat162_rn(u, v);
            w[e] = *reinterpret_cast<const uint32_t*>(&pr);
          }
          if (t < t_end && pbase + half * 32 + c * 8 < a.p) st16(dst + c * 8, make_uint4(w[0], w[1], w[2], w[3]));
        }
      }
      tc_fence_before();
    }
    if (alive) alive = sync_on(&sm->bar_st, nchunks - 1);
    if (alive) {
      tc_fence_after();
      float s[32], lo[32];
      tmem_ld32(st_at, s);
      tmem_ld32(st_at + kLtP, lo);
#pragma unroll
      for (int c = 0; c < 32; ++c) s[c] += lo[c];
      float* dst = kStateOnly ? sg.start + ((int64_t)bh * sg.count + seg) * np : (t_end == ntok ? final_state : nullptr);
      if (dst != nullptr && row < a.n) {
#pragma unroll
        for (int c = 0; c < 32; c += 4) {
          const int p = pbase + half * 32 + c;
          if (p < a.p) *reinterpret_cast<float4*>(dst + (int64_t)row * a.p + p) = make_float4(s[c], s[c + 1], s[c + 2], s[c + 3]);
        }
      }
    } else if (lane == 0 && *abort_flag == 0) {
      *abort_flag = 1; report(status, TKV_DEV_TIMEOUT);
    }
  }
  tc_fence_before();
  __syncthreads();
  // An aborting CTA drains the copies it started before its shared memory is released.
  if (tid == kLtRows && *abort_flag != 0) {
    if (qk_issued > 0) mbar_wait(&sm->bar_qk, (qk_issued - 1) & 1);
    for (int i = max(0, v_issued - 2); i < v_issued; ++i) mbar_wait(&sm->bar_v[i & 1], (i >> 1) & 1);
  }
  __syncthreads();
  if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kLtCols));
}

bool linrec_tc_shape(int n, int p, int max_tokens, int64_t tokens) {
  return n > 64 && n <= 128 && p >= kLtP && max_tokens >= kLtC && tokens < INT32_MAX - kLtC;
}

LinrecSegs linrec_tc_segments(int batch, int max_tokens, int heads, int p) {
  const int64_t ctas = (int64_t)batch * heads * ((p + kLtP - 1) / kLtP);
  const int chunks = (max_tokens + kLtC - 1) / kLtC;
  int segs = ctas > 0 ? (int)(148 / ctas) : 1;             // one CTA per SM
  if (segs > chunks / 4) segs = chunks / 4;                // segments of at least four chunks
  if (segs < 1) segs = 1;
  LinrecSegs s = {};
  const int per = (chunks + segs - 1) / segs;
  s.tokens = per * kLtC;
  s.count = (chunks + per - 1) / per;
  return s;
}

int launch_linrec_tc(const LinrecParams& a, const LinrecSegs& sg, int64_t tokens, int32_t* status, cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(linrec_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLtSmemBytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(linrec_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLtSmemBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk(tc): %s", cudaGetErrorString(e));
    configured = true;
  }
  CUtensorMap mq, mk, mv;
  int rc = make_map_3d_bf16(&mq, a.q, a.n, a.groups, tokens, a.q_stride, 64, kLtC);
  if (rc == TKV_OK) rc = make_map_3d_bf16(&mk, a.k, a.n, a.groups, tokens, a.k_stride, 64, kLtC);
  if (rc == TKV_OK) rc = make_map_3d_bf16(&mv, a.v, a.p, a.heads, tokens, a.v_stride, 64, kLtC);
  if (rc != TKV_OK) return rc;
  const int64_t grid = (int64_t)a.batch * a.heads * ((a.p + kLtP - 1) / kLtP) * sg.count;
  if (grid > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_chunk: %lld blocks", (long long)grid);
  cudaError_t e = cudaSuccess;
  if (sg.count > 1) {
    e = launch_pdl(linrec_tc_kernel<true>, dim3((unsigned)grid), dim3(kLtThreads), (size_t)kLtSmemBytes, st, mq, mk, mv, a, sg, status);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk(tc): %s", cudaGetErrorString(e));
    rc = launch_linrec_chain(a, sg, st);
    if (rc != TKV_OK) return rc;
  }
  e = launch_pdl(linrec_tc_kernel<false>, dim3((unsigned)grid), dim3(kLtThreads), (size_t)kLtSmemBytes, st, mq, mk, mv, a, sg, status);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk(tc): %s", cudaGetErrorString(e));
  return check_launch("tkv_linrec_chunk(tc)");
}

}  // namespace tkv
