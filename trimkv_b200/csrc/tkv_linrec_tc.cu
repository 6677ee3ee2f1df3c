// Chunked scalar-decay linear recurrence on tcgen05 + TMEM (the mathematics: tkv_linrec_chunk.cu), for state rows n up to
// 128 (padded to the MMA's 128), 64 value columns per CTA, chunks of 128 tokens.
//
// One CTA walks the chunks of one (request, head, 64 columns of v, segment).  Per chunk, D in TMEM:
//   S  [128 tok x 128 tok] = Q . K^T                     A = Q, B = K as TMA wrote them (K-major)
//   O1 [128 tok x 64]      = Q . S_prev                  B = the state before the chunk, high and low bf16 part (MN-major)
//   O2 [128 tok x 64]      = P . V                       A = P, the weighted scores, high and low part, read from TMEM;
//                                                        B = V (MN-major)
//   ST [128 n x 64]        = e^{L_end} ST + K^T . (w V)  A = K read MN-major, B = weighted values, high and low part
// The state stays in TMEM as the accumulator of its own update; once per chunk its rows pass through registers to be scaled
// and to be written as the operand of O1.  fp32 factors of a product enter as two bf16 parts, so nothing that recurs is
// rounded to 16 bits.
//
// Roles.  TMEM lane = token, or state row; a row is shared by two threads, one per column half.
//   warps 0-7   weight the scores: S -> P;
//   warps 8-15  pass the state through registers, weight the values, and write the output; they run the state side one
//               chunk ahead of the output side, so the chain ST -> operand -> ST never waits for scores;
//   warp 16     copies of Q and K, products S, O1, ST;   warp 17  running log decays;   warp 18  copies of V, product O2.
// O1 has two TMEM buffers; Q and K, and V, have two stages.  With M = 128 rows and N = 64 columns a product reads more operand
// bytes than shared memory delivers in the time of its multiplications, which is why P goes through TMEM.  A barrier is waited for in every phase by each of its waiters, or its next phase
// depends on the waiter, so that a parity never stands for two phases.  Every wait is bounded; on expiry the CTA records
// TKV_DEV_TIMEOUT, drains its copies, frees its TMEM and returns.
#include <cuda.h>
#include "tkv_linrec.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kLtC = 128, kLtP = 64;                       // tokens per chunk, value columns per CTA
constexpr int kLtRows = 256, kLtThreads = 2 * kLtRows + 96;   // threads of one row role; all
constexpr int kLtHalf = 16384;                             // 128 rows x 64 bf16
constexpr int kLtS = 0, kLtPm = 128, kLtO1 = 256, kLtO2 = 384, kLtST = 448, kLtCols = 512;   // P: high | low; O1: two buffers

struct LtSmem {
  float2 lv[2][kLtC];                                      // running log2 decay and value scale; by chunk parity
  uint64_t bar_qk[2], bar_v[2], bar_l[2], bar_s, bar_sfree, bar_sp, bar_o1, bar_wv, bar_st, bar_p, bar_o2, bar_e, bar_clr;
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

__device__ __forceinline__ void lt_st16(uint32_t taddr, const uint32_t* v) {   // without waiting
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
        "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
      : "memory");
}
// D += A . B with A in TMEM: lane = row, one 32-bit column holds two consecutive elements of a row.
__device__ __forceinline__ void lt_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t accum) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accum), "r"(0u) : "memory");
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

  uint8_t* q_s = base;                                     // two stages of two 64-column halves
  uint8_t* k_s = q_s + 4 * kLtHalf;
  uint8_t* v_s = k_s + 4 * kLtHalf;                        // two stages
  uint8_t* wv_s = v_s + 2 * kLtHalf;                       // high, low
  uint8_t* sp_s = wv_s + 2 * kLtHalf;                      // high, low
  LtSmem* sm = reinterpret_cast<LtSmem*>(sp_s + 2 * kLtHalf);
  volatile int* abort_flag = &sm->abort_flag;

  int issued = 0;                                          // of this thread's copies (a copy thread)
  const int row_first = tok0 + t_first;
  auto load_qk = [&](int i) {
    uint64_t* bar = &sm->bar_qk[i & 1];
    mbar_expect_tx(bar, (kStateOnly ? 2 : 4) * kLtHalf);
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int at = (2 * (i & 1) + hh) * kLtHalf;
      if (!kStateOnly) tma_load_3d(q_s + at, &map_q, bar, hh * 64, g, row_first + i * kLtC);
      tma_load_3d(k_s + at, &map_k, bar, hh * 64, g, row_first + i * kLtC);
    }
    ++issued;
  };
  auto load_v = [&](int i) {
    mbar_expect_tx(&sm->bar_v[i & 1], kLtHalf);
    tma_load_3d(v_s + (i & 1) * kLtHalf, &map_v, &sm->bar_v[i & 1], pbase, h, row_first + i * kLtC);
    ++issued;
  };
  constexpr int kCopyQK = 2 * kLtRows, kCopyV = 2 * kLtRows + 64;   // the two copy threads
  if (tid == kCopyQK) {
    for (int i = 0; i < 2; ++i) { mbar_init(&sm->bar_qk[i], 1); mbar_init(&sm->bar_v[i], 1); mbar_init(&sm->bar_l[i], 32); }
    mbar_init(&sm->bar_s, 1); mbar_init(&sm->bar_sfree, kLtRows);
    mbar_init(&sm->bar_o1, 1); mbar_init(&sm->bar_st, 1); mbar_init(&sm->bar_o2, 1);
    mbar_init(&sm->bar_sp, kLtRows); mbar_init(&sm->bar_wv, kLtRows); mbar_init(&sm->bar_p, kLtRows); mbar_init(&sm->bar_e, kLtRows);
    mbar_init(&sm->bar_clr, kLtRows);
    sm->abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncwarp();
  if (warp == 16) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kLtCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;
  const int64_t np = (int64_t)a.n * a.p;
  float* const final_state = a.state + ((int64_t)a.slots[b] * a.heads + h) * np;
  // operand descriptors: K-major, step k covers 16 columns; MN-major over 128 rows, step k covers 16 rows
  auto kmaj = [&](uint32_t at, int k) { return make_desc(at + (k >> 2) * kLtHalf + (k & 3) * 32, 16, 1024, 2); };
  auto mnmaj = [&](uint32_t at, int k) { return make_desc(at + k * 2048, kLtHalf, 1024, 2); };
  const int row = tid & 127, half = (tid >> 7) & 1;        // of a row thread
  const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  auto sync_on = [&](uint64_t* bar, int parity) {          // a whole warp
    const bool ok = mbar_wait_or_abort(bar, parity & 1, abort_flag);
    return (bool)__all_sync(0xffffffffu, ok);
  };
  bool alive = true;

  if (warp == 16) {
    // ------------------------------------------------------------------------------------ Q, K; S, O1, ST (one lane)
    if (lane == 0) {
      const uint32_t id_s = lt_idesc(128, 0, 0), id_o = lt_idesc(kLtP, 0, 1), id_st = lt_idesc(kLtP, 1, 1);
      const uint32_t sp = smem_u32(sp_s), wv = smem_u32(wv_s);
      load_qk(0);
      if (nchunks > 1) load_qk(1);
      for (int i = 0; i < nchunks; ++i) {
        const int ph = i & 1;
        const uint32_t qa = smem_u32(q_s + 2 * ph * kLtHalf), ka = smem_u32(k_s + 2 * ph * kLtHalf);
        alive = mbar_wait_or_abort(&sm->bar_qk[ph], (i >> 1) & 1, abort_flag);
        if (alive && i == nchunks - 1 && last_rows < kLtC) alive = mbar_wait_or_abort(&sm->bar_clr, 0, abort_flag);
        if (alive && !kStateOnly && i > 0) alive = mbar_wait_or_abort(&sm->bar_sfree, (i - 1) & 1, abort_flag);
        if (!alive) break;
        tc_fence_after();
        if (!kStateOnly) {
#pragma unroll
          for (int k = 0; k < 8; ++k) umma(tmem + kLtS, kmaj(qa, k), kmaj(ka, k), id_s, k > 0);
          umma_commit(&sm->bar_s);
        }
        if (i > 0 && i + 1 < nchunks) {                    // the other stage is free once the products of chunk i - 1 have completed
          alive = mbar_wait_or_abort(&sm->bar_st, (i - 1) & 1, abort_flag);
          if (alive && !kStateOnly) alive = mbar_wait_or_abort(&sm->bar_o1, (i - 1) & 1, abort_flag);
          if (!alive) break;
          load_qk(i + 1);
        }
        alive = mbar_wait_or_abort(&sm->bar_sp, ph, abort_flag);   // the state is scaled and its operand written; O1 of i - 2 is read
        if (!alive) break;
        tc_fence_after();
        if (!kStateOnly) {
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int k = 0; k < 8; ++k) umma(tmem + kLtO1 + 64 * ph, kmaj(qa, k), mnmaj(sp + part * kLtHalf, k), id_o, part > 0 || k > 0);
          umma_commit(&sm->bar_o1);
        }
        alive = mbar_wait_or_abort(&sm->bar_wv, ph, abort_flag);
        if (!alive) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 8; ++k) umma(tmem + kLtST, mnmaj(ka, k), mnmaj(wv + part * kLtHalf, k), id_st, 1);
        umma_commit(&sm->bar_st);
      }
    }
    __syncwarp();
  } else if (warp == 18) {
    // ------------------------------------------------------------------------------------ V; O2 (one lane)
    if (lane == 0) {
      const uint32_t id_o = lt_idesc(kLtP, 0, 1);
      load_v(0);
      if (nchunks > 1) load_v(1);
      for (int i = 0; i < nchunks; ++i) {
        // Chunk i - 1 is out: its V stage and O2 are free.  (Without outputs the last phases go unwatched: nothing holds them back.)
        if (i > 0 && (!kStateOnly || i + 1 < nchunks)) {
          alive = mbar_wait_or_abort(&sm->bar_e, (i - 1) & 1, abort_flag);
          if (!alive) break;
          if (i + 1 < nchunks) load_v(i + 1);
        }
        if (kStateOnly) continue;
        alive = mbar_wait_or_abort(&sm->bar_p, i & 1, abort_flag);
        if (alive) alive = mbar_wait_or_abort(&sm->bar_v[i & 1], (i >> 1) & 1, abort_flag);
        if (!alive) break;
        tc_fence_after();
        const uint32_t va = smem_u32(v_s + (i & 1) * kLtHalf);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 8; ++k) lt_umma_ts(tmem + kLtO2, tmem + kLtPm + part * 64 + k * 8, mnmaj(va, k), id_o, part > 0 || k > 0);
        umma_commit(&sm->bar_o2);
      }
    }
    __syncwarp();
  } else if (warp == 17) {
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
    for (int i = 0; i < nchunks; ++i) {
      d[1] += d[0]; d[2] += d[1]; d[3] += d[2];
      float sum = d[3];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += y;
      }
      const float before = sum - d[3];
      // The buffer last served chunk i - 2 (chunk i - 1 is only finished once lv of chunk i is there: one phase at a time)
      if (i >= 2) alive = sync_on(&sm->bar_e, i - 2);
      if (!alive) break;
      constexpr float kLog2e = 1.4426950408889634f;
#pragma unroll
      for (int e = 0; e < 4; ++e) sm->lv[i & 1][4 * lane + e] = make_float2((before + d[e]) * kLog2e, s[e]);
      seg_log += __shfl_sync(0xffffffffu, sum, 31) * kLog2e;
      lt_arrive(&sm->bar_l[i & 1]);
      if (i + 1 < nchunks) fetch(i + 1);
    }
    if (kStateOnly && alive && lane == 0 && pt == 0) sg.log_sum[(int64_t)bh * sg.count + seg] = seg_log;
  } else if (warp < 8) {
    // ------------------------------------------------------------------------------------ scores -> P: 64 columns of a row
    if (!kStateOnly) {
      const int j0 = half * 64, r0 = row & ~31;            // rows r0 .. r0 + 31 of this warp
      for (int i = 0; i < nchunks; ++i) {
        const float2* lv = sm->lv[i & 1];
        alive = sync_on(&sm->bar_l[i & 1], i >> 1) && sync_on(&sm->bar_s, i);
        if (alive && i > 0) alive = sync_on(&sm->bar_o2, i - 1);   // P of the previous chunk has been read
        if (!alive) break;
        tc_fence_after();
        const float l_row = lv[row].x;
#pragma unroll
        for (int c2 = 0; c2 < 2; ++c2) {
          const int jb = j0 + c2 * 32;
          const bool future = jb > r0 + 31;                // all of it (warp-uniform)
          uint32_t sv[32], hi[16], lo[16];
          if (!future) {
            lt_ld32_nowait(lanes + kLtS + jb, sv);
            lt_wait_ld();
          }
          if (c2 == 1) {
            tc_fence_before();
            lt_arrive(&sm->bar_sfree);
          }
          if (future) {
#pragma unroll
            for (int e = 0; e < 16; ++e) hi[e] = lo[e] = 0;
          } else {
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const int j = jb + 2 * e;
              const float4 w = *reinterpret_cast<const float4*>(&lv[j]);   // two tokens: log decay, scale
              const float x = j <= row ? __uint_as_float(sv[2 * e]) * exp2_weight(l_row - w.x) * w.y : 0.f;
              const float y = j + 1 <= row ? __uint_as_float(sv[2 * e + 1]) * exp2_weight(l_row - w.z) * w.w : 0.f;
              lt_split(x, y, &hi[e], &lo[e]);
            }
          }
          lt_st16(lanes + kLtPm + jb / 2, hi);
          lt_st16(lanes + kLtPm + 64 + jb / 2, lo);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        tc_fence_before();
        lt_arrive(&sm->bar_p);
      }
    }
  } else {
    // ------------------------------------------------------------------------------------ state, values, output: 32 columns of a row
    const uint32_t st_at = lanes + kLtST + half * 32;
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
    }
    const float skip = a.skip != nullptr ? a.skip[h] : 0.f;

    // State side of chunk i: the state before it becomes the operand of O1 and is scaled for its update; weighted values.
    auto state_side = [&](int i) -> bool {
      const float2* lv = sm->lv[i & 1];
      uint8_t* v_t = v_s + (i & 1) * kLtHalf;
      if (!sync_on(&sm->bar_l[i & 1], i >> 1)) return false;
      if (i > 0 && !sync_on(&sm->bar_st, i - 1)) return false;
      if (!kStateOnly && i > 0 && !sync_on(&sm->bar_o1, i - 1)) return false;   // the operand of the previous chunk has been read
      tc_fence_after();
      if (i == nchunks - 1 && last_rows < kLtC) {          // tokens beyond the end belong to another request: they read as zeros
        if (!sync_on(&sm->bar_qk[i & 1], i >> 1) || !sync_on(&sm->bar_v[i & 1], i >> 1)) return false;
        if (row >= last_rows) {
#pragma unroll
          for (int c = 0; c < 8; ++c) st16(k_s + (2 * (i & 1) + half) * kLtHalf + row * 128 + c * 16, make_uint4(0, 0, 0, 0));
#pragma unroll
          for (int c = 0; c < 4; ++c) st16(v_t + row * 128 + half * 64 + c * 16, make_uint4(0, 0, 0, 0));
        }
        fence_async_smem();
        lt_arrive(&sm->bar_clr);
      }
      const float lend = lv[kLtC - 1].x;
      {
        float s[32];
        tmem_ld32(st_at, s);
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
      }
      fence_async_smem();
      tc_fence_before();
      lt_arrive(&sm->bar_sp);
      if (!sync_on(&sm->bar_v[i & 1], i >> 1)) return false;
      const float w_row = exp2_weight(lend - lv[row].x) * lv[row].y;
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
      return true;
    };

    alive = state_side(0);
    for (int i = 0; i < nchunks && alive; ++i) {
      if (i + 1 < nchunks) alive = state_side(i + 1);
      else if (!kStateOnly) alive = sync_on(&sm->bar_o1, i);
      if (kStateOnly) {
        if (alive) lt_arrive(&sm->bar_e);
        continue;
      }
      if (alive) alive = sync_on(&sm->bar_o2, i);
      if (!alive) break;
      tc_fence_after();
      uint32_t o1[32], o2[32];
      lt_ld32_nowait(lanes + kLtO1 + 64 * (i & 1) + half * 32, o1);
      lt_ld32_nowait(lanes + kLtO2 + half * 32, o2);
      lt_wait_ld();
      const float er = exp2_weight(sm->lv[i & 1][row].x);
      const uint8_t* v_t = v_s + (i & 1) * kLtHalf;
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
          const float u = fmaf(er, __uint_as_float(o1[at]), __uint_as_float(o2[at])) + skip * __uint_as_float(xs[e] << 16);
          const float v = fmaf(er, __uint_as_float(o1[at + 1]), __uint_as_float(o2[at + 1])) + skip * __uint_as_float(xs[e] & 0xffff0000u);
          const __nv_bfloat162 pr = __floats2bfloat162_rn(u, v);
          w[e] = *reinterpret_cast<const uint32_t*>(&pr);
        }
        if (t < t_end && pbase + half * 32 + c * 8 < a.p) st16(dst + c * 8, make_uint4(w[0], w[1], w[2], w[3]));
      }
      tc_fence_before();
      lt_arrive(&sm->bar_e);
    }
    if (alive) alive = sync_on(&sm->bar_st, nchunks - 1);
    if (alive) {
      tc_fence_after();
      float s[32];
      tmem_ld32(st_at, s);
      float* dst = kStateOnly ? sg.start + ((int64_t)bh * sg.count + seg) * np : (t_end == ntok ? final_state : nullptr);
      if (dst != nullptr && row < a.n) {
#pragma unroll
        for (int c = 0; c < 32; c += 4) {
          const int p = pbase + half * 32 + c;
          if (p < a.p) *reinterpret_cast<float4*>(dst + (int64_t)row * a.p + p) = make_float4(s[c], s[c + 1], s[c + 2], s[c + 3]);
        }
      }
    }
  }
  if (!alive && *abort_flag == 0) { *abort_flag = 1; report(status, TKV_DEV_TIMEOUT); }
  tc_fence_before();
  __syncthreads();
  // An aborting CTA drains the copies it started before its shared memory is released.
  if (*abort_flag != 0) {
    if (tid == kCopyQK || tid == kCopyV)
      for (int i = max(0, issued - 2); i < issued; ++i) mbar_wait(tid == kCopyQK ? &sm->bar_qk[i & 1] : &sm->bar_v[i & 1], (i >> 1) & 1);
  }
  __syncthreads();
  if (warp == 16) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kLtCols));
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
