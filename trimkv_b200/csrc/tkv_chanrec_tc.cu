// Chunked channel-decay recurrence on tcgen05 + TMEM, for 64 < n <= 128 state rows and 128 value columns per CTA, chunks of 32
// tokens.  With P_i the product of the forget gates of the chunk up to token i, R_j the product of those after token j, E = P_32
// (all per state row) and S the state before the chunk:
//   O^T  [128 p x 32 tok] = S^T . (q P) + V^T . a^T        a_ij = (q_i / R_i) . (k_j R_j),  j <= i,  k = 1 - f
//   S^T  [128 p x 128 n]  = E S^T + V^T . (k R)
// The state stays in TMEM as the accumulator of its own update (lane = value column, column = state row); once per chunk it
// passes through registers to be written as the operand of the read-out, a high and a low bf16 part, and to be scaled by E.  k R
// and a enter their products as two parts as well, v is 16-bit exactly, q P and q / R are rounded once, which is what rounding
// q to 16 bits does.  k R and q P exist for all gates; q / R is used where every channel's gates keep kCtWide over eight tokens.
// Where they keep kCtNarrow, products and quotients of a reach over 16 tokens only (between the halves of the chunk: the gates
// before the one and after the other); below that a is summed up pair by pair in fp32.
//
// Roles, each ahead of the next by up to one chunk:
//   warps 0-7   gates and scaled vectors (a thread walks two channels of eight tokens), the blocks of a (mma.sync), the
//               copies of the projections;
//   warps 8-15  the state's way through registers, the outputs of the chunk before; one lane of warp 8 issues the products.
// Every wait is bounded; on expiry the CTA records TKV_DEV_TIMEOUT, lets its copies land, frees its TMEM and returns.
#include "tkv_attn_block.cuh"
#include "tkv_chanrec_math.cuh"

namespace tkv {

constexpr int kCtTok = 32, kCtP = 128, kCtN = 128;
constexpr int kCtGroup = 256, kCtThreads = 2 * kCtGroup;
constexpr int kCtTile = 8192, kCtHalf = 4096;              // 32 rows x 128 columns: two halves of 64 columns, 128-byte swizzle
constexpr int kCtSop = 65536;                              // state operand: [part][64-column half][128 rows x 128 bytes]
constexpr int kCtStage = 3 * kCtTile + 4096;               // q P | k R high | k R low | a
constexpr int kCtSt = 0, kCtO = 128, kCtCols = 256;        // TMEM columns: state, two output buffers of 32
constexpr float kCtWide = 3e-8f, kCtNarrow = 1e-15f;        // product of eight gates

struct CtSmem {
  float oct[2][4][kCtN];                                   // product of eight tokens' gates, and of their reciprocals
  float end[2][kCtN];                                      // E, by chunk parity
  uint64_t full[2], done[2], sop, sync[3];
  int level[2];                                            // by chunk parity: 0 wide, 1 narrow, 2 pair by pair
  uint32_t tmem_base;
  int abort_flag;
};
constexpr int kCtRaw = 2 * kCtTile;                        // z_q | z_f of a chunk, rows of 256 bytes
constexpr int kCtBytes = kCtSop + 2 * kCtStage + 3 * kCtTile + 3 * kCtTile + 2 * kCtRaw + (int)sizeof(CtSmem);
static_assert(kCtBytes <= 232448, "shared memory of the kernel");

__device__ __forceinline__ uint32_t ct_idesc(int n, int a_mn, int b_mn) {   // bf16 operands, fp32 D, M = 128
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)b_mn << 16) | ((uint32_t)(n >> 3) << 17) | ((128u >> 4) << 24);
}
// Byte of 16-byte piece c (0 .. 15) of row r of a 32 x 128 tile.
__device__ __forceinline__ uint32_t ct_at(int r, int c) { return (uint32_t)((c >> 3) * kCtHalf + r * 128 + (((c & 7) ^ (r & 7)) << 4)); }
// Byte of the pair of columns (j, j + 1), j even, of row i of the block a (part 1: low).
__device__ __forceinline__ uint32_t ct_a(int i, int j, int part) {
  const int col = part * 32 + j;
  return (uint32_t)(i * 128 + (((col >> 3) ^ (i & 7)) << 4) + (col & 7) * 2);
}

// One arrival per warp, after what all its lanes have written.
__device__ __forceinline__ void ct_arrive(uint64_t* bar) {
  __syncwarp();
  if ((threadIdx.x & 31) == 0) da_arrive(bar);
}

template <bool kStateOnly>
__global__ void __launch_bounds__(kCtThreads, 1) chanrec_tc_kernel(ChanrecParams a, ChanrecSegs sg, int32_t* status) {
  extern __shared__ __align__(1024) uint8_t base[];
  grid_dependency_wait();
  grid_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ptiles = (a.p + kCtP - 1) / kCtP, per_seg = a.batch * a.heads * ptiles;
  const int seg = blockIdx.x / per_seg, item = blockIdx.x - seg * per_seg;      // kStateOnly: a piece of a segment
  const int pt = item % ptiles, bh = item / ptiles, b = bh / a.heads, h = bh - b * a.heads;
  const int tok0 = a.cu[b], ntok = a.cu[b + 1] - tok0;
  const int seg_tokens = kStateOnly ? sg.tokens / sg.pieces : sg.tokens;
  const int t_first = seg * seg_tokens, t_end = min(ntok, t_first + seg_tokens);
  if (t_first >= t_end) return;
  if (kStateOnly && (seg / sg.pieces + 1) * sg.tokens >= ntok) return;          // nobody starts from the end of the last segment
  if ((smem_u32(base) & 1023u) != 0) {                     // the swizzled tiles need it; the launch gives it
    if (tid == 0) report(status, TKV_DEV_TIMEOUT);
    return;
  }
  const int nchunks = (t_end - t_first + kCtTok - 1) / kCtTok, pbase = pt * kCtP;
  uint8_t* sop_s = base;
  uint8_t* op_s = sop_s + kCtSop;                          // two stages
  uint8_t* v_s = op_s + 2 * kCtStage;                      // three stages
  uint8_t* qh_s = v_s + 3 * kCtTile;                       // q / R
  uint8_t* k16_s = qh_s + kCtTile;                         // narrow: k times the gates after it in its half, high | low (rows 0-15); q
                                                           // times those before it in its half (rows 16-31 of the first tile)
  uint8_t* raw_s = k16_s + 2 * kCtTile;                    // two stages
  CtSmem* sm = reinterpret_cast<CtSmem*>(raw_s + 2 * kCtRaw);
  volatile int* abort_flag = &sm->abort_flag;

  if (tid == 0) {
    for (int i = 0; i < 2; ++i) { mbar_init(&sm->full[i], kCtGroup / 32); mbar_init(&sm->done[i], 1); sm->level[i] = 0; }
    mbar_init(&sm->sop, kCtGroup / 32);
    for (int i = 0; i < 3; ++i) mbar_init(&sm->sync[i], kCtGroup / 32);
    sm->abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 8) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_base)), "r"(kCtCols));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
  }
  // the upper right block of a stays zero
  for (int i = tid; i < 2 * kCtStage / 16; i += kCtThreads) st16(op_s + i * 16, make_uint4(0, 0, 0, 0));
  fence_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm->tmem_base;
  const int64_t np = (int64_t)a.n * a.p;
  float* const final_state = a.state + ((int64_t)a.slots[b] * a.heads + h) * np;

  if (warp < 8) {
    // ------------------------------------------------------------------------------------ gates, scaled vectors, a
    const __nv_bfloat16* Q = (const __nv_bfloat16*)a.q + (int64_t)(tok0 + t_first) * a.row_stride + (int64_t)h * a.n;
    const __nv_bfloat16* F = (const __nv_bfloat16*)a.f + (int64_t)(tok0 + t_first) * a.row_stride + (int64_t)h * a.n;
    const __nv_bfloat16* V = (const __nv_bfloat16*)a.v + (int64_t)(tok0 + t_first) * a.row_stride + (int64_t)h * a.p + pbase;
    const float *bias = a.f_bias + (int64_t)h * a.n, *lower = a.lower + (int64_t)h * a.n;
    const int tokens = t_end - t_first;
    // copies: this thread's 16-byte piece of rows cr, cr + 16
    const int cr = tid >> 4, cc = tid & 15;
    const bool q_in = cc * 8 < a.n, v_in = pbase + cc * 8 < a.p;
    const int64_t step16 = 16 * a.row_stride;
    const __nv_bfloat16 *Qt = Q + (int64_t)cr * a.row_stride + cc * 8, *Ft = F + (int64_t)cr * a.row_stride + cc * 8, *Vt = V + (int64_t)cr * a.row_stride + cc * 8;
    const uint32_t raw_to = smem_u32(raw_s) + cr * 256 + cc * 16, v_to = smem_u32(v_s) + ct_at(cr, cc);   // rows 16 apart: + 4096, + 2048
    auto copy = [&](uint32_t to, const __nv_bfloat16* from, const __nv_bfloat16* any, bool live) {
      const int bytes = live ? 16 : 0;                     // 0: the 16 bytes are zero-filled
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(live ? from : any), "r"(bytes) : "memory");
    };
    auto load = [&](int i, int vst) {
      const uint32_t raw = raw_to + (i & 1) * kCtRaw, vt = v_to + vst * kCtTile;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const bool in = i * kCtTok + cr + 16 * e < tokens;
        if (!kStateOnly) copy(raw + e * 4096, Qt + e * step16, Q, in && q_in);
        copy(raw + kCtTile + e * 4096, Ft + e * step16, F, in && q_in);
        copy(vt + e * 2048, Vt + e * step16, V, in && v_in);
      }
      Qt += 2 * step16; Ft += 2 * step16; Vt += 2 * step16;
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto meet = [&](int which, int i) {
      ct_arrive(&sm->sync[which]);
      const bool ok = mbar_wait_or_abort(&sm->sync[which], i & 1, abort_flag);
      return (bool)__all_sync(0xffffffffu, ok);
    };
    const int oct = warp & 3, r0 = oct * 8, c = (warp >> 2) * 64 + 2 * lane;
    // a channel that does not exist keeps its (zero) state: lower bound 1
    const float2 bi = c < a.n ? mul2(*reinterpret_cast<const float2*>(bias + c), pair(kMinusLog2e)) : pair(0.f);
    const float2 lo = c < a.n ? *reinterpret_cast<const float2*>(lower + c) : pair(1.f);
    const float2 rest = make_float2(1.0f - lo.x, 1.0f - lo.y);
    uint32_t at8[8];                                       // byte of this thread's channels in its eight rows of a tile
#pragma unroll
    for (int j = 0; j < 8; ++j) at8[j] = ct_at(r0 + j, c >> 3) + (c & 7) * 2;
    float2 seg_decay = pair(1.0f);
    bool alive = true;
    int vnext = 1;                                         // (i + 1) mod 3
    load(0, 0);
    for (int i = 0; i < nchunks; ++i, vnext = vnext == 2 ? 0 : vnext + 1) {
      const int st = i & 1;
      uint8_t* op = op_s + st * kCtStage;
      const uint8_t* raw = raw_s + st * kCtRaw;
      if (i >= 2) {                                        // the products that read this stage, and the values of chunk i - 2, are done
        alive = mbar_wait_or_abort(&sm->done[st], ((i - 2) >> 1) & 1, abort_flag);
        alive = __all_sync(0xffffffffu, alive);
        if (!alive) break;
      }
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      alive = meet(0, i);                                  // this chunk is here; everyone is done with the last one
      if (!alive) break;
      if (i + 1 < nchunks) load(i + 1, vnext);
      float2 f[8], fi[8], k[8], fp = pair(1.0f), ip = fp;
      auto walk8 = [&](int live) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const uint32_t z = *reinterpret_cast<const uint32_t*>(raw + kCtTile + (r0 + j) * 256 + c * 2);
          const float2 y = fma2(make_float2(__uint_as_float(z << 16), __uint_as_float(z & 0xffff0000u)), pair(kMinusLog2e), bi);
          if (kStateOnly) { cr_gate(y, lo, rest, &f[j], &k[j]); fi[j] = f[j]; }
          else cr_gate(y, lo, rest, &f[j], &fi[j], &k[j]);
          if (j >= live) { f[j] = pair(1.0f); fi[j] = f[j]; k[j] = pair(0.0f); }
          fp = mul2(fp, f[j]);
          if (!kStateOnly) ip = mul2(ip, fi[j]);
        }
      };
      if ((i + 1) * kCtTok <= tokens) walk8(8);
      else walk8(tokens - i * kCtTok - r0);
      *reinterpret_cast<float2*>(&sm->oct[0][oct][c]) = fp;
      if (!kStateOnly) {
        *reinterpret_cast<float2*>(&sm->oct[1][oct][c]) = ip;
        if (!(fp.x >= kCtWide && fp.y >= kCtWide)) atomicMax(&sm->level[st], fp.x >= kCtNarrow && fp.y >= kCtNarrow ? 1 : 2);
      }
      alive = meet(1, i);
      if (!alive) break;
      const int level = kStateOnly ? 0 : *(volatile int*)&sm->level[st];
      if (tid == 0) sm->level[st ^ 1] = 0;
      // ---- q P forward, k R and q / R backward
      float2 before = pair(1.0f), after = before, iafter = before;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 x = *reinterpret_cast<const float2*>(&sm->oct[0][q][c]);
        if (q < oct) before = mul2(before, x);
        if (q > oct) {
          after = mul2(after, x);
          if (!kStateOnly) iafter = mul2(iafter, *reinterpret_cast<const float2*>(&sm->oct[1][q][c]));
        }
      }
      if (oct == 3) {
        const float2 end = mul2(before, fp);
        *reinterpret_cast<float2*>(&sm->end[st][c]) = end;
        seg_decay = mul2(seg_decay, end);
      }
      float2 qv[8];
      if (!kStateOnly) {
        float2 P = before;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const uint32_t z = *reinterpret_cast<const uint32_t*>(raw + (r0 + j) * 256 + c * 2);
          qv[j] = cr_silu2(make_float2(__uint_as_float(z << 16), __uint_as_float(z & 0xffff0000u)));
          P = mul2(P, f[j]);
          const float2 x = mul2(qv[j], P);
          *reinterpret_cast<__nv_bfloat162*>(op + at8[j]) = __floats2bfloat162_rn(x.x, x.y);
        }
      }
#pragma unroll
      for (int j = 7; j >= 0; --j) {
        uint32_t hi, lo_;
        cr_split(mul2(k[j], after), &hi, &lo_);
        *reinterpret_cast<uint32_t*>(op + kCtTile + at8[j]) = hi;
        *reinterpret_cast<uint32_t*>(op + 2 * kCtTile + at8[j]) = lo_;
        after = mul2(after, f[j]);
        if (!kStateOnly) {
          const float2 x = mul2(qv[j], iafter);
          *reinterpret_cast<__nv_bfloat162*>(qh_s + at8[j]) = __floats2bfloat162_rn(x.x, x.y);
          iafter = mul2(iafter, fi[j]);
        }
      }
      if (!kStateOnly) {
        uint8_t* at = op + 3 * kCtTile;
        if (level == 1) {
          if (oct < 2) {
            float2 a16 = pair(1.0f), i16 = a16;
            if (oct == 0) { a16 = *reinterpret_cast<const float2*>(&sm->oct[0][1][c]); i16 = *reinterpret_cast<const float2*>(&sm->oct[1][1][c]); }
#pragma unroll
            for (int j = 7; j >= 0; --j) {
              uint32_t hi, lo_;
              cr_split(mul2(k[j], a16), &hi, &lo_);
              *reinterpret_cast<uint32_t*>(k16_s + at8[j]) = hi;
              *reinterpret_cast<uint32_t*>(k16_s + kCtTile + at8[j]) = lo_;
              const float2 x = mul2(qv[j], i16);
              *reinterpret_cast<__nv_bfloat162*>(qh_s + at8[j]) = __floats2bfloat162_rn(x.x, x.y);
              a16 = mul2(a16, f[j]);
              i16 = mul2(i16, fi[j]);
            }
          } else {
            float2 p16 = oct == 3 ? *reinterpret_cast<const float2*>(&sm->oct[0][2][c]) : pair(1.0f);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              p16 = mul2(p16, f[j]);
              const float2 x = mul2(qv[j], p16);
              *reinterpret_cast<__nv_bfloat162*>(k16_s + at8[j]) = __floats2bfloat162_rn(x.x, x.y);
            }
          }
        }
        if (level < 2) {
          alive = meet(2, i);
          if (!alive) break;
          if (warp < 6) {
            // ---- a task is 16 tokens against 8; the last two cross the middle of the chunk
            const int gr = lane >> 2, gc = lane & 3;
            const int ib = warp < 4 ? warp >> 1 : 1, jb = warp < 4 ? ib : 0, j0 = jb * 16 + (warp & 1) * 8;
            const uint32_t qa = smem_u32(level == 1 && warp >= 4 ? k16_s : qh_s);
            const uint32_t ka = smem_u32(level == 1 && jb == 0 ? k16_s : op + kCtTile) + (lane >> 4) * kCtTile;
            const int qrow = ib * 16 + (lane & 15), krow = j0 + (lane & 7);
            float sc[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < kCtN / 16; ++kk) {
              uint32_t aq[4], kf[4];                       // kf: 8 tokens of the high part, then of the low part
              asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                           : "=r"(aq[0]), "=r"(aq[1]), "=r"(aq[2]), "=r"(aq[3]) : "r"(qa + ct_at(qrow, kk * 2 + (lane >> 4))) : "memory");
              asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                           : "=r"(kf[0]), "=r"(kf[1]), "=r"(kf[2]), "=r"(kf[3]) : "r"(ka + ct_at(krow, kk * 2 + ((lane >> 3) & 1))) : "memory");
              cr_mma(sc[0], aq, kf[0], kf[1]);
              cr_mma(sc[1], aq, kf[2], kf[3]);
            }
            const int j = j0 + 2 * gc;
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
              const int r = ib * 16 + gr + (e >> 1) * 8;
              uint32_t hi, lo_;
              cr_split(make_float2(j <= r ? sc[0][e] + sc[1][e] : 0.f, j + 1 <= r ? sc[0][e + 1] + sc[1][e + 1] : 0.f), &hi, &lo_);
              *reinterpret_cast<uint32_t*>(at + ct_a(r, j, 0)) = hi;
              *reinterpret_cast<uint32_t*>(at + ct_a(r, j, 1)) = lo_;
            }
          }
        } else {
          // ---- a pair by pair: a warp takes rows warp, warp + 8, ..; a lane four channels
          const int n0 = lane * 4;
          const bool in = n0 < a.n;
          float bz[4] = {0.f, 0.f, 0.f, 0.f}, lz[4] = {1.f, 1.f, 1.f, 1.f};
          if (in)
#pragma unroll
            for (int e = 0; e < 4; ++e) { bz[e] = bias[n0 + e]; lz[e] = lower[n0 + e]; }
          auto raw4 = [&](int off, int r, float* x) {
            const uint2 z = *reinterpret_cast<const uint2*>(raw + off + r * 256 + n0 * 2);
            x[0] = __uint_as_float(z.x << 16); x[1] = __uint_as_float(z.x & 0xffff0000u);
            x[2] = __uint_as_float(z.y << 16); x[3] = __uint_as_float(z.y & 0xffff0000u);
          };
          for (int r = warp; r < kCtTok; r += 8) {
            float q4[4], x[4];
            raw4(0, r, q4);
#pragma unroll
            for (int e = 0; e < 4; ++e) q4[e] = cr_silu(q4[e]);     // then times the gates between the pair
            float row = 0.f;                               // lane j: a of the pair (r, j)
            for (int j = r; j >= 0; --j) {
              raw4(kCtTile, j, x);
              float part = 0.f;
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                float pos, neg;
                cr_sigmoid(x[e] + bz[e], &pos, &neg);
                part = fmaf(q4[e], (1.0f - lz[e]) * neg, part);
                q4[e] *= fmaf(1.0f - lz[e], pos, lz[e]);
              }
              part = warp_add(part);
              if (lane == j) row = part;
            }
            const __nv_bfloat16 hi = __float2bfloat16_rn(row);
            const uint32_t odd = (lane & 1) * 2;
            *reinterpret_cast<__nv_bfloat16*>(at + ct_a(r, lane & ~1, 0) + odd) = hi;
            *reinterpret_cast<__nv_bfloat16*>(at + ct_a(r, lane & ~1, 1) + odd) = __float2bfloat16_rn(row - __bfloat162float(hi));
          }
          alive = meet(2, i);
          if (!alive) break;
        }
      }
      fence_async_smem();
      ct_arrive(&sm->full[st]);
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    if (!alive && lane == 0 && *abort_flag == 0) { *abort_flag = 1; report(status, TKV_DEV_TIMEOUT); }
    if (kStateOnly && alive && oct == 3 && pt == 0 && c < a.n)
      *reinterpret_cast<float2*>(sg.decay + ((int64_t)bh * sg.count * sg.pieces + seg) * a.n + c) = seg_decay;
  } else {
    // ------------------------------------------------------------------------------------ state and outputs: lane = value column
    const int quarter = warp & 3, half = (warp - 8) >> 2, row = quarter * 32 + lane, pc = pbase + row;
    const uint32_t lanes = tmem + ((uint32_t)(quarter * 32) << 16);
    const uint32_t st_at = lanes + kCtSt + half * 64;
    auto sync_on = [&](uint64_t* bar, int parity) {
      const bool ok = mbar_wait_or_abort(bar, parity & 1, abort_flag);
      return (bool)__all_sync(0xffffffffu, ok);
    };
    {
      const float* S = kStateOnly ? nullptr : sg.count > 1 ? sg.start + ((int64_t)bh * sg.count + seg) * sg.pieces * np : a.pos0[b] == 0 ? nullptr : final_state;
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        float s[32];
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const int n = half * 64 + c2 * 32 + c;
          s[c] = S != nullptr && n < a.n && pc < a.p ? S[(int64_t)n * a.p + pc] : 0.f;
        }
        da_st32(st_at + c2 * 32, s);
      }
    }
    // outputs of chunk i: 16 tokens of this column; neighbouring lanes exchange, so that a store holds two columns
    const bool odd = lane & 1;
    const int64_t out_row = (int64_t)a.heads * a.p;        // elements between tokens
    __nv_bfloat16* const out0 = (__nv_bfloat16*)a.out + (int64_t)(tok0 + t_first + half * 16 + (odd ? 1 : 0)) * out_row + (int64_t)h * a.p + (pc & ~1);
    auto outputs = [&](int i) {
      float v[16];
      tmem_ld16(lanes + kCtO + (i & 1) * kCtTok + half * 16, v);
      const int live = pc < a.p ? t_end - (t_first + i * kCtTok + half * 16 + (odd ? 1 : 0)) : 0;
      __nv_bfloat16* dst = out0 + (int64_t)i * kCtTok * out_row;
#pragma unroll
      for (int c = 0; c < 16; c += 2) {
        const float mine = odd ? v[c + 1] : v[c], y = __shfl_xor_sync(0xffffffffu, odd ? v[c] : v[c + 1], 1);
        if (c < live) *reinterpret_cast<uint32_t*>(dst) = odd ? da_pack2(y, mine) : da_pack2(mine, y);
        dst += 2 * out_row;
      }
    };
    const uint32_t id_o = ct_idesc(kCtTok, 0, 0), id_a = ct_idesc(kCtTok, 1, 0), id_s = ct_idesc(kCtN, 1, 1);
    // descriptors of the first stage; another place is the address field (16-byte units) moved on
    const uint64_t d_sop = make_desc(smem_u32(sop_s), 16, 1024, 2), d_q = make_desc(smem_u32(op_s), 16, 1024, 2);
    const uint64_t d_k = make_desc(smem_u32(op_s) + kCtTile, kCtHalf, 1024, 2), d_v = make_desc(smem_u32(v_s), kCtHalf, 1024, 2);
    auto products = [&](int i, int vst) {                  // one thread, once the chunk's operands and the state's are there
      tc_fence_after();
      const uint64_t q = d_q + (i & 1) * (kCtStage >> 4), k = d_k + (i & 1) * (kCtStage >> 4), v = d_v + vst * (kCtTile >> 4), at = q + (3 * kCtTile >> 4);
      const uint32_t o = tmem + kCtO + (i & 1) * kCtTok;
#pragma unroll
      for (int e = 0; e < 4; ++e)                          // high and low part of k R, 16 tokens each
        umma(tmem + kCtSt, v + (e & 1) * 128, k + (e >> 1) * (kCtTile >> 4) + (e & 1) * 128, id_s, 1);
      if (!kStateOnly) {
#pragma unroll
        for (int e = 0; e < 16; ++e)
          umma(o, d_sop + (e >> 3) * 2048 + ((e >> 2) & 1) * 1024 + (e & 3) * 2, q + ((e >> 2) & 1) * (kCtHalf >> 4) + (e & 3) * 2, id_o, e > 0);
#pragma unroll
        for (int e = 0; e < 4; ++e) umma(o, v + (e & 1) * 128, at + e * 2, id_a, 1);
      }
      umma_commit(&sm->done[i & 1]);
    };
    bool alive = true;
    int vst = 0;                                           // i mod 3
    for (int i = 0; i < nchunks; ++i, vst = vst == 2 ? 0 : vst + 1) {
      if (i > 0) alive = sync_on(&sm->done[(i - 1) & 1], (i - 1) >> 1);
      if (alive) alive = sync_on(&sm->full[i & 1], i >> 1);
      if (!alive) break;
      tc_fence_after();
      const float4* end = reinterpret_cast<const float4*>(&sm->end[i & 1][half * 64]);
      uint32_t x[64];
      da_ld32_nowait(st_at, x);
      da_ld32_nowait(st_at + 32, x + 32);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        float s[32];
#pragma unroll
        for (int c = 0; c < 32; c += 8) {
          if (!kStateOnly) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e)
              cr_split(make_float2(__uint_as_float(x[c2 * 32 + c + 2 * e]), __uint_as_float(x[c2 * 32 + c + 2 * e + 1])), &hi[e], &lo[e]);
            const uint32_t at = half * 16384 + row * 128 + (((c2 * 4 + c / 8) ^ (row & 7)) << 4);
            st16(sop_s + at, make_uint4(hi[0], hi[1], hi[2], hi[3]));
            st16(sop_s + 32768 + at, make_uint4(lo[0], lo[1], lo[2], lo[3]));
          }
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float4 d = end[c2 * 8 + c / 4 + e];
            const int at = c + 4 * e;
            const float2 u = mul2(make_float2(__uint_as_float(x[c2 * 32 + at]), __uint_as_float(x[c2 * 32 + at + 1])), make_float2(d.x, d.y));
            const float2 w = mul2(make_float2(__uint_as_float(x[c2 * 32 + at + 2]), __uint_as_float(x[c2 * 32 + at + 3])), make_float2(d.z, d.w));
            s[at] = u.x; s[at + 1] = u.y; s[at + 2] = w.x; s[at + 3] = w.y;
          }
        }
        da_st32(st_at + c2 * 32, s);
      }
      if (!kStateOnly) fence_async_smem();
      tc_fence_before();
      ct_arrive(&sm->sop);
      if (warp == 8) {
        alive = sync_on(&sm->sop, i);
        if (!alive) break;
        if (lane == 0) products(i, vst);
        __syncwarp();
      }
      if (!kStateOnly && i > 0) outputs(i - 1);
    }
    if (alive) alive = sync_on(&sm->done[(nchunks - 1) & 1], (nchunks - 1) >> 1);
    if (alive) {
      tc_fence_after();
      if (!kStateOnly) outputs(nchunks - 1);
      float* dst = kStateOnly ? sg.start + ((int64_t)bh * sg.count * sg.pieces + seg) * np : (t_end == ntok ? final_state : nullptr);
#pragma unroll
      for (int c2 = 0; c2 < 2; ++c2) {
        float s[32];
        tmem_ld32(st_at + c2 * 32, s);
        if (dst != nullptr && pc < a.p)
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            const int n = half * 64 + c2 * 32 + c;
            if (n < a.n) dst[(int64_t)n * a.p + pc] = s[c];
          }
      }
    } else if (lane == 0 && *abort_flag == 0) {
      *abort_flag = 1; report(status, TKV_DEV_TIMEOUT);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kCtCols));
}

bool chanrec_tc_shape(int n, int p, int max_tokens) { return n > 64 && n <= kCtN && p > 64 && max_tokens >= 2 * kCtTok; }
int chanrec_tc_columns() { return kCtP; }

int launch_chanrec_tc(const ChanrecParams& a, const ChanrecSegs& sg, int32_t* status, cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(chanrec_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kCtBytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chanrec_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kCtBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_chunk(tc): %s", cudaGetErrorString(e));
    configured = true;
  }
  const int64_t grid = (int64_t)a.batch * a.heads * ((a.p + kCtP - 1) / kCtP) * sg.count, pieces = grid * sg.pieces;
  if (pieces > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_chunk: %lld blocks", (long long)grid);
  cudaError_t e = cudaSuccess;
  if (sg.count > 1) {
    e = launch_pdl(chanrec_tc_kernel<true>, dim3((unsigned)pieces), dim3(kCtThreads), (size_t)kCtBytes, st, a, sg, status);
    if (e == cudaSuccess) {
      int rc = launch_chanrec_chain(a, sg, st);
      if (rc != TKV_OK) return rc;
    }
  }
  if (e == cudaSuccess) e = launch_pdl(chanrec_tc_kernel<false>, dim3((unsigned)grid), dim3(kCtThreads), (size_t)kCtBytes, st, a, sg, status);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_chunk(tc): %s", cudaGetErrorString(e));
  return check_launch("tkv_chanrec_chunk(tc)");
}

}  // namespace tkv
