// Chunked form of the channel-decay recurrence (tkv_chanrec.cuh) for prompts, 16-bit operands with fp32 state.
//
// A block of tokens, with P_i the product of the forget gates of its tokens up to i (per state row), S the state before it:
//   a_ij = (q_i P_i) . (k_j / P_j)           j <= i, k = 1 - f
//   o_i  = S^T (q_i P_i) + sum_j a_ij v_j
//   S   <- diag(P_end) (S + sum_j (k_j / P_j) v_j^T) .
// k / P is fp32 and enters the 16-bit products as a high and a low part, as do the state and a; v is 16-bit exactly, and q P is
// rounded once, which is what rounding q itself to 16 bits does.  1 / P must stay in the range of fp32: a chunk of 32 tokens is
// one block where every channel's gates keep kWide over eight tokens, two blocks of 16 where they keep kNarrow, and is walked
// token by token below that (gates near zero).
//
// One CTA walks the chunks of one (request, head, block of 16 * kWarps value columns, segment of the sequence).  The state never
// leaves registers: a warp owns 16 columns of v and holds S^T [16 x n] as fp32 MMA accumulators, whose layout is also the
// A-operand layout of the read-out.  Per chunk: gates and scaled vectors of all channels (a thread walks two channels of eight
// tokens), the 16 x 16 blocks of a, then every warp its own columns without further barriers.
// Where (request, head, column) blocks alone do not fill the GPU, the sequence is cut into segments: a first pass computes
// every segment's own state (with the products of the gates AFTER a token, which need no quotient and hold for all gates), a
// small kernel chains them, and the main pass starts each segment from its true state.
#include <type_traits>
#include "tkv_chanrec_math.cuh"

namespace tkv {

constexpr int kCrTokens = 32;
constexpr float kWide = 3e-8f, kNarrow = 1e-15f;          // product of eight gates

template <int NP, int kWarps> struct CrSmem {
  static constexpr int PT = kWarps * 16, QS = NP + 8, VS = PT + 8, PS = kCrTokens + 8;
  __nv_bfloat16 zq[2][kCrTokens * QS], zf[2][kCrTokens * QS], v[2][kCrTokens * VS];
  __nv_bfloat16 q[kCrTokens * QS], k_hi[kCrTokens * QS], k_lo[kCrTokens * QS];
  __nv_bfloat16 a_hi[kCrTokens * PS], a_lo[kCrTokens * PS];
  float oct[2][4][NP];                                    // product of eight tokens' gates, and of their reciprocals
  float end[2][NP];                                       // product of the gates of a block (one block: the first)
  int level[2];                                           // by chunk parity: 0 one block, 1 two blocks, 2 token by token
  float gate[2][3][NP];                                   // q, f, k of one token (token-by-token path)
};

template <int NP, int kWarps, bool kStateOnly>
__global__ void __launch_bounds__(kWarps * 32, NP == 256 ? 1 : kWarps == 8 ? 2 : 3) chanrec_chunk_kernel(ChanrecParams a, ChanrecSegs sg) {
  using Sm = CrSmem<NP, kWarps>;
  constexpr int PT = Sm::PT, QS = Sm::QS, VS = Sm::VS, PS = Sm::PS, kThreads = kWarps * 32;
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  grid_dependency_wait();
  grid_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gr = lane >> 2, gc = lane & 3;
  const int ptiles = (a.p + PT - 1) / PT;
  const int per_seg = a.batch * a.heads * ptiles;
  const int seg = blockIdx.x / per_seg, item = blockIdx.x - seg * per_seg;
  const int pt = item % ptiles, bh = item / ptiles, b = bh / a.heads, h = bh - b * a.heads;
  const int tok0 = a.cu[b], ntok = a.cu[b + 1] - tok0;
  const int nchunks = (ntok + kCrTokens - 1) / kCrTokens;
  const int per = (kStateOnly ? sg.tokens / sg.pieces : sg.tokens) / kCrTokens, c0 = seg * per, c1 = min(nchunks, c0 + per);
  if (c0 >= c1) return;
  if (kStateOnly && (seg / sg.pieces + 1) * sg.tokens >= ntok) return;           // nobody starts from the end of the last segment
  const int pbase = pt * PT, p0 = warp * 16;              // this CTA's columns, this warp's columns within them
  const __nv_bfloat16* Q = (const __nv_bfloat16*)a.q + (int64_t)tok0 * a.row_stride + (int64_t)h * a.n;
  const __nv_bfloat16* F = (const __nv_bfloat16*)a.f + (int64_t)tok0 * a.row_stride + (int64_t)h * a.n;
  const __nv_bfloat16* V = (const __nv_bfloat16*)a.v + (int64_t)tok0 * a.row_stride + (int64_t)h * a.p + pbase;
  const float *bias = a.f_bias + (int64_t)h * a.n, *lower = a.lower + (int64_t)h * a.n;

  // This thread's pieces of a chunk: rows fr0 + i * (kThreads / pieces of a row), one column.
  constexpr int kQPieces = NP / 8, kVPieces = PT / 8, kQStep = kThreads / kQPieces, kVStep = kThreads / kVPieces;
  const int qr = tid / kQPieces, qc = (tid - qr * kQPieces) * 8, vr = tid / kVPieces, vc = (tid - vr * kVPieces) * 8;
  const bool q_in = qc < a.n, v_in = pbase + vc < a.p;
  auto fetch = [&](int chunk) {
    const int st = chunk & 1, t0 = chunk * kCrTokens;
    const int64_t at = (int64_t)(t0 + qr) * a.row_stride + qc;
#pragma unroll
    for (int i = 0; i < kCrTokens / kQStep; ++i) {
      const int r = qr + i * kQStep;
      const bool live = q_in && t0 + r < ntok;
      const int64_t from = live ? at + (int64_t)(i * kQStep) * a.row_stride : 0;
      if (!kStateOnly) cr_cp16(&sm.zq[st][r * QS + qc], Q + from, live);
      cr_cp16(&sm.zf[st][r * QS + qc], F + from, live);
    }
    const __nv_bfloat16* from_v = V + (int64_t)(t0 + vr) * a.row_stride + vc;
#pragma unroll
    for (int i = 0; i < kCrTokens / kVStep; ++i) {
      const int r = vr + i * kVStep;
      const bool live = v_in && t0 + r < ntok;
      cr_cp16(&sm.v[st][r * VS + vc], live ? from_v + (int64_t)(i * kVStep) * a.row_stride : V, live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // ---- state: S^T rows p0 + gr (+ 8), columns 8 nt + 2 gc (+ 1)
  float s[NP / 8][4];
  const int pc0 = pbase + p0 + gr, pc1 = pc0 + 8;
  const int64_t np = (int64_t)a.n * a.p;
  float* const final_state = a.state + ((int64_t)a.slots[b] * a.heads + h) * np;
  {
    const float* S = kStateOnly ? nullptr : sg.count > 1 ? sg.start + ((int64_t)bh * sg.count + seg) * sg.pieces * np : a.pos0[b] == 0 ? nullptr : final_state;
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + 2 * gc + (e & 1), p = e < 2 ? pc0 : pc1;
        s[nt][e] = (S != nullptr && n < a.n && p < a.p) ? S[(int64_t)n * a.p + p] : 0.f;
      }
  }
  constexpr int kOwn = (NP + kThreads - 1) / kThreads;
  float seg_decay[kOwn];                                  // of channels tid, tid + kThreads, ..
#pragma unroll
  for (int i = 0; i < kOwn; ++i) seg_decay[i] = 1.0f;

  // S += V^T k of 16 tokens, both parts of k
  auto add_keys = [&](const uint32_t* vf, int first) {
    const int krow = (first + ((lane >> 3) & 1) * 8 + (lane & 7)) * QS + ((lane >> 4) & 1) * 8;
#pragma unroll
    for (int n = 0; n < NP / 16; ++n) {
      uint32_t bf[4];
      cr_ldmt(bf, sm.k_hi + krow + n * 16);
      cr_mma(s[2 * n], vf, bf[0], bf[1]);
      cr_mma(s[2 * n + 1], vf, bf[2], bf[3]);
      cr_ldmt(bf, sm.k_lo + krow + n * 16);
      cr_mma(s[2 * n], vf, bf[0], bf[1]);
      cr_mma(s[2 * n + 1], vf, bf[2], bf[3]);
    }
  };
  auto rescale = [&](const float* by) {
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt) {
      const float2 d = *reinterpret_cast<const float2*>(by + nt * 8 + 2 * gc);
      const float2 x = mul2(make_float2(s[nt][0], s[nt][1]), d), y = mul2(make_float2(s[nt][2], s[nt][3]), d);
      s[nt][0] = x.x; s[nt][1] = x.y; s[nt][2] = y.x; s[nt][3] = y.y;
    }
  };
  if (tid < 2) sm.level[tid] = 0;
  fetch(c0);
  for (int chunk = c0; chunk < c1; ++chunk) {
    const int st = chunk & 1, t0 = chunk * kCrTokens;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // this chunk is here; everyone is done with the last one
    if (chunk + 1 < c1) fetch(chunk + 1);
    // ---- gates and scaled vectors: a thread walks two channels of eight tokens, four warps take 64 channels
    constexpr int kRounds = (NP + kWarps * 16 - 1) / (kWarps * 16);
    float2 P[kRounds][8], kp[kRounds][8];                  // product up to a token, k over it
    const int oct = warp & 3, r0 = oct * 8;
#pragma unroll
    for (int rd = 0; rd < kRounds; ++rd) {
      const int c = rd * kWarps * 16 + (warp >> 2) * 64 + 2 * lane;
      if (c >= NP) continue;
      // a channel that does not exist keeps its (zero) state: lower bound 1
      const float2 bi = c < a.n ? mul2(*reinterpret_cast<const float2*>(bias + c), pair(kMinusLog2e)) : pair(0.f);
      const float2 lo = c < a.n ? *reinterpret_cast<const float2*>(lower + c) : pair(1.f);
      const float2 rest = make_float2(1.0f - lo.x, 1.0f - lo.y);
      float2 inv = pair(1.0f);
      auto walk8 = [&](int live) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const uint32_t z = *reinterpret_cast<const uint32_t*>(&sm.zf[st][(r0 + j) * QS + c]);
          const float2 y = fma2(make_float2(__uint_as_float(z << 16), __uint_as_float(z & 0xffff0000u)), pair(kMinusLog2e), bi);
          float2 f, fi, k;
          if (kStateOnly) cr_gate(y, lo, rest, &f, &k);
          else cr_gate(y, lo, rest, &f, &fi, &k);
          if (j >= live) { f = pair(1.0f); fi = f; k = pair(0.0f); }
          if (kStateOnly) {
            P[rd][j] = f;
            kp[rd][j] = k;
            inv = mul2(inv, f);
          } else {
            P[rd][j] = j > 0 ? mul2(P[rd][j - 1], f) : f;
            inv = mul2(inv, fi);
            kp[rd][j] = mul2(k, inv);
          }
        }
      };
      if (t0 + kCrTokens <= ntok) walk8(8);
      else walk8(ntok - t0 - r0);
      if (kStateOnly) {
        *reinterpret_cast<float2*>(&sm.oct[0][oct][c]) = inv;
      } else {
        *reinterpret_cast<float2*>(&sm.oct[0][oct][c]) = P[rd][7];
        *reinterpret_cast<float2*>(&sm.oct[1][oct][c]) = inv;
        if (!(P[rd][7].x >= kWide && P[rd][7].y >= kWide)) // not a number counts as below
          atomicMax(&sm.level[st], P[rd][7].x >= kNarrow && P[rd][7].y >= kNarrow ? 1 : 2);
      }
    }
    __syncthreads();
    if constexpr (kStateOnly) {
      // ---- k_j times the gates after it; the state moves on by the whole chunk
#pragma unroll
      for (int rd = 0; rd < kRounds; ++rd) {
        const int c = rd * kWarps * 16 + (warp >> 2) * 64 + 2 * lane;
        if (c >= NP) continue;
        float2 after = pair(1.0f);
        for (int q = oct + 1; q < 4; ++q) after = mul2(after, *reinterpret_cast<const float2*>(&sm.oct[0][q][c]));
#pragma unroll
        for (int j = 7; j >= 0; --j) {
          uint32_t hi, lo_;
          cr_split(mul2(kp[rd][j], after), &hi, &lo_);
          *reinterpret_cast<uint32_t*>(&sm.k_hi[(r0 + j) * QS + c]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.k_lo[(r0 + j) * QS + c]) = lo_;
          after = mul2(after, P[rd][j]);
        }
        if (oct == 0) *reinterpret_cast<float2*>(&sm.end[0][c]) = after;
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < kOwn; ++i) {
        const int c = tid + i * kThreads;
        if (c < NP) seg_decay[i] *= sm.end[0][c];
      }
      rescale(sm.end[0]);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        uint32_t vf[4];
        cr_ldmt(vf, sm.v[st] + (i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * VS + p0 + ((lane >> 3) & 1) * 8);
        add_keys(vf, i * 16);
      }
      continue;
    }
    const int level = sm.level[st];
    if (tid == 0) sm.level[st ^ 1] = 0;
    if (level < 2) {
#pragma unroll
      for (int rd = 0; rd < kRounds; ++rd) {
        const int c = rd * kWarps * 16 + (warp >> 2) * 64 + 2 * lane;
        if (c >= NP) continue;
        float2 p0 = pair(1.0f), i0 = p0;                   // products of the block's tokens before this thread's
        for (int q = level == 0 ? 0 : oct & 2; q < oct; ++q) {
          p0 = mul2(p0, *reinterpret_cast<const float2*>(&sm.oct[0][q][c]));
          i0 = mul2(i0, *reinterpret_cast<const float2*>(&sm.oct[1][q][c]));
        }
        if (oct == 3 || (level == 1 && oct == 1)) *reinterpret_cast<float2*>(&sm.end[level == 0 ? 0 : oct >> 1][c]) = mul2(p0, P[rd][7]);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int at = (r0 + j) * QS + c;
          uint32_t hi, lo_;
          cr_split(mul2(kp[rd][j], i0), &hi, &lo_);
          *reinterpret_cast<uint32_t*>(&sm.k_hi[at]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.k_lo[at]) = lo_;
          const uint32_t z = *reinterpret_cast<const uint32_t*>(&sm.zq[st][at]);
          const float2 x = mul2(cr_silu2(make_float2(__uint_as_float(z << 16), __uint_as_float(z & 0xffff0000u))), mul2(P[rd][j], p0));
          *reinterpret_cast<__nv_bfloat162*>(&sm.q[at]) = __floats2bfloat162_rn(x.x, x.y);
        }
      }
      __syncthreads();
    }
    __nv_bfloat16* v_s = sm.v[st];
    // ---- kTiles groups of 16 tokens from token `first` on, as one block
    auto block = [&](auto tiles, int first, const float* end) {
      constexpr int kTiles = decltype(tiles)::value;
      uint32_t vf[kTiles][4];                              // V^T of this warp's columns, as A fragments
#pragma unroll
      for (int i = 0; i < kTiles; ++i)
        cr_ldmt(vf[i], v_s + (first + i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * VS + p0 + ((lane >> 3) & 1) * 8);
      float o[2 * kTiles][4] = {};
      const int qrow = (first + ((lane >> 4) & 1) * 8 + (lane & 7)) * QS + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {
        uint32_t hi[4], lo[4];
        cr_split(make_float2(s[2 * kk][0], s[2 * kk][1]), &hi[0], &lo[0]);
        cr_split(make_float2(s[2 * kk][2], s[2 * kk][3]), &hi[1], &lo[1]);
        cr_split(make_float2(s[2 * kk + 1][0], s[2 * kk + 1][1]), &hi[2], &lo[2]);
        cr_split(make_float2(s[2 * kk + 1][2], s[2 * kk + 1][3]), &hi[3], &lo[3]);
#pragma unroll
        for (int i = 0; i < kTiles; ++i) {
          uint32_t bf[4];
          cr_ldm(bf, sm.q + qrow + i * 16 * QS + kk * 16);
          cr_mma(o[2 * i], hi, bf[0], bf[1]);
          cr_mma(o[2 * i + 1], hi, bf[2], bf[3]);
          cr_mma(o[2 * i], lo, bf[0], bf[1]);
          cr_mma(o[2 * i + 1], lo, bf[2], bf[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < kTiles; ++i)
#pragma unroll
        for (int j = 0; j <= i; ++j) {
          uint32_t bf[4];
          const int at = (first + i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * PS + first + j * 16 + ((lane >> 3) & 1) * 8;
          cr_ldm(bf, sm.a_hi + at);
          cr_mma(o[2 * i], vf[j], bf[0], bf[1]);
          cr_mma(o[2 * i + 1], vf[j], bf[2], bf[3]);
          cr_ldm(bf, sm.a_lo + at);
          cr_mma(o[2 * i], vf[j], bf[0], bf[1]);
          cr_mma(o[2 * i + 1], vf[j], bf[2], bf[3]);
        }
      __syncwarp();
      // over this warp's own columns of the V tile (nobody else reads them), 16 tokens x 16 columns at a time
#pragma unroll
      for (int i = 0; i < kTiles; ++i) {
        uint32_t w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const __nv_bfloat162 x = __floats2bfloat162_rn(o[2 * i + (e >> 1)][2 * (e & 1)], o[2 * i + (e >> 1)][2 * (e & 1) + 1]);
          w[e] = *reinterpret_cast<const uint32_t*>(&x);
        }
        // fragments: tokens 0 .. 7 of columns 0 .. 7 and 8 .. 15, then tokens 8 .. 15
        cr_stmt(v_s + (first + i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * VS + p0 + ((lane >> 3) & 1) * 8, w);
      }
#pragma unroll
      for (int i = 0; i < kTiles; ++i) add_keys(vf[i], first + i * 16);
      rescale(end);
    };
    if (level < 2) {
      // ---- the blocks a: a task is 16 tokens against 8; the last two cross the middle (one block of 32 only)
      for (int task = warp; task < (level == 0 ? 6 : 4); task += kWarps) {
        const int ib = task < 4 ? task >> 1 : 1, jb = task < 4 ? ib : 0, j0 = jb * 16 + (task & 1) * 8;
        float sc[2][4] = {};
#pragma unroll 4
        for (int kk = 0; kk < NP / 16; ++kk) {
          uint32_t aq[4];
          cr_ldm(aq, sm.q + (ib * 16 + (lane & 15)) * QS + kk * 16 + (lane >> 4) * 8);
          const int at = (j0 + gr) * QS + kk * 16 + 2 * gc;
          const uint32_t* kh = reinterpret_cast<const uint32_t*>(sm.k_hi + at);
          const uint32_t* kl = reinterpret_cast<const uint32_t*>(sm.k_lo + at);
          cr_mma(sc[0], aq, kh[0], kh[4]);
          cr_mma(sc[1], aq, kl[0], kl[4]);
        }
        const int j = j0 + 2 * gc;
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int i = ib * 16 + gr + (e >> 1) * 8;
          uint32_t hi, lo;
          cr_split(make_float2(j <= i ? sc[0][e] + sc[1][e] : 0.f, j + 1 <= i ? sc[0][e + 1] + sc[1][e + 1] : 0.f), &hi, &lo);
          *reinterpret_cast<uint32_t*>(sm.a_hi + i * PS + j) = hi;
          *reinterpret_cast<uint32_t*>(sm.a_lo + i * PS + j) = lo;
        }
      }
      __syncthreads();
      if (level == 0) {
        block(std::integral_constant<int, 2>{}, 0, sm.end[0]);
      } else {
        block(std::integral_constant<int, 1>{}, 0, sm.end[0]);
        block(std::integral_constant<int, 1>{}, 16, sm.end[1]);
      }
    } else {
      // ---- token by token
      const int live_tokens = min(kCrTokens, ntok - t0);
      for (int r = 0; r < live_tokens; ++r) {
        float (*g)[NP] = sm.gate[r & 1];
#pragma unroll
        for (int i = 0; i < kOwn; ++i) {
          const int c = tid + i * kThreads;
          if (c >= NP) continue;
          const bool ch = c < a.n;
          float pos, neg;
          cr_sigmoid(__bfloat162float(sm.zf[st][r * QS + c]) + (ch ? bias[c] : 0.f), &pos, &neg);
          const float lo = ch ? lower[c] : 1.0f;
          g[1][c] = fmaf(1.0f - lo, pos, lo);
          g[2][c] = (1.0f - lo) * neg;
          g[0][c] = cr_silu(__bfloat162float(sm.zq[st][r * QS + c]));
        }
        __syncthreads();                                   // two buffers: one barrier per token
        const float v0 = __bfloat162float(v_s[r * VS + p0 + gr]), v1 = __bfloat162float(v_s[r * VS + p0 + gr + 8]);
        float o0 = 0.f, o1 = 0.f;
#pragma unroll
        for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int n = nt * 8 + 2 * gc + e;
            const float f = g[1][n], k = g[2][n];
            s[nt][e] = fmaf(f, s[nt][e], k * v0);
            s[nt][2 + e] = fmaf(f, s[nt][2 + e], k * v1);
            o0 = fmaf(g[0][n], s[nt][e], o0);
            o1 = fmaf(g[0][n], s[nt][2 + e], o1);
          }
#pragma unroll
        for (int d = 1; d <= 2; d <<= 1) {
          o0 += __shfl_xor_sync(0xffffffffu, o0, d);
          o1 += __shfl_xor_sync(0xffffffffu, o1, d);
        }
        __syncwarp();
        if (gc == 0) {
          v_s[r * VS + p0 + gr] = __float2bfloat16_rn(o0);
          v_s[r * VS + p0 + gr + 8] = __float2bfloat16_rn(o1);
        }
      }
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < kCrTokens / 16; ++i) {
      const int r = i * 16 + (lane >> 1), col = p0 + (lane & 1) * 8;
      if (t0 + r < ntok && pbase + col < a.p)
        st16((__nv_bfloat16*)a.out + ((int64_t)(tok0 + t0 + r) * a.heads + h) * a.p + pbase + col, ld16(v_s + r * VS + col));
    }
  }
  float* dst = kStateOnly ? sg.start + ((int64_t)bh * sg.count * sg.pieces + seg) * np : (c1 == nchunks ? final_state : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + 2 * gc + (e & 1), p = e < 2 ? pc0 : pc1;
        if (n < a.n && p < a.p) dst[(int64_t)n * a.p + p] = s[nt][e];
      }
  }
  if (kStateOnly && pt == 0) {
#pragma unroll
    for (int i = 0; i < kOwn; ++i) {
      const int c = tid + i * kThreads;
      if (c < a.n) sg.decay[((int64_t)bh * sg.count * sg.pieces + seg) * a.n + c] = seg_decay[i];
    }
  }
}

// start[first piece of a segment] <- state before the segment.  Thread per state element; on entry every piece of the segments
// before the last holds its own state.
__global__ void __launch_bounds__(256) chanrec_chain_kernel(ChanrecParams a, ChanrecSegs sg) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int bh = blockIdx.y, b = bh / a.heads, h = bh - b * a.heads;
  const int64_t np = (int64_t)a.n * a.p, i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= np) return;
  const int n = (int)(i / a.p);
  const int used = (a.cu[b + 1] - a.cu[b] - 1) / sg.tokens * sg.pieces + 1, all = sg.count * sg.pieces;
  float run = a.pos0[b] == 0 ? 0.f : a.state[((int64_t)a.slots[b] * a.heads + h) * np + i];
  float* at = sg.start + (int64_t)bh * all * np + i;
  const float* decay = sg.decay + (int64_t)bh * all * a.n + n;
  constexpr int kAhead = 8;                               // pieces requested before the first is used
  for (int k0 = 0; k0 < used; k0 += kAhead) {
    float own[kAhead], f[kAhead];
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      const bool more = k0 + k + 1 < used;
      own[k] = more ? at[(int64_t)(k0 + k) * np] : 0.f;
      f[k] = more ? decay[(int64_t)(k0 + k) * a.n] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < kAhead; ++k)
      if (k0 + k < used) {
        if ((k0 + k) % sg.pieces == 0) at[(int64_t)(k0 + k) * np] = run;
        run = fmaf(f[k], run, own[k]);
      }
  }
}

int launch_chanrec_chain(const ChanrecParams& a, const ChanrecSegs& sg, cudaStream_t st) {
  cudaError_t e = launch_pdl(chanrec_chain_kernel, dim3((unsigned)(((int64_t)a.n * a.p + 255) / 256), a.batch * a.heads), dim3(256), 0, st, a, sg);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_chunk: %s", cudaGetErrorString(e));
  return TKV_OK;
}

static bool chanrec_chunk_shape(int n, int p) { return n % 8 == 0 && p % 8 == 0 && n <= 256; }
static int chanrec_columns(int n, int p) { return (n <= 128 && p > 64) ? 128 : 64; }

static ChanrecSegs plan_chanrec(int batch, int max_tokens, int heads, int n, int p) {
  const bool tc = chanrec_tc_shape(n, p, max_tokens);
  const int pt = tc ? chanrec_tc_columns() : chanrec_columns(n, p);
  const int64_t ctas = (int64_t)batch * heads * ((p + pt - 1) / pt);
  const int64_t room = 148 * (tc || n > 128 ? 1 : 2);      // CTAs that run at the same time
  const int chunks = (max_tokens + kCrTokens - 1) / kCrTokens;
  // segments of at least eight chunks, pieces of at least four: the fewest steps of a CTA, a step of the pass over states alone
  // (all segments but one) counting half, and a little for every piece's state that goes through memory
  auto waves = [&](int64_t n_ctas) { return (double)((n_ctas + room - 1) / room); };
  int segs = 1, pieces = 1;
  double best = waves(ctas);
  for (int k = 2; k <= chunks / 8 && ctas * (k - 1) < 2 * room; ++k)
    for (int m = 1; m <= 4 && chunks / (k * m) >= 4; ++m) {
      const double cost = waves(ctas * k) / k + 0.5 * waves(ctas * (k - 1) * m) / (k * m) + 0.003 * k * m;
      if (cost < best) { best = cost; segs = k; pieces = m; }
    }
  ChanrecSegs s = {};
  int per = (chunks + segs - 1) / segs;
  per = (per + pieces - 1) / pieces * pieces;
  s.tokens = per * kCrTokens;
  s.pieces = pieces;
  s.count = per > 0 ? (chunks + per - 1) / per : 1;
  return s;
}

template <int NP, int kWarps>
static int launch_chanrec(const ChanrecParams& a, const ChanrecSegs& sg, cudaStream_t st) {
  constexpr int kBytes = (int)sizeof(CrSmem<NP, kWarps>);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(chanrec_chunk_kernel<NP, kWarps, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chanrec_chunk_kernel<NP, kWarps, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_chunk: %s", cudaGetErrorString(e));
    configured = true;
  }
  const int64_t grid = (int64_t)a.batch * a.heads * ((a.p + kWarps * 16 - 1) / (kWarps * 16)) * sg.count, pieces = grid * sg.pieces;
  if (pieces > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_chunk: %lld blocks", (long long)grid);
  cudaError_t e = cudaSuccess;
  if (sg.count > 1) {
    e = launch_pdl(chanrec_chunk_kernel<NP, kWarps, true>, dim3((unsigned)pieces), dim3(kWarps * 32), (size_t)kBytes, st, a, sg);
    if (e == cudaSuccess) {
      int rc = launch_chanrec_chain(a, sg, st);
      if (rc != TKV_OK) return rc;
    }
  }
  if (e == cudaSuccess)
    e = launch_pdl(chanrec_chunk_kernel<NP, kWarps, false>, dim3((unsigned)grid), dim3(kWarps * 32), (size_t)kBytes, st, a, sg);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_chanrec_chunk: %s", cudaGetErrorString(e));
  return check_launch("tkv_chanrec_chunk");
}

}  // namespace tkv

using namespace tkv;

extern "C" int64_t tkv_chanrec_chunk_workspace_bytes(int batch, int max_tokens, int heads, int n, int vdim, int dtype) {
  if (dtype != TKV_BF16 || batch <= 0 || heads <= 0 || n <= 0 || vdim <= 0 || max_tokens <= 0 || !chanrec_chunk_shape(n, vdim)) return -1;
  const ChanrecSegs s = plan_chanrec(batch, max_tokens, heads, n, vdim);
  return s.count > 1 ? (int64_t)batch * heads * s.count * s.pieces * n * ((int64_t)vdim + 1) * (int64_t)sizeof(float) : 0;
}

extern "C" int tkv_chanrec_chunk(const void* q, const void* f, const void* v, int64_t row_stride, const float* f_bias,
                                 const float* lower, void* out, float* state, const int32_t* slots, const int32_t* cu_tokens,
                                 const int32_t* pos0, void* workspace, int64_t workspace_bytes, int batch, int max_tokens, int heads,
                                 int n, int vdim, int dtype, int32_t* status, tkv_stream_t stream) {
  if (!q || !f || !v || !f_bias || !lower || !out || !state || !slots || !cu_tokens || !pos0)
    return fail(TKV_ERR_ARG, "tkv_chanrec_chunk: NULL pointer argument");
  if (batch < 0 || max_tokens < 0 || heads <= 0 || n <= 0 || vdim <= 0 || row_stride < (int64_t)heads * n || row_stride < (int64_t)heads * vdim)
    return fail(TKV_ERR_ARG, "tkv_chanrec_chunk: bad sizes heads=%d n=%d vdim=%d", heads, n, vdim);
  if (dtype != TKV_BF16 || !chanrec_chunk_shape(n, vdim))
    return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_chunk: dtype=%d n=%d vdim=%d (bf16, n <= 256, multiples of 8; others: tkv_chanrec_scan)", dtype, n, vdim);
  if (row_stride % 8 || !aligned16(q) || !aligned16(f) || !aligned16(v) || !aligned16(out))
    return fail(TKV_ERR_ARG, "tkv_chanrec_chunk: rows must start on 16-byte boundaries");
  if (batch == 0 || max_tokens == 0) return TKV_OK;
  if ((int64_t)batch * heads > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_chanrec_chunk: batch * heads = %lld", (long long)batch * heads);
  const int64_t need = tkv_chanrec_chunk_workspace_bytes(batch, max_tokens, heads, n, vdim, dtype);
  if (need > 0 && (!workspace || workspace_bytes < need))
    return fail(TKV_ERR_ARG, "tkv_chanrec_chunk: workspace of %lld bytes, %lld needed", (long long)workspace_bytes, (long long)need);
  ChanrecParams a = {q, f, v, row_stride, f_bias, lower, out, state, slots, cu_tokens, pos0, batch, heads, n, vdim};
  ChanrecSegs s = plan_chanrec(batch, max_tokens, heads, n, vdim);
  s.start = (float*)workspace;
  s.decay = s.start + (s.count > 1 ? (int64_t)batch * heads * s.count * s.pieces * n * vdim : 0);
  cudaStream_t st = (cudaStream_t)stream;
  if (chanrec_tc_shape(n, vdim, max_tokens)) return launch_chanrec_tc(a, s, status, st);
  const bool wide = chanrec_columns(n, vdim) == 128;
  if (n <= 64) return wide ? launch_chanrec<64, 8>(a, s, st) : launch_chanrec<64, 4>(a, s, st);
  if (n <= 128) return wide ? launch_chanrec<128, 8>(a, s, st) : launch_chanrec<128, 4>(a, s, st);
  return launch_chanrec<256, 4>(a, s, st);
}
