// Chunked form of the scalar-decay linear recurrence for prompts, 16-bit operands with fp32 state.
//
// With L_i the running sum of log a inside a chunk of 64 tokens and S the state before it,
//   o_i = e^{L_i} S^T q_i + sum_{j <= i} (q_i . k_j) e^{L_i - L_j} s_j v_j + d v_i
//   S  <- e^{L_64} S + sum_j e^{L_64 - L_j} s_j k_j v_j^T .
// One CTA walks the chunks of one (request, head, block of 16 * kWarps value columns, segment of the sequence).  The state
// never leaves registers: a warp owns 16 columns of v and holds S^T [16 x n] as fp32 MMA accumulators, whose layout is also
// the A-operand layout of the read-out S^T q.  All products are transposed accordingly (rows = value columns):
//   scores   S_ij = Q K^T           the CTA's warps share the 64 x 64 block, weights applied in fp32, result in shared memory
//   O^T      = S^T Q^T, scaled, + V^T P^T
//   S^T      = e^{L_64} S^T + (w V)^T K
// fp32 factors (state, weights P, scaled values) enter the 16-bit products as a high and a low part, two MMAs each, so the
// recurrence keeps about 16 bits more than the operands' type; q, k, v themselves are 16-bit exactly.
// Where (request, head, column) blocks alone do not fill the GPU, the sequence is cut into segments: a first pass computes
// every segment's own state, a small kernel chains them, and the main pass starts each segment from its true state.
#include "tkv_linrec.cuh"
#include "tkv_tc.cuh"

namespace tkv {

constexpr int kCk = 64;                                   // tokens per chunk

__device__ __forceinline__ void lc_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lc_ldm(uint32_t* r, const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void lc_ldmt(uint32_t* r, const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void lc_cp16(void* dst, const void* src, bool live) {
  const int bytes = live ? 16 : 0;                        // 0: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
// x = hi + lo in bf16, two values at a time.
__device__ __forceinline__ void lc_split(float a, float b, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(*hi << 16), b - __uint_as_float(*hi & 0xffff0000u));
  *lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int NP, int kWarps> struct LcSmem {
  static constexpr int PT = kWarps * 16, QS = NP + 8, VS = PT + 8, PS = kCk + 8;
  __nv_bfloat16 q[2][kCk * QS], k[2][kCk * QS], v[2][kCk * VS];
  __nv_bfloat16 p_hi[kCk * PS], p_lo[kCk * PS];
  float l2[2][kCk], vs[2][kCk];                           // running log2 decay, value scale; by chunk parity
};

template <int NP, int kWarps, bool kStateOnly>
__global__ void __launch_bounds__(kWarps * 32) linrec_chunk_kernel(LinrecParams a, LinrecSegs sg) {
  using Sm = LcSmem<NP, kWarps>;
  constexpr int PT = Sm::PT, QS = Sm::QS, VS = Sm::VS, PS = Sm::PS, kThreads = kWarps * 32;
  extern __shared__ __align__(16) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  grid_dependency_wait();
  grid_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gr = lane >> 2, gc = lane & 3;
  const int ptiles = (a.p + PT - 1) / PT;
  const int per_seg = a.batch * a.heads * ptiles;
  const int seg = blockIdx.x / per_seg, item = blockIdx.x - seg * per_seg;
  const int pt = item % ptiles, bh = item / ptiles, b = bh / a.heads, h = bh - b * a.heads, g = h / (a.heads / a.groups);
  const int tok0 = a.cu[b], ntok = a.cu[b + 1] - tok0;
  const int nchunks_all = (ntok + kCk - 1) / kCk;
  const int per = sg.tokens / kCk, c0 = seg * per, c1 = min(nchunks_all, c0 + per);
  if (c0 >= c1) return;
  if (kStateOnly && c1 == nchunks_all) return;            // nobody starts from the end of the last segment
  const int pbase = pt * PT, p0 = warp * 16;              // this CTA's columns, this warp's columns within them
  const __nv_bfloat16* Q = (const __nv_bfloat16*)a.q + (int64_t)tok0 * a.q_stride + (int64_t)g * a.n;
  const __nv_bfloat16* K = (const __nv_bfloat16*)a.k + (int64_t)tok0 * a.k_stride + (int64_t)g * a.n;
  const __nv_bfloat16* V = (const __nv_bfloat16*)a.v + (int64_t)tok0 * a.v_stride + (int64_t)h * a.p + pbase;

  auto fetch = [&](int chunk) {
    const int st = chunk & 1, t0 = chunk * kCk;
    for (int i = tid; i < kCk * (NP / 8); i += kThreads) {
      const int r = i / (NP / 8), c = (i - r * (NP / 8)) * 8;
      const bool live = t0 + r < ntok && c < a.n;
      const int64_t t = live ? t0 + r : 0;
      const int cc = live ? c : 0;
      if (!kStateOnly) lc_cp16(&sm.q[st][r * QS + c], Q + t * a.q_stride + cc, live);
      lc_cp16(&sm.k[st][r * QS + c], K + t * a.k_stride + cc, live);
    }
    for (int i = tid; i < kCk * (PT / 8); i += kThreads) {
      const int r = i / (PT / 8), c = (i - r * (PT / 8)) * 8;
      const bool live = t0 + r < ntok && pbase + c < a.p;
      lc_cp16(&sm.v[st][r * VS + c], V + (live ? (int64_t)(t0 + r) * a.v_stride + c : 0), live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  constexpr float kLog2e = 1.4426950408889634f;
  auto decays = [&](int chunk) {                           // warp 0: running sum over the chunk, two tokens per lane
    const int st = chunk & 1, t = chunk * kCk + 2 * lane;
    float d0 = 0.f, d1 = 0.f, s0 = 0.f, s1 = 0.f;
    if (t < ntok) { d0 = a.log_decay ? a.log_decay[(int64_t)(tok0 + t) * a.heads + h] : a.head_log_decay[h];
                    s0 = a.v_scale ? a.v_scale[(int64_t)(tok0 + t) * a.heads + h] : 1.f; }
    if (t + 1 < ntok) { d1 = a.log_decay ? a.log_decay[(int64_t)(tok0 + t + 1) * a.heads + h] : a.head_log_decay[h];
                        s1 = a.v_scale ? a.v_scale[(int64_t)(tok0 + t + 1) * a.heads + h] : 1.f; }
    float sum = d0 + d1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += y;
    }
    sm.l2[st][2 * lane] = (sum - d1) * kLog2e;
    sm.l2[st][2 * lane + 1] = sum * kLog2e;
    sm.vs[st][2 * lane] = s0;
    sm.vs[st][2 * lane + 1] = s1;
  };

  // ---- state: S^T rows p0 + gr (+ 8), columns 8 nt + 2 gc (+ 1)
  float s[NP / 8][4];
  const int pc0 = pbase + p0 + gr, pc1 = pc0 + 8;
  auto state_at = [&](const float* S) {
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + 2 * gc + (e & 1), p = e < 2 ? pc0 : pc1;
        s[nt][e] = (S != nullptr && n < a.n && p < a.p) ? S[(int64_t)n * a.p + p] : 0.f;
      }
  };
  const int64_t np = (int64_t)a.n * a.p;
  float* const final_state = a.state + ((int64_t)a.slots[b] * a.heads + h) * np;
  if (kStateOnly) state_at(nullptr);
  else if (sg.count > 1) state_at(sg.start + ((int64_t)bh * sg.count + seg) * np);
  else state_at(a.pos0[b] == 0 ? nullptr : final_state);
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
  float seg_log = 0.f;

  fetch(c0);
  if (warp == 0) decays(c0);
  for (int chunk = c0; chunk < c1; ++chunk) {
    const int st = chunk & 1, t0 = chunk * kCk;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // this chunk is here; everyone is done with the other stage
    if (chunk + 1 < c1) {
      fetch(chunk + 1);
      if (warp == 0) decays(chunk + 1);
    }
    const float *l2 = sm.l2[st], *vs = sm.vs[st];
    const __nv_bfloat16 *qs = sm.q[st], *ks = sm.k[st];
    __nv_bfloat16* v_s = sm.v[st];
    if (!kStateOnly) {
      // ---- scores of a 16-token row block, causal tiles only; two warps share a row block when there are eight
      const int rb = warp & 3, tiles = 2 * rb + 2;
      const int jt0 = kWarps == 8 ? (warp >> 2) * (rb + 1) : 0, jt1 = kWarps == 8 ? jt0 + rb + 1 : tiles;
      float sc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[j][e] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < NP / 16; ++kk) {
        uint32_t af[4];
        lc_ldm(af, qs + (rb * 16 + (lane & 15)) * QS + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int jt = jt0 + j;
          if (jt < jt1) {
            const uint32_t* kp = reinterpret_cast<const uint32_t*>(ks + (jt * 8 + gr) * QS + kk * 16 + 2 * gc);
            lc_mma(sc[j], af, kp[0], kp[4]);
          }
        }
      }
      const int i0 = rb * 16 + gr;
      const float li0 = l2[i0], li1 = l2[i0 + 8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int jt = jt0 + j;
        if (jt < jt1) {
          const int jc = jt * 8 + 2 * gc;
          const float w0 = vs[jc], w1 = vs[jc + 1], lj0 = l2[jc], lj1 = l2[jc + 1];
          uint32_t hi, lo;
          lc_split(jc <= i0 ? sc[j][0] * exp2_weight(li0 - lj0) * w0 : 0.f, jc + 1 <= i0 ? sc[j][1] * exp2_weight(li0 - lj1) * w1 : 0.f, &hi, &lo);
          *reinterpret_cast<uint32_t*>(sm.p_hi + i0 * PS + jc) = hi;
          *reinterpret_cast<uint32_t*>(sm.p_lo + i0 * PS + jc) = lo;
          lc_split(jc <= i0 + 8 ? sc[j][2] * exp2_weight(li1 - lj0) * w0 : 0.f, jc + 1 <= i0 + 8 ? sc[j][3] * exp2_weight(li1 - lj1) * w1 : 0.f, &hi, &lo);
          *reinterpret_cast<uint32_t*>(sm.p_hi + (i0 + 8) * PS + jc) = hi;
          *reinterpret_cast<uint32_t*>(sm.p_lo + (i0 + 8) * PS + jc) = lo;
        }
      }
      __syncthreads();
    }
    uint32_t vf[4][4];                                     // V^T of this warp's columns, as A fragments per 16 tokens
#pragma unroll
    for (int k = 0; k < 4; ++k) lc_ldmt(vf[k], v_s + (k * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * VS + p0 + ((lane >> 3) & 1) * 8);
    if (!kStateOnly) {
      float o[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
#pragma unroll
      for (int kk = 0; kk < NP / 16; ++kk) {
        uint32_t hi[4], lo[4];
        lc_split(s[2 * kk][0], s[2 * kk][1], &hi[0], &lo[0]);
        lc_split(s[2 * kk][2], s[2 * kk][3], &hi[1], &lo[1]);
        lc_split(s[2 * kk + 1][0], s[2 * kk + 1][1], &hi[2], &lo[2]);
        lc_split(s[2 * kk + 1][2], s[2 * kk + 1][3], &hi[3], &lo[3]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {                      // 16 tokens: B fragments of two n8 tiles
          uint32_t bf[4];
          lc_ldm(bf, qs + (i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * QS + kk * 16 + ((lane >> 3) & 1) * 8);
          lc_mma(o[2 * i], hi, bf[0], bf[1]);
          lc_mma(o[2 * i + 1], hi, bf[2], bf[3]);
          lc_mma(o[2 * i], lo, bf[0], bf[1]);
          lc_mma(o[2 * i + 1], lo, bf[2], bf[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float e0 = exp2_weight(l2[i * 8 + 2 * gc]), e1 = exp2_weight(l2[i * 8 + 2 * gc + 1]);
        o[i][0] *= e0; o[i][1] *= e1; o[i][2] *= e0; o[i][3] *= e1;
      }
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int i = k; i < 4; ++i) {                      // tokens i * 16 .. + 15 see the tokens k * 16 .. of their past
          uint32_t bf[4];
          const int at = (i * 16 + ((lane >> 4) & 1) * 8 + (lane & 7)) * PS + k * 16 + ((lane >> 3) & 1) * 8;
          lc_ldm(bf, sm.p_hi + at);
          lc_mma(o[2 * i], vf[k], bf[0], bf[1]);
          lc_mma(o[2 * i + 1], vf[k], bf[2], bf[3]);
          lc_ldm(bf, sm.p_lo + at);
          lc_mma(o[2 * i], vf[k], bf[0], bf[1]);
          lc_mma(o[2 * i + 1], vf[k], bf[2], bf[3]);
        }
      __syncwarp();
      // ---- output: over this warp's own columns of the V tile (nobody else reads them), then out in 32-byte pieces
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          __nv_bfloat16* x = v_s + (i * 8 + 2 * gc + (e & 1)) * VS + p0 + gr + (e >> 1) * 8;
          *x = __float2bfloat16_rn(fmaf(skip, __bfloat162float(*x), o[i][e]));
        }
      __syncwarp();
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = i * 16 + (lane >> 1), col = p0 + (lane & 1) * 8;
        if (t0 + r < ntok && pbase + col < a.p)
          st16((__nv_bfloat16*)a.out + ((int64_t)(tok0 + t0 + r) * a.heads + h) * a.p + pbase + col, ld16(v_s + r * VS + col));
      }
    }
    // ---- state
    const float lend = l2[kCk - 1], ec = exp2_weight(lend);
    seg_log += lend;
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] *= ec;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int j = k * 16 + 2 * gc;
      const float w0 = exp2_weight(lend - l2[j]) * vs[j], w1 = exp2_weight(lend - l2[j + 1]) * vs[j + 1];
      const float w2 = exp2_weight(lend - l2[j + 8]) * vs[j + 8], w3 = exp2_weight(lend - l2[j + 9]) * vs[j + 9];
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) {                        // fragments 0, 1: tokens j, j + 1; fragments 2, 3: j + 8, j + 9
        const float x = __uint_as_float(vf[k][q] << 16), y = __uint_as_float(vf[k][q] & 0xffff0000u);
        lc_split(x * (q < 2 ? w0 : w2), y * (q < 2 ? w1 : w3), &hi[q], &lo[q]);
      }
#pragma unroll
      for (int n = 0; n < NP / 16; ++n) {
        uint32_t bf[4];
        lc_ldmt(bf, ks + (k * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * QS + n * 16 + ((lane >> 4) & 1) * 8);
        lc_mma(s[2 * n], hi, bf[0], bf[1]);
        lc_mma(s[2 * n + 1], hi, bf[2], bf[3]);
        lc_mma(s[2 * n], lo, bf[0], bf[1]);
        lc_mma(s[2 * n + 1], lo, bf[2], bf[3]);
      }
    }
  }
  float* dst = kStateOnly ? sg.start + ((int64_t)bh * sg.count + seg) * np : (c1 == nchunks_all ? final_state : nullptr);
  if (dst != nullptr) {
#pragma unroll
    for (int nt = 0; nt < NP / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = nt * 8 + 2 * gc + (e & 1), p = e < 2 ? pc0 : pc1;
        if (n < a.n && p < a.p) dst[(int64_t)n * a.p + p] = s[nt][e];
      }
  }
  if (kStateOnly && tid == 0 && pt == 0) sg.log_sum[(int64_t)bh * sg.count + seg] = seg_log;
}

// start[seg] <- state before the segment.  Thread per state element; on entry start[seg] holds the segment's own state.
__global__ void __launch_bounds__(256) linrec_chain_kernel(LinrecParams a, LinrecSegs sg) {
  grid_dependency_wait();
  grid_launch_dependents();
  const int bh = blockIdx.y, b = bh / a.heads, h = bh - b * a.heads;
  const int64_t np = (int64_t)a.n * a.p, i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (i >= np) return;
  const int used = (a.cu[b + 1] - a.cu[b] + sg.tokens - 1) / sg.tokens;
  float run = a.pos0[b] == 0 ? 0.f : a.state[((int64_t)a.slots[b] * a.heads + h) * np + i];
  float* at = sg.start + (int64_t)bh * sg.count * np + i;
  for (int k = 0; k < used; ++k) {
    const float own = k + 1 < used ? at[(int64_t)k * np] : 0.f;
    at[(int64_t)k * np] = run;
    if (k + 1 < used) run = fmaf(exp2f(sg.log_sum[(int64_t)bh * sg.count + k]), run, own);
  }
}

static bool chunk_shape(int n, int p) { return n % 8 == 0 && p % 8 == 0 && n <= 256; }

static LinrecSegs plan_segments(int batch, int max_tokens, int heads, int n, int p) {
  const int pt = (n <= 128 && p > 64) ? 128 : 64;
  const int64_t ctas = (int64_t)batch * heads * ((p + pt - 1) / pt);
  const int chunks = (max_tokens + kCk - 1) / kCk;
  int segs = 1;
  if (ctas < 148 && chunks >= 8) {                         // segments of at least four chunks
    segs = (int)((2 * 148 + ctas - 1) / ctas);
    if (segs > chunks / 4) segs = chunks / 4;
  }
  LinrecSegs s = {};
  const int per = segs > 0 ? (chunks + segs - 1) / segs : 1;
  s.tokens = per * kCk;
  s.count = per > 0 ? (chunks + per - 1) / per : 1;
  return s;
}

int launch_linrec_chain(const LinrecParams& a, const LinrecSegs& sg, cudaStream_t st) {
  cudaError_t e = launch_pdl(linrec_chain_kernel, dim3((unsigned)(((int64_t)a.n * a.p + 255) / 256), a.batch * a.heads), dim3(256), 0, st, a, sg);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk: %s", cudaGetErrorString(e));
  return TKV_OK;
}

template <int NP, int kWarps>
static int launch_chunk(const LinrecParams& a, const LinrecSegs& sg, cudaStream_t st) {
  constexpr int kBytes = (int)sizeof(LcSmem<NP, kWarps>);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(linrec_chunk_kernel<NP, kWarps, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(linrec_chunk_kernel<NP, kWarps, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, kBytes);
    if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk: %s", cudaGetErrorString(e));
    configured = true;
  }
  const int64_t per_seg = (int64_t)a.batch * a.heads * ((a.p + kWarps * 16 - 1) / (kWarps * 16));
  if (per_seg * sg.count > INT32_MAX) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_chunk: %lld blocks", (long long)per_seg * sg.count);
  cudaError_t e = cudaSuccess;
  if (sg.count > 1) {
    e = launch_pdl(linrec_chunk_kernel<NP, kWarps, true>, dim3((unsigned)(per_seg * sg.count)), dim3(kWarps * 32), (size_t)kBytes, st, a, sg);
    if (e == cudaSuccess) {
      int rc = launch_linrec_chain(a, sg, st);
      if (rc != TKV_OK) return rc;
    }
  }
  if (e == cudaSuccess)
    e = launch_pdl(linrec_chunk_kernel<NP, kWarps, false>, dim3((unsigned)(per_seg * sg.count)), dim3(kWarps * 32), (size_t)kBytes, st, a, sg);
  if (e != cudaSuccess) return fail(TKV_ERR_LAUNCH, "tkv_linrec_chunk: %s", cudaGetErrorString(e));
  return check_launch("tkv_linrec_chunk");
}

}  // namespace tkv

using namespace tkv;

namespace tkv {
static LinrecSegs plan(int batch, int max_tokens, int64_t tokens, int heads, int n, int vdim) {
  return linrec_tc_shape(n, vdim, max_tokens, tokens) ? linrec_tc_segments(batch, max_tokens, heads, vdim) : plan_segments(batch, max_tokens, heads, n, vdim);
}
}  // namespace tkv

extern "C" int64_t tkv_linrec_chunk_workspace_bytes(int batch, int max_tokens, int tokens, int heads, int n, int vdim, int dtype) {
  if (dtype != TKV_BF16 || !chunk_shape(n, vdim) || batch <= 0 || heads <= 0 || n <= 0 || vdim <= 0 || max_tokens <= 0) return -1;
  const LinrecSegs s = plan(batch, max_tokens, tokens, heads, n, vdim);
  return s.count > 1 ? (int64_t)batch * heads * s.count * ((int64_t)n * vdim + 1) * (int64_t)sizeof(float) : 0;
}

extern "C" int tkv_linrec_chunk(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride,
                                const float* log_decay, const float* head_log_decay, const float* v_scale, const float* skip,
                                void* out, float* state, const int32_t* slots, const int32_t* cu_tokens, const int32_t* pos0,
                                void* workspace, int64_t workspace_bytes, int batch, int max_tokens, int tokens, int heads,
                                int groups, int n, int vdim, int dtype, int32_t* status, tkv_stream_t stream) {
  if (!q || !k || !v || (!log_decay && !head_log_decay) || !out || !state || !slots || !cu_tokens || !pos0)
    return fail(TKV_ERR_ARG, "tkv_linrec_chunk: NULL pointer argument");
  if (batch < 0 || max_tokens < 0 || tokens < max_tokens || heads <= 0 || groups <= 0 || heads % groups || n <= 0 || vdim <= 0 ||
      q_stride < (int64_t)groups * n || k_stride < (int64_t)groups * n || v_stride < (int64_t)heads * vdim)
    return fail(TKV_ERR_ARG, "tkv_linrec_chunk: bad sizes");
  if (dtype != TKV_BF16 || !chunk_shape(n, vdim))
    return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_chunk: dtype=%d n=%d vdim=%d (bf16, n <= 256, multiples of 8; others: tkv_linrec_scan)", dtype, n, vdim);
  if (q_stride % 8 || k_stride % 8 || v_stride % 8 || !aligned16(q) || !aligned16(k) || !aligned16(v) || !aligned16(out))
    return fail(TKV_ERR_ARG, "tkv_linrec_chunk: rows must start on 16-byte boundaries");
  if (batch == 0 || max_tokens == 0) return TKV_OK;
  if ((int64_t)batch * heads > 65535) return fail(TKV_ERR_UNSUPPORTED, "tkv_linrec_chunk: batch * heads = %lld", (long long)batch * heads);
  const int64_t need = tkv_linrec_chunk_workspace_bytes(batch, max_tokens, tokens, heads, n, vdim, dtype);
  if (need > 0 && (!workspace || workspace_bytes < need))
    return fail(TKV_ERR_ARG, "tkv_linrec_chunk: workspace of %lld bytes, %lld needed", (long long)workspace_bytes, (long long)need);
  LinrecParams a = {q, q_stride, k, k_stride, v, v_stride, log_decay, nullptr, head_log_decay, v_scale, skip, out, state, slots,
                    cu_tokens, pos0, batch, heads, groups, n, vdim};
  LinrecSegs s = plan(batch, max_tokens, tokens, heads, n, vdim);
  s.start = (float*)workspace;
  s.log_sum = s.start + (s.count > 1 ? (int64_t)batch * heads * s.count * n * vdim : 0);
  cudaStream_t st = (cudaStream_t)stream;
  if (linrec_tc_shape(n, vdim, max_tokens, tokens)) return launch_linrec_tc(a, s, tokens, status, st);
  if (n <= 64) return vdim > 64 ? launch_chunk<64, 8>(a, s, st) : launch_chunk<64, 4>(a, s, st);
  if (n <= 128) return vdim > 64 ? launch_chunk<128, 8>(a, s, st) : launch_chunk<128, 4>(a, s, st);
  return launch_chunk<256, 4>(a, s, st);
}
