// Register-level pieces shared by the prompt kernels of the channel-decay recurrence.
#pragma once
#include "tkv_chanrec.cuh"
#include "tkv_tc.cuh"

namespace tkv {

__device__ __forceinline__ void cr_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cr_ldm(uint32_t* r, const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void cr_ldmt(uint32_t* r, const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void cr_stmt(__nv_bfloat16* p, const uint32_t* r) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};"
               ::"r"(smem_u32(p)), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]) : "memory");
}
__device__ __forceinline__ void cr_cp16(void* dst, const void* src, bool live) {
  const int bytes = live ? 16 : 0;                        // 0: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
// Two fp32 operations in one instruction.
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 r;
  asm("{\n\t.reg .b64 a, b, r;\n\tmov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tmul.rn.f32x2 r, a, b;\n\tmov.b64 {%0, %1}, r;\n\t}"
      : "=f"(r.x), "=f"(r.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return r;
}
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 r;
  asm("{\n\t.reg .b64 a, b, c, r;\n\tmov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tmov.b64 c, {%6, %7};\n\tfma.rn.f32x2 r, a, b, c;\n\t"
      "mov.b64 {%0, %1}, r;\n\t}"
      : "=f"(r.x), "=f"(r.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return r;
}
__device__ __forceinline__ float2 add2(float2 a, float2 b) {
  float2 r;
  asm("{\n\t.reg .b64 a, b, r;\n\tmov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tadd.rn.f32x2 r, a, b;\n\tmov.b64 {%0, %1}, r;\n\t}"
      : "=f"(r.x), "=f"(r.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return r;
}
constexpr float kMinusLog2e = -1.4426950408889634f;
__device__ __forceinline__ float2 pair(float x) { return make_float2(x, x); }
// x = hi + lo in bf16, two values at a time.
__device__ __forceinline__ void cr_split(float2 x, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x.x, x.y);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 r = fma2(make_float2(__uint_as_float(*hi << 16), __uint_as_float(*hi & 0xffff0000u)), pair(-1.0f), x);
  const __nv_bfloat162 l = __floats2bfloat162_rn(r.x, r.y);
  *lo = *reinterpret_cast<const uint32_t*>(&l);
}
// sigmoid(x) and sigmoid(-x), each to a few units in the last place of fp32.
__device__ __forceinline__ void cr_sigmoid(float x, float* pos, float* neg) {
  const float e = exp2_weight(fabsf(x) * -1.4426950408889634f), r = __frcp_rn(1.0f + e);
  const float small = e * r;
  *pos = x >= 0.f ? r : small;
  *neg = x >= 0.f ? small : r;
}

__device__ __forceinline__ float cr_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// f, 1 / f and k = 1 - f of two channels with one reciprocal each, from -x / ln 2 of the gate's argument x: with e = exp(-x),
// f = (lo (1 + e) + 1 - lo) / (1 + e) and k = (1 - lo) e / (1 + e).  e is held below 2^60 (sigmoid 1e-18), which only gates
// that send the chunk to the token-by-token path ever reach.
__device__ __forceinline__ void cr_gate(float2 y, float2 lo, float2 rest, float2* f, float2* inv, float2* k) {
  const float2 e = make_float2(exp2_weight(fminf(y.x, 60.0f)), exp2_weight(fminf(y.y, 60.0f)));
  const float2 den = add2(e, pair(1.0f)), num = fma2(lo, den, rest), dn = mul2(den, num);
  const float2 t = make_float2(cr_rcp(dn.x), cr_rcp(dn.y)), u = mul2(num, t);      // u = 1 / den
  *f = mul2(num, u);
  *inv = mul2(den, mul2(den, t));
  *k = mul2(mul2(rest, e), u);
}
// The same without 1 / f.
__device__ __forceinline__ void cr_gate(float2 y, float2 lo, float2 rest, float2* f, float2* k) {
  const float2 e = make_float2(exp2_weight(fminf(y.x, 60.0f)), exp2_weight(fminf(y.y, 60.0f)));
  const float2 den = add2(e, pair(1.0f)), t = make_float2(cr_rcp(den.x), cr_rcp(den.y));
  *f = mul2(fma2(lo, den, rest), t);
  *k = mul2(mul2(rest, e), t);
}
__device__ __forceinline__ float cr_silu(float z) { return z * cr_rcp(1.0f + exp2_weight(z * -1.4426950408889634f)); }
__device__ __forceinline__ float2 cr_silu2(float2 z) {
  const float2 y = mul2(z, pair(kMinusLog2e));
  const float2 d = add2(make_float2(exp2_weight(y.x), exp2_weight(y.y)), pair(1.0f));
  return mul2(z, make_float2(cr_rcp(d.x), cr_rcp(d.y)));
}

}  // namespace tkv
