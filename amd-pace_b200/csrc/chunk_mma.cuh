// Helpers of recurrences in chunks on mma.sync: products of operands in two bf16 terms, copies, the two-wide softplus.
#pragma once

#include "hybrid.cuh"
#include "umma.cuh"

namespace pace {

#ifdef __CUDACC__
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (hi + lo) x (hi + lo) without the last term
__device__ __forceinline__ void mma_split(float* c, const uint32_t* ah, const uint32_t* al, const uint32_t* bh, const uint32_t* bl) {
  mma16816(c, ah, bh[0], bh[1]);
  mma16816(c, ah, bl[0], bl[1]);
  mma16816(c, al, bh[0], bh[1]);
}
__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void copy16(void* dst, const void* src, bool live = true) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}

__device__ __forceinline__ uint64_t both(float v) { return pack64(__float_as_uint(v), __float_as_uint(v)); }
// softplus_fast of two values, two-wide
__device__ __forceinline__ uint64_t softplus2(float x0, float x1) {
  const float u0 = fast_exp2(-fabsf(x0) * kLog2e), u1 = fast_exp2(-fabsf(x1) * kLog2e);
  const uint64_t u = pack64(__float_as_uint(u0), __float_as_uint(u1));
  uint32_t d0, d1;
  unpack64(add2(u, both(2.0f)), d0, d1);
  const float r0 = rcp_t<__nv_bfloat16>(__uint_as_float(d0)), r1 = rcp_t<__nv_bfloat16>(__uint_as_float(d1));
  const uint64_t s = fma2(u, pack64(__float_as_uint(r0), __float_as_uint(r1)), 0ull), q = fma2(s, s, 0ull);
  uint64_t p = fma2(q, both(1.0f / 13), both(1.0f / 11));
  p = fma2(p, q, both(1.0f / 9));
  p = fma2(p, q, both(1.0f / 7));
  p = fma2(p, q, both(1.0f / 5));
  p = fma2(p, q, both(1.0f / 3));
  p = fma2(p, q, both(1.0f));
  return fma2(add2(s, s), p, pack64(__float_as_uint(fmaxf(x0, 0.f)), __float_as_uint(fmaxf(x1, 0.f))));
}
#endif  // __CUDACC__

}  // namespace pace
