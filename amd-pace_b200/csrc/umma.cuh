// tcgen05 (5th-generation tensor cores), tensor memory and tiled-TMA helpers shared by the kernels that use them.
#pragma once

#include <cuda.h>

#include <mutex>

#include "common.cuh"

namespace pace {

// ------------------------------- host side: tensor maps -------------------------------
typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                             const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                             CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeFn encode_fn() {
  static EncodeFn fn = nullptr;
  static std::once_flag once;
  std::call_once(once, [] {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) == cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeFn>(ptr);
  });
  return fn;
}

// bf16 tensor of `rank` dimensions, innermost first (strides in bytes, of dimensions 1 ..), 128-byte swizzle, zeros out of
// bounds
inline int tensor_map_bf16(CUtensorMap* tm, const void* base, int rank, const uint64_t* dims, const uint64_t* strides,
                           const uint32_t* box) {
  EncodeFn fn = encode_fn();
  if (!fn) {
    set_cuda_error(cudaErrorNotSupported, "cuTensorMapEncodeTiled entry point");
    return PACE_ERR_CUDA;
  }
  cuuint64_t d[5], st[5];
  cuuint32_t b[5], one[5] = {1, 1, 1, 1, 1};
  for (int i = 0; i < rank; ++i) {
    d[i] = dims[i];
    b[i] = box[i];
    if (i) st[i - 1] = strides[i - 1];
  }
  const CUresult r = fn(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void*>(base), d, st, b, one,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) {
    set_cuda_error(cudaErrorInvalidValue, "cuTensorMapEncodeTiled");
    return PACE_ERR_CUDA;
  }
  return PACE_OK;
}

#ifdef __CUDACC__
// ------------------------------- device side -------------------------------
constexpr int kUmmaRows = 128;          // rows of the A operand (UMMA M)
// high half of a shared-memory matrix descriptor: SBO 1024 B, version 1, 128-byte swizzle
constexpr uint32_t kDescHi = (1024u >> 4) | (1u << 14) | (2u << 29);

__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }

// shared-memory matrix descriptor, 128-byte swizzle (layout type 2), descriptor version 1
__device__ __forceinline__ uint64_t umma_desc(uint32_t smem_addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  const uint32_t lo = ((smem_addr >> 4) & 0x3FFFu) | (((lbo_bytes >> 4) & 0x3FFFu) << 16);
  const uint32_t hi = ((sbo_bytes >> 4) & 0x3FFFu) | (1u << 14) | (2u << 29);
  return ((uint64_t)hi << 32) | lo;
}
// instruction descriptor: bf16 x bf16 -> fp32, M = 128, A K-major
__host__ __device__ constexpr uint32_t umma_idesc(int n, bool b_mn_major) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((b_mn_major ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) |
         ((uint32_t)(kUmmaRows >> 4) << 24);
}
// the same with A M-major (its 64-element column blocks lie LBO apart)
__host__ __device__ constexpr uint32_t umma_idesc_at(int n) { return umma_idesc(n, false) | (1u << 15); }
__device__ __forceinline__ void umma_bf16(uint32_t tmem_d, uint64_t a_desc, uint64_t b_desc, uint32_t idesc,
                                          uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t}"
      :
      : "r"(tmem_d), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
// A operand in tensor memory (128 lanes x 8 columns of packed bf16 pairs per 16-wide k-step)
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t b_desc, uint32_t idesc,
                                             uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t}"
      :
      : "r"(tmem_d), "r"(tmem_a), "l"(b_desc), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
// Blackwell's two-wide fp32 arithmetic and three-input maximum: a row of 64 scores takes 32 instructions
// for the maximum, 32 for scale-and-shift and 32 for the row sum instead of 64 each - the softmax
// warps share their schedulers' issue slots with each other and the exp2 unit is the pipe to keep busy.
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// 2^x for two values at once on the FMA pipe (any x; below -126 the result is 2^-126): round to the
// nearest integer with the 1.5 * 2^23 trick, a degree-3 polynomial for 2^f on [-0.5, 0.5] (relative error
// 1e-4, a twentieth of the bf16 rounding of P) and the integer part added into the exponent field.
__device__ __forceinline__ void exp2_poly2(float x0, float x1, float& p0, float& p1) {
  const uint32_t kMagic = 0x4B400000u, kNegMagic = 0xCB400000u, kNegOne = 0xBF800000u;  // 1.5 * 2^23, -1.5 * 2^23, -1.0
  x0 = fmaxf(x0, -126.f);
  x1 = fmaxf(x1, -126.f);
  uint64_t x, r, f, q;
  asm("mov.b64 %0, {%1, %2};" : "=l"(x) : "r"(__float_as_uint(x0)), "r"(__float_as_uint(x1)));
  uint64_t magic, neg_magic, neg_one, c0, c1, c2, c3;
  asm("mov.b64 %0, {%1, %1};" : "=l"(magic) : "r"(kMagic));
  asm("mov.b64 %0, {%1, %1};" : "=l"(neg_magic) : "r"(kNegMagic));
  asm("mov.b64 %0, {%1, %1};" : "=l"(neg_one) : "r"(kNegOne));
  asm("mov.b64 %0, {%1, %1};" : "=l"(c0) : "r"(__float_as_uint(0.9999281764f)));
  asm("mov.b64 %0, {%1, %1};" : "=l"(c1) : "r"(__float_as_uint(0.6932609677f)));
  asm("mov.b64 %0, {%1, %1};" : "=l"(c2) : "r"(__float_as_uint(0.2426091731f)));
  asm("mov.b64 %0, {%1, %1};" : "=l"(c3) : "r"(__float_as_uint(0.05517086014f)));
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(x), "l"(magic));  // low mantissa bits: the rounded integer
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(f) : "l"(r), "l"(neg_magic));
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(f) : "l"(f), "l"(neg_one), "l"(x));  // x - round(x)
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(q) : "l"(c3), "l"(f), "l"(c2));
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(q) : "l"(q), "l"(f), "l"(c1));
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(q) : "l"(q), "l"(f), "l"(c0));
  uint32_t r0, r1, q0, q1;
  asm("mov.b64 {%0, %1}, %2;" : "=r"(r0), "=r"(r1) : "l"(r));
  asm("mov.b64 {%0, %1}, %2;" : "=r"(q0), "=r"(q1) : "l"(q));
  p0 = __uint_as_float(q0 + (r0 << 23));
  p1 = __uint_as_float(q1 + (r1 << 23));
}
// The same with a degree-5 polynomial (minimax for the relative error on [-0.5, 0.5], found with the Remez exchange:
// 7e-8, 2.4e-7 with fp32 arithmetic): weights that are split keep what this gives them.
__device__ __forceinline__ void exp2_poly2_fine(float x0, float x1, float& p0, float& p1) {
  x0 = fmaxf(x0, -126.f);
  x1 = fmaxf(x1, -126.f);
  uint64_t x, r, f, q;
  asm("mov.b64 %0, {%1, %2};" : "=l"(x) : "r"(__float_as_uint(x0)), "r"(__float_as_uint(x1)));
  auto both = [](float v) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "r"(__float_as_uint(v)));
    return d;
  };
  r = add2(x, both(12582912.0f));        // 1.5 * 2^23: the low mantissa bits are the rounded integer
  f = add2(r, both(-12582912.0f));
  f = fma2(f, both(-1.0f), x);           // x - round(x)
  q = fma2(both(0.0013276472632f), f, both(0.0096755413431f));
  q = fma2(q, f, both(0.0555071327186f));
  q = fma2(q, f, both(0.2402211972371f));
  q = fma2(q, f, both(0.6931469670651f));
  q = fma2(q, f, both(1.0000000716547f));
  uint32_t r0, r1, q0, q1;
  asm("mov.b64 {%0, %1}, %2;" : "=r"(r0), "=r"(r1) : "l"(r));
  asm("mov.b64 {%0, %1}, %2;" : "=r"(q0), "=r"(q1) : "l"(q));
  p0 = __uint_as_float(q0 + (r0 << 23));
  p1 = __uint_as_float(q1 + (r1 << 23));
}
__device__ __forceinline__ void unpack64(uint64_t v, uint32_t& lo, uint32_t& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=r"(lo), "=r"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t pack64(uint32_t lo, uint32_t hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "r"(lo), "r"(hi));
  return d;
}
// arrive on an mbarrier once every tcgen05.mma issued so far by this thread has completed
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
               : "memory");
}
// 32 TMEM lanes (this warp's) x 32 consecutive 32-bit columns -> 32 registers per thread
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr));
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]),
      "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]),
      "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr));
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
      "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tmem_st8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"r"(taddr), "r"(r[0]), "r"(r[1]),
               "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
__device__ __forceinline__ void tmem_ld2(uint32_t taddr, uint32_t& r0, uint32_t& r1) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x2.b32 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(taddr));
}
__device__ __forceinline__ void tmem_st2(uint32_t taddr, uint32_t r0, uint32_t r1) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x2.b32 [%0], {%1, %2};" ::"r"(taddr), "r"(r0), "r"(r1) : "memory");
}
__device__ __forceinline__ void tmem_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ bool elect_one() {
  uint32_t pred;
  asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(pred));
  return pred != 0;
}

constexpr unsigned kSoftmaxBackoffNs = 100;  // a waiting softmax warp leaves its scheduler's issue slots to the MMA issuer
// Bounded wait that also gives up when another role has raised the abort flag.  Called by whole
// warps; the answer is the same for every lane (the tcgen05 instructions that follow are .aligned).
__device__ __forceinline__ bool umma_wait(uint64_t* bar, uint32_t parity, volatile int* abort) {
  bool ok = false;
  for (int i = 0; i < (1 << 18); ++i) {
    if (mbar_try_wait(bar, parity)) {
      ok = true;
      break;
    }
    if (*abort) break;
    if (i >= 8) __nanosleep(i > 64 ? 256 : kSoftmaxBackoffNs);  // (the first probes back to back: most waits are nearly over)
  }
  if (!ok) *abort = 1;
  return __all_sync(0xffffffffu, ok);
}
// The same for an issuer warp: no sleeping between the probes (each of them may wait up to a microsecond).
__device__ __forceinline__ bool umma_issuer_wait(uint64_t* bar, uint32_t parity, volatile int* abort) {
  for (int k = 0; k < (1 << 20); ++k) {
    if (__all_sync(0xffffffffu, mbar_try_wait(bar, parity))) return true;
    if ((k & 15) == 15 && __any_sync(0xffffffffu, *abort != 0)) break;
  }
  *abort = 1;
  return false;
}
__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* tm, int c0, int c1, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(
          smem_u32(dst)),
      "l"(tm), "r"(smem_u32(bar)), "r"(c0), "r"(c1)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* tm, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];" ::"r"(
          smem_u32(dst)),
      "l"(tm), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
// the same box on its way into L2 only
__device__ __forceinline__ void tma_prefetch_3d(const CUtensorMap* tm, int c0, int c1, int c2) {
  asm volatile("cp.async.bulk.prefetch.tensor.3d.L2.global.tile [%0, {%1, %2, %3}];" ::"l"(tm), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
// four rows of a two-dimensional tensor, given by their numbers (the map's box is one row high)
__device__ __forceinline__ void tma_gather4(void* dst, const CUtensorMap* tm, int c0, int r0, int r1, int r2, int r3,
                                            uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cta.global.tile::gather4.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, "
      "%7}], [%2];" ::"r"(smem_u32(dst)),
      "l"(tm), "r"(smem_u32(bar)), "r"(c0), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
      : "memory");
}
#endif  // __CUDACC__

}  // namespace pace
