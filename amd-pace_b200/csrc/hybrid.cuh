// Helpers of the hybrid-decoder kernels (norms, general attention, recurrences): activations are bf16 or
// fp32 (template parameter T), everything else is fp32.
#pragma once

#include "common.cuh"

namespace pace {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
// a value as an activation of type T holds it
template <typename T> __device__ __forceinline__ float round_to(float v) { return to_f<T>(from_f<T>(v)); }

// N consecutive elements <-> fp32 registers; N is 1 or makes an 8- or 16-byte access the caller has aligned
template <typename T, int N> struct Vec;
template <> struct Vec<float, 1> {
  static __device__ __forceinline__ void load(const float* p, float* o) { o[0] = *p; }
  static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; }
};
template <> struct Vec<float, 2> {
  static __device__ __forceinline__ void load(const float* p, float* o) {
    const float2 t = *reinterpret_cast<const float2*>(p);
    o[0] = t.x; o[1] = t.y;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  }
};
template <> struct Vec<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float* o) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    o[0] = t.x; o[1] = t.y; o[2] = t.z; o[3] = t.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct Vec<float, 8> {
  static __device__ __forceinline__ void load(const float* p, float* o) {
    Vec<float, 4>::load(p, o);
    Vec<float, 4>::load(p + 4, o + 4);
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    Vec<float, 4>::store(p, v);
    Vec<float, 4>::store(p + 4, v + 4);
  }
};
template <> struct Vec<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* o) { o[0] = __bfloat162float(*p); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Vec<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* o) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf2_to_f2(t.x), b = bf2_to_f2(t.y);
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf2(v[0], v[1]), f2_to_bf2(v[2], v[3]));
  }
};
template <> struct Vec<__nv_bfloat16, 8> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* o) {
    const uint4 t = *reinterpret_cast<const uint4*>(p);
    const float2 a = bf2_to_f2(t.x), b = bf2_to_f2(t.y), c = bf2_to_f2(t.z), d = bf2_to_f2(t.w);
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y; o[4] = c.x; o[5] = c.y; o[6] = d.x; o[7] = d.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    *reinterpret_cast<uint4*>(p) =
        make_uint4(f2_to_bf2(v[0], v[1]), f2_to_bf2(v[2], v[3]), f2_to_bf2(v[4], v[5]), f2_to_bf2(v[6], v[7]));
  }
};

// fp32 with a few ulp of error.  T names the activation type of the caller: fp32 models take the library's
// exp and divide, bf16 models the hardware's approximate ones (relative error about 1e-6).
template <typename T> __device__ __forceinline__ float exp_t(float x) { return fast_exp2(x * kLog2e); }
template <> __device__ __forceinline__ float exp_t<float>(float x) { return expf(x); }
template <typename T> __device__ __forceinline__ float rcp_t(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
template <> __device__ __forceinline__ float rcp_t<float>(float x) { return 1.0f / x; }
// sigmoid(x) = 1 / (1 + e^-x)   (1 / infinity = 0 at the far end)
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) { return rcp_t<T>(1.0f + exp_t<T>(-x)); }
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }
// 0.5 z (1 + tanh w) = z sigmoid(2 w)
template <typename T> __device__ __forceinline__ float gelu_tanh_t(float z) {
  return z * sigmoid_t<T>(1.5957691216057308f * (z + 0.044715f * z * z * z));
}
__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.7071067811865476f)); }
// ln(1 + e^x), with a relative error of a few ulp at both ends
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// the same with the hardware's exponential and reciprocal: ln(1 + u) = 2 artanh(u / (2 + u)), whose argument is at most 1/3 (the
// first term left out is below 1e-8 of the sum)
__device__ __forceinline__ float softplus_fast(float x) {
  const float u = fast_exp2(-fabsf(x) * kLog2e);
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(2.0f + u));
  const float s = u * r, q = s * s;
  float p = fmaf(q, 1.0f / 13, 1.0f / 11);
  p = fmaf(p, q, 1.0f / 9);
  p = fmaf(p, q, 1.0f / 7);
  p = fmaf(p, q, 1.0f / 5);
  p = fmaf(p, q, 1.0f / 3);
  p = fmaf(p, q, 1.0f);
  return fmaf(2.0f * s, p, fmaxf(x, 0.f));
}
template <typename T> __device__ __forceinline__ float softplus_t(float x) { return softplus_fast(x); }
template <> __device__ __forceinline__ float softplus_t<float>(float x) { return softplus(x); }
template <typename T> __device__ __forceinline__ float act_t(int act, float z) {
  return act == PACE_ACT_SILU ? silu_t<T>(z) : act == PACE_ACT_GELU_TANH ? gelu_tanh_t<T>(z) : act == PACE_ACT_GELU_ERF ? gelu_erf(z) : z;
}
// sqrt(1 - e^x) for x <= 0 (exp_x = e^x) without cancellation: near zero 1 - e^x is the Taylor series
// -x (1 + x/2 (1 + x/3 (1 + ...))), further out the plain difference
template <typename T> __device__ __forceinline__ float sqrt_one_minus_exp(float x, float exp_x) {
  // |x| < 1/16: the first term left out, x^4 / 120, is below 2e-7; the difference has lost four bits at most
  const float s = -x * fmaf(x * (1.0f / 2), fmaf(x * (1.0f / 3), fmaf(x, 1.0f / 4, 1.0f), 1.0f), 1.0f);
  float r;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x > -0.0625f ? s : 1.0f - exp_x));
  return r;
}
template <> __device__ __forceinline__ float sqrt_one_minus_exp<float>(float x, float exp_x) {
  const float s = -x * (1.0f + x * (1.0f / 2) * (1.0f + x * (1.0f / 3) * (1.0f + x * (1.0f / 4) *
                  (1.0f + x * (1.0f / 5) * (1.0f + x * (1.0f / 6) * (1.0f + x * (1.0f / 7)))))));
  return sqrtf(x > -0.25f ? s : 1.0f - exp_x);
}

// Sum over the thread block, the same value in every thread; `red` holds one float per warp.
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int warps = (blockDim.x + 31) >> 5;
  if (warps == 1) return v;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < warps; ++w) s += red[w];
  return s;
}

// One channel of a short convolution for the one new token of a sequence: its inputs are asked for by load() and used by sum().
// NT: taps where known at compile time, else 0 (the inputs are then fetched by sum()).
template <typename T, int NT> struct ConvNow {
  float now, x[NT ? NT : 1], w[NT ? NT : 1], bias;
  __device__ __forceinline__ void load(const T* row, const float* ring, int ring_rows, int64_t ring_stride, const float* taps, int channels,
                                       int n_taps, const float* b, int pos, int ch) {
    now = to_f<T>(row[ch]);
    bias = b ? b[ch] : 0.f;
    if constexpr (NT > 0) {
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        w[j] = taps[(size_t)j * channels + ch];
        if (j < NT - 1) x[j] = pos >= NT - 1 - j ? ring[(size_t)((pos - (NT - 1 - j)) % ring_rows) * ring_stride + ch] : 0.f;
      }
    }
  }
  __device__ __forceinline__ float sum(const float* ring, int ring_rows, int64_t ring_stride, const float* taps, int channels, int n_taps,
                                       int pos, int ch) const {
    float acc = bias;
    if constexpr (NT > 0) {
#pragma unroll
      for (int j = 0; j < NT; ++j) acc = fmaf(w[j], j < NT - 1 ? x[j] : now, acc);
    } else {
      for (int j = 0; j < n_taps; ++j) {
        const int back = n_taps - 1 - j;
        if (back > pos) continue;
        acc = fmaf(taps[(size_t)j * channels + ch], back ? ring[(size_t)((pos - back) % ring_rows) * ring_stride + ch] : now, acc);
      }
    }
    return acc;
  }
};

inline bool step_ok(const pace_step_t* s) {
  return s && s->n_tokens >= 0 && s->n_entries >= 0 && s->n_tokens >= s->n_entries &&
         (s->n_tokens == 0 || (s->token && s->tok_entry && s->tok_pos && s->q_row && s->cu && s->start && s->slot));
}
inline bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace pace
