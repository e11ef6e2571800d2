// Which keys a query sees: plain causality, a sliding window or chunks counted from position 0.
#pragma once

#include <cooperative_groups.h>

#include "hybrid.cuh"

namespace pace {

// first position the query at `pos` sees
__host__ __device__ __forceinline__ int span_first(int span, int size, int pos) {
  if (span == PACE_SPAN_WINDOW) return pos - size + 1 > 0 ? pos - size + 1 : 0;
  if (span == PACE_SPAN_CHUNK) return pos - pos % size;
  return 0;
}

// elements between the tokens of an output
inline int64_t span_out_row(const pace_attn_span_args_t& a) { return a.out_row ? a.out_row : (int64_t)a.n_q_heads * a.out_elems; }

// Capped scores in log2 units, cap log2(e) tanh(s scale / cap): tanh x = 1 - 2 / (1 + e^2x).
struct ScoreCap {
  float in, out;   // 2 log2(e) scale / cap and cap log2(e); out 0: no cap
};
inline ScoreCap score_cap(float scale, float cap) {
  ScoreCap c;
  c.in = cap > 0.f ? 2.0f * kLog2e * scale / cap : 0.f;
  c.out = cap > 0.f ? cap * kLog2e : 0.f;
  return c;
}

// attn_span_keys.cu: latents on tcgen05; attn_general.cu: the CUDA-core kernel behind pace_attn_span
int attn_span_keys(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_attn_span_args_t& a, cudaStream_t s);
int attn_general_span(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_attn_span_args_t& a,
                      cudaStream_t s);

#ifdef __CUDACC__
__device__ __forceinline__ float capped(const ScoreCap& c, float s) {
  return fmaf(-2.0f * c.out, rcp_t<__nv_bfloat16>(1.0f + fast_exp2(s * c.in)), c.out);
}

// The blocks of a cluster have (maximum, sum) ml[row] (log2 units) and weighted values O[row][stride] of their shares of the
// keys in shared memory, at the same places; every block merges and stores its part of the outputs.  ns (at most 8): blocks
// of the cluster, `share` this one's number; `threads` threads of the block take part, fac: 8 floats of shared memory per
// row, sink: the rows' sinks in log2 units (-infinity: none) in shared memory.  The caller has synchronised the cluster and does so again before anyone leaves.
__device__ __forceinline__ void span_merge(const float* O, int stride, const float2* ml, const float* sink, float* fac, int ns, int share, int tid,
                                           int threads, int live, int r0, int t0, int g, int Gq, int dv, int dv16,
                                           __nv_bfloat16* out, int64_t out_row, int out_elems) {
  cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
  // what each share's values are multiplied by, per row
  for (int r = tid; r < live; r += threads) {
    float2 st[8];
#pragma unroll
    for (int k = 0; k < 8; ++k)
      st[k] = k < ns ? (ns > 1 ? *cl.map_shared_rank(ml + r, k) : ml[r]) : make_float2(-INFINITY, 0.f);
    float top = sink[r];
#pragma unroll
    for (int k = 0; k < 8; ++k) top = fmaxf(top, st[k].x);
    float den = sink[r] == -INFINITY ? 0.f : fast_exp2(sink[r] - top);
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      st[k].x = st[k].x == -INFINITY ? 0.f : fast_exp2(st[k].x - top);
      den = fmaf(st[k].y, st[k].x, den);
    }
    const float inv = den > 0.f ? 1.0f / den : 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) fac[r * 8 + k] = st[k].x * inv;
  }
  asm volatile("bar.sync 1, %0;" ::"r"(threads) : "memory");
  const int v4 = dv16 / 4;
#pragma unroll 2
  for (int i = share * threads + tid; i < live * v4; i += ns * threads) {
    const int r = i / v4, c = (i - r * v4) * 4;
    const int rr = r0 + r, tok = rr / Gq, hh = g * Gq + rr - tok * Gq;
    float4 v[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < ns && fac[r * 8 + k] != 0.f)   // (a share without keys has nothing there)
        v[k] = *reinterpret_cast<const float4*>(ns > 1 ? cl.map_shared_rank(O + r * stride + c, k) : O + r * stride + c);
    }
    float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const float f = fac[r * 8 + k];
      y[0] = fmaf(v[k].x, f, y[0]);
      y[1] = fmaf(v[k].y, f, y[1]);
      y[2] = fmaf(v[k].z, f, y[2]);
      y[3] = fmaf(v[k].w, f, y[3]);
    }
    __nv_bfloat16* dst = out + (t0 + tok) * out_row + (int64_t)hh * out_elems + c;
    if (c + 4 <= dv && ((out_elems | out_row) & 3) == 0) {
      Vec<__nv_bfloat16, 4>::store(dst, y);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < dv) dst[j] = __float2bfloat16_rn(y[j]);
    }
  }
}
#endif  // __CUDACC__

inline bool span_args_ok(const pace_step_t* st, const pace_attn_span_args_t* a, int n_kv_heads) {
  return a && a->q && a->out && a->n_q_heads >= 1 && n_kv_heads >= 1 && a->n_q_heads % n_kv_heads == 0 && a->dim >= 1 &&
         a->vdim >= 1 && a->q_elems >= a->dim && a->out_elems >= a->vdim && a->entry_begin >= 0 &&
         a->entry_end >= a->entry_begin && a->entry_end <= st->n_entries && a->max_tokens >= 0 && a->max_keys >= 0 && a->softcap >= 0.f &&
         (a->out_row == 0 || a->out_row >= (int64_t)a->n_q_heads * a->out_elems) &&
         (a->dtype == PACE_DTYPE_BF16 || a->dtype == PACE_DTYPE_FP32) && a->span >= PACE_SPAN_ALL &&
         a->span <= PACE_SPAN_CHUNK && (a->span == PACE_SPAN_ALL || a->span_size >= 1);
}

}  // namespace pace
