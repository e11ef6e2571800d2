// Which keys a query sees: plain causality, a sliding window or chunks counted from position 0.
#pragma once

#include "hybrid.cuh"

namespace pace {

// first position the query at `pos` sees
__host__ __device__ __forceinline__ int span_first(int span, int size, int pos) {
  if (span == PACE_SPAN_WINDOW) return pos - size + 1 > 0 ? pos - size + 1 : 0;
  if (span == PACE_SPAN_CHUNK) return pos - pos % size;
  return 0;
}

// attn_general.cu: the CUDA-core kernel behind pace_attn_span
int attn_general_span(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_attn_span_args_t& a,
                      cudaStream_t s);

inline bool span_args_ok(const pace_step_t* st, const pace_attn_span_args_t* a, int n_kv_heads) {
  return a && a->q && a->out && a->n_q_heads >= 1 && n_kv_heads >= 1 && a->n_q_heads % n_kv_heads == 0 && a->dim >= 1 &&
         a->vdim >= 1 && a->q_elems >= a->dim && a->out_elems >= a->vdim && a->entry_begin >= 0 &&
         a->entry_end >= a->entry_begin && a->entry_end <= st->n_entries && a->max_tokens >= 0 && a->max_keys >= 0 &&
         (a->dtype == PACE_DTYPE_BF16 || a->dtype == PACE_DTYPE_FP32) && a->span >= PACE_SPAN_ALL &&
         a->span <= PACE_SPAN_CHUNK && (a->span == PACE_SPAN_ALL || a->span_size >= 1);
}

}  // namespace pace
