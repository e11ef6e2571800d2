// Attention over a sliding window of tokens and, further back, the means of whole blocks of tokens.
#pragma once

#include "hybrid.cuh"

namespace pace {

// Blocks (from 0) a query at `pos` sees: those whose last token is `window` or more positions back.
__host__ __device__ __forceinline__ int blocks_seen(int pos, int window, int block) {
  return block > 0 && pos >= window ? (pos - window + 1) / block : 0;
}
// first token it sees
__host__ __device__ __forceinline__ int window_first(int pos, int window) { return pos - window + 1 > 0 ? pos - window + 1 : 0; }

inline bool pooled_args_ok(const pace_kv_pool_t* p, int layer, const pace_kv_pool_t* bp, int block_layer, const pace_step_t* st,
                           const pace_attn_pooled_args_t* a) {
  if (!p || !p->pages || !p->block_table || !step_ok(st) || !a || layer < 0 || layer >= p->n_layers || p->n_kv_heads < 1) return false;
  if (!a->q || !a->out || a->n_q_heads < 1 || a->n_q_heads % p->n_kv_heads || a->dim < 1 || a->vdim < 1 || a->window < 1 || a->block < 0 ||
      a->max_keys < 0 || (a->dtype != PACE_DTYPE_BF16 && a->dtype != PACE_DTYPE_FP32) || a->out_stride < (int64_t)a->n_q_heads * a->vdim ||
      (a->gate && a->gate_stride < (int64_t)a->n_q_heads * a->vdim))
    return false;
  if (p->row_format == PACE_ROWS_SHARED || row_tokens(*p) != 1) return false;
  if (a->block > 0 && (!bp || !bp->pages || !bp->block_table || block_layer < 0 || block_layer >= bp->n_layers || row_tokens(*bp) != a->block ||
                       bp->n_kv_heads != p->n_kv_heads || bp->head_dim != p->head_dim || bp->row_format != p->row_format))
    return false;
  const int row = a->dtype == PACE_DTYPE_BF16 ? p->head_dim : p->head_dim / 2;
  return a->q_elems == row && a->dim <= row && a->vdim <= row && (p->row_format != PACE_ROWS_BF16 || a->dtype == PACE_DTYPE_BF16);
}

}  // namespace pace
