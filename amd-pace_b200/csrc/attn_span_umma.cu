#include "span.cuh"
extern "C" int pace_attn_span_prefill(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step,
                           const pace_attn_span_prefill_args_t* a, void* stream) { return PACE_ERR_UNSUPPORTED; }
