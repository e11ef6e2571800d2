// Forms of the gated delta rule.
#pragma once

#include "hybrid.cuh"

namespace pace {

// delta_chunk.cu: many tokens in chunks on the tensor cores
bool delta_chunked_fits(const pace_delta_args_t& a);
int delta_chunked(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s);

}  // namespace pace
