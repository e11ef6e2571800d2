// Forms of the state-space recurrence.
#pragma once

#include "hybrid.cuh"

namespace pace {

// ssd_chunk.cu: many tokens in chunks on the tensor cores
bool ssd_chunked_fits(const pace_ssd_args_t& a);
int ssd_chunked(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s);

}  // namespace pace
