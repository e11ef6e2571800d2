// Forms of gated linear attention.
#pragma once

#include "hybrid.cuh"

namespace pace {

// gla_chunk.cu: many tokens in chunks on the tensor cores
bool gla_chunked_fits(const pace_gla_args_t& a);
int gla_chunked(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s);

// ln of a decay: sigmoid(z)^(1 / tau) = e^(-softplus(-z) / tau)
template <typename T> __device__ __forceinline__ float gla_log_decay(float z, float inv_tau) { return -softplus_t<T>(-z) * inv_tau; }

}  // namespace pace
