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

}  // namespace pace
