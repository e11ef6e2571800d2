#include "delta.cuh"
namespace pace {
bool delta_chunked_fits(const pace_delta_args_t& a) { return false; }
int delta_chunked(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) { return PACE_ERR_UNSUPPORTED; }
}
extern "C" uint64_t pace_delta_workspace_bytes(int32_t n_tokens, int32_t n_entries, int32_t heads, int32_t dim, int32_t vdim, int32_t dtype) { return 0; }
