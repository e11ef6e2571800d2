// Gated linear attention with a decay per key channel, token by token: fp32 models and shapes the chunked form (gla_chunk.cu) does
// not take; and one token per sequence with state update, head norm and output gate in one launch.
// States are fp32 and live in per-slot arrays; a sequence that starts at position 0 begins from zeros.
#include "gla.cuh"

namespace pace {
namespace {

// The state in registers: a block owns 32 value columns of one (entry, head), eight lanes share a column; lane s of them holds
// rows 32 i + 4 s .. + 3, so that the eight read 128 neighbouring bytes of a token's key.
constexpr int kSeqTokens = 16;

template <typename T, int D4>
__global__ void __launch_bounds__(256) gla_seq_kernel(pace_step_t st, pace_gla_args_t a) {
  extern __shared__ float smem[];
  constexpr int dp = 32 * D4;
  float* qs = smem;                        // [kSeqTokens][dp], times q_scale
  float* ks = qs + kSeqTokens * dp;        // [kSeqTokens][dp]
  float* gs = ks + kSeqTokens * dp;        // [kSeqTokens][dp], decays
  float* vs = gs + kSeqTokens * dp;        // [kSeqTokens][32]
  float* os = vs + kSeqTokens * 32;        // [kSeqTokens][32]
  const int d = a.dim, vd = a.vdim, H = a.heads, e = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 32;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, slice = lane & 7, cc = warp * 4 + (lane >> 3), col = v0 + cc;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0;
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  float S[D4][4];
#pragma unroll
  for (int i = 0; i < D4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = 32 * i + 4 * slice + j;
      S[i][j] = (st.start[e] != 0 && r < d && col < vd) ? state[(size_t)r * vd + col] : 0.f;
    }
  for (int l0 = 0; l0 < count; l0 += kSeqTokens) {
    const int n = min(kSeqTokens, count - l0);
    __syncthreads();
    for (int j = warp; j < n; j += 8) {
      const size_t t = (size_t)(t0 + l0 + j);
      const T* row = static_cast<const T*>(a.qkv) + t * a.qkv_stride;
      const T* z = static_cast<const T*>(a.z) + t * a.z_stride + (size_t)h * d;
      for (int r = lane; r < dp; r += 32) {
        qs[j * dp + r] = r < d ? to_f<T>(row[(size_t)h * d + r]) * a.q_scale : 0.f;
        ks[j * dp + r] = r < d ? to_f<T>(row[(size_t)(H + h) * d + r]) : 0.f;
        gs[j * dp + r] = r < d ? exp_t<T>(gla_log_decay<T>(to_f<T>(z[r]) + a.z_bias[(size_t)h * d + r], a.inv_tau)) : 1.f;
      }
      vs[j * 32 + lane] = v0 + lane < vd ? to_f<T>(row[2 * (size_t)H * d + (size_t)h * vd + v0 + lane]) : 0.f;
    }
    __syncthreads();
    for (int j = 0; j < n; ++j) {
      const float *kr = ks + j * dp + 4 * slice, *gr = gs + j * dp + 4 * slice, *qr = qs + j * dp + 4 * slice;
      const float u = vs[j * 32 + cc];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < D4; ++i) {
        float k[4], gg[4], q[4];
        Vec<float, 4>::load(kr + 32 * i, k);
        Vec<float, 4>::load(gr + 32 * i, gg);
        Vec<float, 4>::load(qr + 32 * i, q);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          S[i][x] = fmaf(S[i][x], gg[x], k[x] * u);
          o = fmaf(S[i][x], q[x], o);
        }
      }
#pragma unroll
      for (int w = 4; w; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
      if (slice == 0) os[j * 32 + cc] = o;
    }
    __syncthreads();
    for (int i = tid; i < n * 32; i += 256) {
      const int j = i >> 5, c = v0 + (i & 31);
      if (c < vd) static_cast<T*>(a.out)[(size_t)(t0 + l0 + j) * a.out_stride + (size_t)h * vd + c] = from_f<T>(os[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < D4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = 32 * i + 4 * slice + j;
      if (r < d && col < vd) state[(size_t)r * vd + col] = S[i][j];
    }
}

// One token per entry.  A block has a whole head, so that its norm and gate follow without another launch: tiles of 32 V value
// columns, of which a warp takes RW rows at a time (rows warp, warp + 8, ...); a pass asks for its rows before any arithmetic.
constexpr int kStepWarps = 8, kStepThreads = 32 * kStepWarps;

template <typename T, int V, int RW>
__global__ void __launch_bounds__(kStepThreads, 2) gla_step_kernel(pace_step_t st, pace_gla_args_t a) {
  extern __shared__ float smem[];
  __shared__ float part[kStepWarps][32 * V];
  __shared__ float red[32];
  const int d = a.dim, vd = a.vdim, H = a.heads, e = blockIdx.y, h = blockIdx.x, t = st.cu[e];
  float *qs = smem, *ks = qs + d, *gs = ks + d, *vs = gs + d, *os = vs + vd;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const bool fresh = st.start[e] == 0;
  const T* row = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride;
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  float S[RW][V];
  auto fetch = [&](int c0, int r0) {
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const int r = r0 + warp + kStepWarps * i, c = c0 + lane * V;
      if (!fresh && r < d && c < vd) Vec<float, V>::load(state + (size_t)r * vd + c, S[i]);
      else
#pragma unroll
        for (int j = 0; j < V; ++j) S[i][j] = 0.f;
    }
  };
  fetch(0, 0);
  for (int r = tid; r < d; r += kStepThreads) {
    qs[r] = to_f<T>(row[(size_t)h * d + r]) * a.q_scale;
    ks[r] = to_f<T>(row[(size_t)(H + h) * d + r]);
    gs[r] = exp_t<T>(gla_log_decay<T>(to_f<T>(static_cast<const T*>(a.z)[(size_t)t * a.z_stride + (size_t)h * d + r]) + a.z_bias[(size_t)h * d + r],
                                      a.inv_tau));
  }
  for (int c = tid; c < vd; c += kStepThreads) vs[c] = to_f<T>(row[2 * (size_t)H * d + (size_t)h * vd + c]);
  __syncthreads();
  float ss = 0.f;
  for (int c0 = 0; c0 < vd; c0 += 32 * V) {
    const int c = c0 + lane * V;
    float acc[V];
#pragma unroll
    for (int j = 0; j < V; ++j) acc[j] = 0.f;
    for (int r0 = 0; r0 < d; r0 += kStepWarps * RW) {
      if (c0 | r0) fetch(c0, r0);
#pragma unroll
      for (int i = 0; i < RW; ++i) {
        const int r = r0 + warp + kStepWarps * i;
        if (r < d && c < vd) {
          const float g = gs[r], k = ks[r], q = qs[r];
#pragma unroll
          for (int j = 0; j < V; ++j) {
            S[i][j] = fmaf(S[i][j], g, k * vs[c + j]);
            acc[j] = fmaf(S[i][j], q, acc[j]);
          }
          Vec<float, V>::store(state + (size_t)r * vd + c, S[i]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) part[warp][lane * V + j] = acc[j];
    __syncthreads();
    for (int i = tid; i < 32 * V && c0 + i < vd; i += kStepThreads) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kStepWarps; ++w) o += part[w][i];
      os[c0 + i] = o;
      ss = fmaf(o, o, ss);
    }
    __syncthreads();
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)vd + a.eps);
  for (int c = tid; c < vd; c += kStepThreads) {
    const float g = to_f<T>(static_cast<const T*>(a.gate)[(size_t)t * a.gate_stride + (size_t)h * vd + c]);
    static_cast<T*>(a.out)[(size_t)t * a.out_stride + (size_t)h * vd + c] = from_f<T>(os[c] * r * a.norm[c] * silu_t<T>(g));
  }
}

template <typename T, int D4>
int launch_seq(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (3 * kSeqTokens * 32 * D4 + 2 * kSeqTokens * 32);
  PACE_CUDA_TRY(cudaFuncSetAttribute(gla_seq_kernel<T, D4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)((a.vdim + 31) / 32), (unsigned)a.heads, (unsigned)st.n_entries);
  gla_seq_kernel<T, D4><<<grid, 256, smem, s>>>(st, a);
  PACE_LAUNCH_CHECK("gla_seq_kernel");
  return PACE_OK;
}

template <typename T>
int gla_seq(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_seq<T, 1>(st, a, s);
  if (a.dim <= 64) return launch_seq<T, 2>(st, a, s);
  if (a.dim <= 128) return launch_seq<T, 4>(st, a, s);
  if (a.dim <= 256) return launch_seq<T, 8>(st, a, s);
  return launch_seq<T, 16>(st, a, s);
}

template <typename T, int V>
int gla_step_v(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (3 * (size_t)a.dim + 2 * (size_t)a.vdim);
  if (smem > 40 * 1024) return PACE_ERR_UNSUPPORTED;
  const dim3 grid((unsigned)a.heads, (unsigned)st.n_entries);
  if (a.dim <= 4 * kStepWarps) gla_step_kernel<T, V, 4><<<grid, kStepThreads, smem, s>>>(st, a);
  else if (a.dim <= 8 * kStepWarps) gla_step_kernel<T, V, 8><<<grid, kStepThreads, smem, s>>>(st, a);
  else gla_step_kernel<T, V, 16><<<grid, kStepThreads, smem, s>>>(st, a);
  PACE_LAUNCH_CHECK("gla_step_kernel");
  return PACE_OK;
}

template <typename T>
int gla_step_t(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s) {
  if (a.vdim % 4 == 0 && a.vdim > 64 && aligned16(a.s_state)) return gla_step_v<T, 4>(st, a, s);
  if (a.vdim % 2 == 0 && a.vdim > 32 && aligned16(a.s_state)) return gla_step_v<T, 2>(st, a, s);
  return gla_step_v<T, 1>(st, a, s);
}

bool gla_ok(const pace_step_t* st, const pace_gla_args_t* a) {
  if (!step_ok(st) || !a || !a->qkv || !a->z || !a->z_bias || !a->s_state || !a->out) return false;
  if (a->heads < 1 || a->dim < 1 || a->vdim < 1) return false;
  return a->qkv_stride >= (int64_t)a->heads * (2 * (int64_t)a->dim + a->vdim) && a->z_stride >= (int64_t)a->heads * a->dim &&
         a->out_stride >= (int64_t)a->heads * a->vdim && (a->dtype == PACE_DTYPE_BF16 || a->dtype == PACE_DTYPE_FP32);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_gla_prefill(const pace_step_t* st, const pace_gla_args_t* a, void* stream) {
  if (!gla_ok(st, a)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("gla_prefill", stream, "entries=%d tokens=%d heads=%d", st->n_entries, st->n_tokens, a->heads);
  if (gla_chunked_fits(*a)) return gla_chunked(*st, *a, (cudaStream_t)stream);
  return a->dtype == PACE_DTYPE_BF16 ? gla_seq<__nv_bfloat16>(*st, *a, (cudaStream_t)stream) : gla_seq<float>(*st, *a, (cudaStream_t)stream);
}

int pace_gla_step(const pace_step_t* st, const pace_gla_args_t* a, void* stream) {
  if (!gla_ok(st, a) || st->n_tokens != st->n_entries || !a->norm || !a->gate || a->gate_stride < (int64_t)a->heads * a->vdim)
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("gla_step", stream, "entries=%d heads=%d", st->n_entries, a->heads);
  return a->dtype == PACE_DTYPE_BF16 ? gla_step_t<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : gla_step_t<float>(*st, *a, (cudaStream_t)stream);
}

}  // extern "C"
