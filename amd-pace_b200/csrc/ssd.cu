// State-space recurrence with a decay per head and token (Mamba-2), token by token: fp32 models and shapes the chunked form
// (ssd_chunk.cu) does not take; and one token per sequence with convolution and state update in one launch.
// States are fp32 and live in per-slot arrays; a sequence that starts at position 0 begins from zeros.
#include "ssd.cuh"

namespace pace {
namespace {

// The state in registers: a block owns 32 value columns of one (entry, head); warp w holds rows [w DR, (w + 1) DR).
constexpr int kSeqTokens = 16;

template <typename T, int DR>
__global__ void __launch_bounds__(256) ssd_seq_kernel(pace_step_t st, pace_ssd_args_t a) {
  extern __shared__ float smem[];
  const int N = a.state, vd = a.vdim, H = a.heads, dp = 8 * DR, inner = H * vd;
  float* cs = smem;                       // [kSeqTokens][dp]
  float* bs = cs + kSeqTokens * dp;       // [kSeqTokens][dp], times dt
  float* xs = bs + kSeqTokens * dp;       // [kSeqTokens][32]
  float* part = xs + kSeqTokens * 32;     // [kSeqTokens][8][32]
  float* dts = part + kSeqTokens * 256;   // [kSeqTokens] dt
  const int e = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 32, g = h / (H / a.groups);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, col = v0 + lane;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0;
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * N * vd;
  const float neg_a = a.neg_a[h], skip = a.d_skip[h], dt_bias = a.dt_bias[h];
  float S[DR];
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = warp * DR + i;
    S[i] = (st.start[e] != 0 && r < N && col < vd) ? state[(size_t)r * vd + col] : 0.f;
  }
  for (int l0 = 0; l0 < count; l0 += kSeqTokens) {
    const int n = min(kSeqTokens, count - l0);
    __syncthreads();
    if (threadIdx.x < n)
      dts[threadIdx.x] = softplus_t<T>(to_f<T>(static_cast<const T*>(a.dt_raw)[(size_t)(t0 + l0 + threadIdx.x) * a.dt_stride + h]) + dt_bias);
    __syncthreads();
    for (int i = threadIdx.x; i < n * dp; i += 256) {
      const int j = i / dp, r = i - j * dp;
      const T* row = static_cast<const T*>(a.xbc) + (size_t)(t0 + l0 + j) * a.xbc_stride + inner + (size_t)g * N;
      bs[i] = r < N ? to_f<T>(row[r]) * dts[j] : 0.f;
      cs[i] = r < N ? to_f<T>(row[(size_t)a.groups * N + r]) : 0.f;
    }
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int j = i >> 5, c = v0 + (i & 31);
      xs[i] = c < vd ? to_f<T>(static_cast<const T*>(a.xbc)[(size_t)(t0 + l0 + j) * a.xbc_stride + (size_t)h * vd + c]) : 0.f;
    }
    __syncthreads();
    for (int j = 0; j < n; ++j) {
      const float x = xs[j * 32 + lane], decay = exp_t<T>(neg_a * dts[j]);
      const float *br = bs + j * dp + warp * DR, *cr = cs + j * dp + warp * DR;
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DR; ++i) {
        S[i] = fmaf(decay, S[i], br[i] * x);
        o = fmaf(S[i], cr[i], o);
      }
      part[(j * 8 + warp) * 32 + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int j = i >> 5, c = i & 31;
      float o = skip * xs[i];
#pragma unroll
      for (int w = 0; w < 8; ++w) o += part[(j * 8 + w) * 32 + c];
      if (v0 + c < vd) static_cast<T*>(a.out)[(size_t)(t0 + l0 + j) * a.out_stride + (size_t)h * vd + v0 + c] = from_f<T>(o);
    }
  }
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = warp * DR + i;
    if (r < N && col < vd) state[(size_t)r * vd + col] = S[i];
  }
}

// One token per entry: the state of V CL value columns of one (entry, head) is on its way to registers while the block convolves what
// it needs of the projections; it is read and written once.  CL lanes share a row, a thread has rows tid / CL + k 256 / CL, k < RW.
template <typename T, int V, int CL, int RW, int NT>
__global__ void __launch_bounds__(256, RW * V <= 16 ? 4 : RW * V <= 32 ? 3 : RW * V <= 64 ? 2 : 1) ssd_step_kernel(pace_step_t st, pace_ssd_args_t a) {
  constexpr int COLS = V * CL, RG = 256 / CL;      // columns of the block, rows of a pass
  __shared__ float bs[512], cs[512], xs[COLS];
  __shared__ float part[8][COLS];
  const int e = blockIdx.z, h = blockIdx.y, N = a.state, vd = a.vdim, H = a.heads, per_g = H / a.groups, g = h / per_g;
  const int inner = H * vd, tid = threadIdx.x, warp = tid >> 5, c0 = blockIdx.x * COLS, cl = tid % CL, col = c0 + cl * V, t = st.cu[e];
  const int pos = st.start[e], channels = inner + 2 * a.groups * N, r0 = tid / CL;
  const T* row = static_cast<const T*>(a.xbc) + (size_t)t * a.xbc_stride;
  float* ring = a.ring + (size_t)st.slot[e] * a.ring_rows * a.ring_stride;
  const int total = 2 * N + COLS;
  // the i-th channel the block needs (-1: none): b and c of the group, then its columns of x
  auto channel = [&](int i) {
    if (i < 2 * N) return inner + (i < N ? 0 : a.groups * N) + g * N + (i < N ? i : i - N);
    return i < total && c0 + i - 2 * N < vd ? h * vd + c0 + i - 2 * N : -1;
  };
  constexpr int AHEAD = 2;
  ConvNow<T, NT> cv[AHEAD];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) {
    const int ch = channel(tid + 256 * k);
    if (ch >= 0) cv[k].load(row, ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, a.conv_bias, pos, ch);
  }
  const float dt_raw = to_f<T>(static_cast<const T*>(a.dt_raw)[(size_t)t * a.dt_stride + h]) + a.dt_bias[h];
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * N * vd;
  float S[RW][V];
#pragma unroll
  for (int k = 0; k < RW; ++k) {
    const int r = r0 + k * RG;
    if (pos != 0 && r < N && col < vd) Vec<float, V>::load(state + (size_t)r * vd + col, S[k]);
    else
#pragma unroll
      for (int j = 0; j < V; ++j) S[k][j] = 0.f;
  }
  const float dt = softplus_t<T>(dt_raw);
  const float decay = exp_t<T>(a.neg_a[h] * dt);
  const int now_row = pos % a.ring_rows;
  auto convolved = [&](int i, int ch, const ConvNow<T, NT>& in) {
    if (ch < 0) {
      if (i < total) xs[i - 2 * N] = 0.f;
      return;
    }
    const float y = round_to<T>(silu_t<T>(in.sum(ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, pos, ch)));
    if (i < N) bs[i] = y * dt;
    else if (i < 2 * N) cs[i - N] = y;
    else xs[i - 2 * N] = y;
    // the current row's place is read by nobody in this launch; one block writes a channel
    if (i >= 2 * N || (h == g * per_g && blockIdx.x == 0)) ring[(size_t)now_row * a.ring_stride + ch] = in.now;
  };
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) convolved(tid + 256 * k, channel(tid + 256 * k), cv[k]);
  for (int i = tid + 256 * AHEAD; i < total; i += 256) {
    const int ch = channel(i);
    ConvNow<T, NT> in;
    if (ch >= 0) in.load(row, ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, a.conv_bias, pos, ch);
    convolved(i, ch, in);
  }
  __syncthreads();
  float x[V], o[V];
#pragma unroll
  for (int j = 0; j < V; ++j) x[j] = xs[cl * V + j], o[j] = 0.f;
#pragma unroll
  for (int k = 0; k < RW; ++k) {
    const int r = r0 + k * RG;
    if (r < N && col < vd) {
      const float b = bs[r], c = cs[r];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        S[k][j] = fmaf(decay, S[k][j], b * x[j]);
        o[j] = fmaf(S[k][j], c, o[j]);
      }
      Vec<float, V>::store(state + (size_t)r * vd + col, S[k]);
    }
  }
#pragma unroll
  for (int w = CL; w < 32; w <<= 1)
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
  if ((tid & 31) < CL) {
#pragma unroll
    for (int j = 0; j < V; ++j) part[warp][cl * V + j] = o[j];
  }
  __syncthreads();
  for (int i = tid; i < COLS; i += 256) {
    if (c0 + i >= vd) break;
    float s = a.d_skip[h] * xs[i];
#pragma unroll
    for (int w = 0; w < 8; ++w) s += part[w][i];
    static_cast<T*>(a.out)[(size_t)t * a.out_stride + (size_t)h * vd + c0 + i] = from_f<T>(s);
  }
}

template <typename T, int DR>
int launch_seq(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (2 * kSeqTokens * 8 * DR + kSeqTokens * 32 + kSeqTokens * 256 + kSeqTokens);
  PACE_CUDA_TRY(cudaFuncSetAttribute(ssd_seq_kernel<T, DR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)((a.vdim + 31) / 32), (unsigned)a.heads, (unsigned)st.n_entries);
  ssd_seq_kernel<T, DR><<<grid, 256, smem, s>>>(st, a);
  PACE_LAUNCH_CHECK("ssd_seq_kernel");
  return PACE_OK;
}

template <typename T>
int ssd_seq(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  if (a.state <= 32) return launch_seq<T, 4>(st, a, s);
  if (a.state <= 64) return launch_seq<T, 8>(st, a, s);
  if (a.state <= 128) return launch_seq<T, 16>(st, a, s);
  if (a.state <= 256) return launch_seq<T, 32>(st, a, s);
  return launch_seq<T, 64>(st, a, s);
}

template <typename T, int V, int CL, int NT>
int launch_step_taps(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  constexpr int RG = 256 / CL;
  const dim3 grid((unsigned)((a.vdim + CL * V - 1) / (CL * V)), (unsigned)a.heads, (unsigned)st.n_entries);
  if (a.state <= 4 * RG) ssd_step_kernel<T, V, CL, 4, NT><<<grid, 256, 0, s>>>(st, a);
  else if (a.state <= 8 * RG) ssd_step_kernel<T, V, CL, 8, NT><<<grid, 256, 0, s>>>(st, a);
  else if (a.state <= 16 * RG) ssd_step_kernel<T, V, CL, 16, NT><<<grid, 256, 0, s>>>(st, a);
  else if (V * CL <= 32) ssd_step_kernel<T, 1, 32, 64, 0><<<grid, 256, 0, s>>>(st, a);
  else return PACE_ERR_UNSUPPORTED;
  PACE_LAUNCH_CHECK("ssd_step_kernel");
  return PACE_OK;
}

template <typename T, int V, int CL>
int launch_step(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  return a.n_taps == 4 ? launch_step_taps<T, V, CL, 4>(st, a, s) : launch_step_taps<T, V, CL, 0>(st, a, s);
}

template <typename T>
int ssd_step_t(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  if (a.vdim % 4 == 0 && aligned16(a.s_state)) {
    if (a.vdim > 64 && a.state <= 128) return launch_step<T, 4, 32>(st, a, s);
    if (a.vdim > 32 && a.state <= 256) return launch_step<T, 4, 16>(st, a, s);
    return launch_step<T, 4, 8>(st, a, s);      // (256 / 8 * 16 rows: any state up to 512)
  }
  return launch_step<T, 1, 32>(st, a, s);
}

bool ssd_ok(const pace_step_t* st, const pace_ssd_args_t* a) {
  if (!step_ok(st) || !a || !a->xbc || !a->dt_raw || !a->dt_bias || !a->neg_a || !a->d_skip || !a->s_state || !a->out) return false;
  if (a->heads < 1 || a->groups < 1 || a->heads % a->groups || a->state < 1 || a->vdim < 1) return false;
  const int64_t inner = (int64_t)a->heads * a->vdim, channels = inner + 2 * (int64_t)a->groups * a->state;
  return a->xbc_stride >= channels && a->out_stride >= inner && a->dt_stride >= a->heads &&
         (a->dtype == PACE_DTYPE_BF16 || a->dtype == PACE_DTYPE_FP32);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_ssd_prefill(const pace_step_t* st, const pace_ssd_args_t* a, void* stream) {
  if (!ssd_ok(st, a)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->state > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("ssd_prefill", stream, "entries=%d tokens=%d heads=%d", st->n_entries, st->n_tokens, a->heads);
  if (ssd_chunked_fits(*a)) return ssd_chunked(*st, *a, (cudaStream_t)stream);
  return a->dtype == PACE_DTYPE_BF16 ? ssd_seq<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : ssd_seq<float>(*st, *a, (cudaStream_t)stream);
}

int pace_ssd_step(const pace_step_t* st, const pace_ssd_args_t* a, void* stream) {
  if (!ssd_ok(st, a) || st->n_tokens != st->n_entries || !a->taps || !a->ring || a->n_taps < 1 || a->ring_rows < a->n_taps ||
      a->ring_stride < a->heads * a->vdim + 2 * a->groups * a->state)
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->state > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("ssd_step", stream, "entries=%d heads=%d", st->n_entries, a->heads);
  return a->dtype == PACE_DTYPE_BF16 ? ssd_step_t<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : ssd_step_t<float>(*st, *a, (cudaStream_t)stream);
}

}  // extern "C"
