// Gated delta rule with a decay per key channel, token by token: fp32 models and shapes the chunked form (delta_chunk.cu) does
// not take; and one token per sequence with convolutions, unit norms and state update in one launch.
// States are fp32 and live in per-slot arrays; a sequence that starts at position 0 begins from zeros.
#include "delta.cuh"

namespace pace {
namespace {

// The state in registers: a block owns 32 value columns of one (entry, head), eight lanes share a column; lane s of them holds
// rows 32 i + 4 s .. + 3, so that the eight read 128 neighbouring bytes of a token's key.
constexpr int kSeqTokens = 16;

template <typename T, int D4>
__global__ void __launch_bounds__(256) delta_seq_kernel(pace_step_t st, pace_delta_args_t a) {
  extern __shared__ float smem[];
  constexpr int dp = 32 * D4;
  float* qs = smem;                        // [kSeqTokens][dp], unit times q_scale
  float* ks = qs + kSeqTokens * dp;        // [kSeqTokens][dp], unit
  float* gs = ks + kSeqTokens * dp;        // [kSeqTokens][dp], decays
  float* vs = gs + kSeqTokens * dp;        // [kSeqTokens][32]
  float* os = vs + kSeqTokens * 32;        // [kSeqTokens][32]
  float* betas = os + kSeqTokens * 32;     // [kSeqTokens]
  const int d = a.dim, vd = a.vdim, H = a.heads, G = a.kv_heads, e = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 32, g = h / (H / G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, slice = lane & 7, cc = warp * 4 + (lane >> 3), col = v0 + cc;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0;
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  const float neg_a = a.neg_a[h];
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
      const T* row = static_cast<const T*>(a.qkv) + t * a.qkv_stride + g * d;
      const T* ar = static_cast<const T*>(a.a_raw) + t * a.a_stride + (size_t)h * d;
      float sq = 0.f, sk = 0.f;
      for (int r = lane; r < dp; r += 32) {
        const float q = r < d ? to_f<T>(row[r]) : 0.f, k = r < d ? to_f<T>(row[(size_t)G * d + r]) : 0.f;
        qs[j * dp + r] = q;
        ks[j * dp + r] = k;
        gs[j * dp + r] = r < d ? exp_t<T>(neg_a * softplus_t<T>(to_f<T>(ar[r]) + a.dt_bias[(size_t)h * d + r])) : 1.f;
        sq = fmaf(q, q, sq);
        sk = fmaf(k, k, sk);
      }
#pragma unroll
      for (int o = 16; o; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
      }
      const float fq = a.q_scale / sqrtf(sq + a.unit_eps), fk = 1.0f / sqrtf(sk + a.unit_eps);
      for (int r = lane; r < dp; r += 32) {
        qs[j * dp + r] *= fq;
        ks[j * dp + r] *= fk;
      }
      vs[j * 32 + lane] = v0 + lane < vd
                              ? to_f<T>(static_cast<const T*>(a.qkv)[t * a.qkv_stride + 2 * (size_t)G * d + (size_t)h * vd + v0 + lane]) : 0.f;
      if (lane == 0) betas[j] = sigmoid_t<T>(to_f<T>(static_cast<const T*>(a.b_raw)[t * a.b_stride + h]));
    }
    __syncthreads();
    for (int j = 0; j < n; ++j) {
      const float *kr = ks + j * dp + 4 * slice, *gr = gs + j * dp + 4 * slice, *qr = qs + j * dp + 4 * slice;
      float k[D4][4], p = 0.f, o = 0.f;
#pragma unroll
      for (int i = 0; i < D4; ++i) {
        float gg[4];
        Vec<float, 4>::load(kr + 32 * i, k[i]);
        Vec<float, 4>::load(gr + 32 * i, gg);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          S[i][x] *= gg[x];
          p = fmaf(S[i][x], k[i][x], p);
        }
      }
#pragma unroll
      for (int w = 4; w; w >>= 1) p += __shfl_xor_sync(0xffffffffu, p, w);
      const float u = betas[j] * (vs[j * 32 + cc] - p);
#pragma unroll
      for (int i = 0; i < D4; ++i) {
        float q[4];
        Vec<float, 4>::load(qr + 32 * i, q);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          S[i][x] = fmaf(k[i][x], u, S[i][x]);
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

// One token per entry.  A block owns 32 V value columns of one (entry, head), its state in registers (RW rows per warp): read
// once, decayed, read out against the key, corrected, read out against the query, written once.
constexpr int kStepWarps = 8;

template <typename T, int V, int RW, int NT>
__global__ void __launch_bounds__(32 * kStepWarps, RW * V <= 16 ? 4 : RW * V <= 32 ? 3 : RW * V <= 64 ? 2 : 1) delta_step_kernel(pace_step_t st, pace_delta_args_t a) {
  __shared__ float qs[512], ks[512], gs[512], vs[32 * V], us[32 * V];
  __shared__ float part[kStepWarps][32 * V];
  __shared__ float unit[2];
  const int d = a.dim, vd = a.vdim, H = a.heads, G = a.kv_heads, e = blockIdx.z, h = blockIdx.y, per_g = H / G, g = h / per_g;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, c0 = blockIdx.x * 32 * V, col = c0 + lane * V, t = st.cu[e];
  const int pos = st.start[e], slot = st.slot[e], channels = 2 * G * d + H * vd;
  constexpr int THREADS = 32 * kStepWarps, AHEAD = 2;
  const T* row = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride;
  float* ring = a.ring + (size_t)slot * a.ring_rows * a.ring_stride;
  const int total = 2 * d + 32 * V;
  // the i-th channel the block needs (-1: none): q and k of the head, then its columns of v
  auto channel = [&](int i) {
    if (i < 2 * d) return (i < d ? 0 : G * d) + g * d + (i < d ? i : i - d);
    return i < total && c0 + i - 2 * d < vd ? 2 * G * d + h * vd + c0 + i - 2 * d : -1;
  };
  ConvNow<T, NT> cv[AHEAD];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) {
    const int ch = channel(tid + THREADS * k);
    if (ch >= 0) cv[k].load(row, ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, nullptr, pos, ch);
  }
  auto decay_in = [&](int r) { return to_f<T>(static_cast<const T*>(a.a_raw)[(size_t)t * a.a_stride + (size_t)h * d + r]) + a.dt_bias[(size_t)h * d + r]; };
  const float first_decay = tid < d ? decay_in(tid) : 0.f, neg_a = a.neg_a[h];
  const float beta_raw = to_f<T>(static_cast<const T*>(a.b_raw)[(size_t)t * a.b_stride + h]);
  float* state = a.s_state + ((size_t)slot * H + h) * d * vd;
  float S[RW][V];
#pragma unroll
  for (int i = 0; i < RW; ++i) {
    const int r = warp * RW + i;
    if (pos != 0 && r < d && col < vd) Vec<float, V>::load(state + (size_t)r * vd + col, S[i]);
    else
#pragma unroll
      for (int j = 0; j < V; ++j) S[i][j] = 0.f;
  }
  const int now_row = pos % a.ring_rows;
  auto convolved = [&](int i, int ch, const ConvNow<T, NT>& in) {
    if (ch < 0) {
      if (i < total) vs[i - 2 * d] = 0.f;
      return;
    }
    const float y = round_to<T>(silu_t<T>(in.sum(ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, pos, ch)));
    if (i < d) qs[i] = y;
    else if (i < 2 * d) ks[i - d] = y;
    else vs[i - 2 * d] = y;
    // the current row's place is read by nobody in this launch; one block writes a channel
    if (i >= 2 * d || (h == g * per_g && blockIdx.x == 0)) ring[(size_t)now_row * a.ring_stride + ch] = in.now;
  };
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) convolved(tid + THREADS * k, channel(tid + THREADS * k), cv[k]);
  for (int i = tid + THREADS * AHEAD; i < total; i += THREADS) {
    const int ch = channel(i);
    ConvNow<T, NT> in;
    if (ch >= 0) in.load(row, ring, a.ring_rows, a.ring_stride, a.taps, channels, a.n_taps, nullptr, pos, ch);
    convolved(i, ch, in);
  }
  for (int r = tid; r < d; r += THREADS) gs[r] = exp_t<T>(neg_a * softplus_t<T>(r == tid ? first_decay : decay_in(r)));
  const float beta = sigmoid_t<T>(beta_raw);
  __syncthreads();
  if (warp < 2) {
    const float* x = warp ? ks : qs;
    float ss = 0.f;
    for (int r = lane; r < d; r += 32) ss = fmaf(x[r], x[r], ss);
#pragma unroll
    for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) unit[warp] = (warp ? 1.0f : a.q_scale) / sqrtf(ss + a.unit_eps);
  }
  float acc[V];
#pragma unroll
  for (int j = 0; j < V; ++j) acc[j] = 0.f;
#pragma unroll
  for (int i = 0; i < RW; ++i) {
    const int r = min(warp * RW + i, d - 1);      // (rows behind the end are zero)
    const float gg = gs[r], k = ks[r];
#pragma unroll
    for (int j = 0; j < V; ++j) {
      S[i][j] *= gg;
      acc[j] = fmaf(S[i][j], k, acc[j]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) part[warp][lane * V + j] = acc[j];
  __syncthreads();
  const float fq = unit[0], fk = unit[1];
  for (int i = tid; i < 32 * V; i += 32 * kStepWarps) {
    float p = 0.f;
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) p += part[w][i];
    us[i] = beta * (vs[i] - p * fk) * fk;         // (times the key's unit factor: k u^T takes the plain key)
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < V; ++j) acc[j] = 0.f;
#pragma unroll
  for (int i = 0; i < RW; ++i) {
    const int r = warp * RW + i;
    if (r < d && col < vd) {
      const float k = ks[r], q = qs[r];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        S[i][j] = fmaf(k, us[lane * V + j], S[i][j]);
        acc[j] = fmaf(S[i][j], q, acc[j]);
      }
      Vec<float, V>::store(state + (size_t)r * vd + col, S[i]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) part[warp][lane * V + j] = acc[j];
  __syncthreads();
  for (int i = tid; i < 32 * V; i += 32 * kStepWarps) {
    if (c0 + i >= vd) break;
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) o += part[w][i];
    static_cast<T*>(a.out)[(size_t)t * a.out_stride + (size_t)h * vd + c0 + i] = from_f<T>(o * fq);
  }
}

template <typename T, int D4>
int launch_seq(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (3 * kSeqTokens * 32 * D4 + 2 * kSeqTokens * 32 + kSeqTokens);
  PACE_CUDA_TRY(cudaFuncSetAttribute(delta_seq_kernel<T, D4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)((a.vdim + 31) / 32), (unsigned)a.heads, (unsigned)st.n_entries);
  delta_seq_kernel<T, D4><<<grid, 256, smem, s>>>(st, a);
  PACE_LAUNCH_CHECK("delta_seq_kernel");
  return PACE_OK;
}

template <typename T>
int delta_seq(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_seq<T, 1>(st, a, s);
  if (a.dim <= 64) return launch_seq<T, 2>(st, a, s);
  if (a.dim <= 128) return launch_seq<T, 4>(st, a, s);
  if (a.dim <= 256) return launch_seq<T, 8>(st, a, s);
  return launch_seq<T, 16>(st, a, s);
}

template <typename T, int V, int NT>
int delta_step_taps(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  const dim3 grid((unsigned)((a.vdim + 32 * V - 1) / (32 * V)), (unsigned)a.heads, (unsigned)st.n_entries);
  if (a.dim <= 4 * kStepWarps) delta_step_kernel<T, V, 4, NT><<<grid, 32 * kStepWarps, 0, s>>>(st, a);
  else if (a.dim <= 8 * kStepWarps) delta_step_kernel<T, V, 8, NT><<<grid, 32 * kStepWarps, 0, s>>>(st, a);
  else if (a.dim <= 16 * kStepWarps) delta_step_kernel<T, V, 16, NT><<<grid, 32 * kStepWarps, 0, s>>>(st, a);
  else if (V == 1 && a.dim <= 32 * kStepWarps) delta_step_kernel<T, 1, 32, 0><<<grid, 32 * kStepWarps, 0, s>>>(st, a);
  else if (V == 1) delta_step_kernel<T, 1, 64, 0><<<grid, 32 * kStepWarps, 0, s>>>(st, a);
  else return PACE_ERR_UNSUPPORTED;
  PACE_LAUNCH_CHECK("delta_step_kernel");
  return PACE_OK;
}

template <typename T, int V>
int delta_step_v(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  return a.n_taps == 4 ? delta_step_taps<T, V, 4>(st, a, s) : delta_step_taps<T, V, 0>(st, a, s);
}

template <typename T>
int delta_step_t(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  if (a.dim <= 128 && a.vdim % 2 == 0 && a.vdim >= 64 && aligned16(a.s_state)) return delta_step_v<T, 2>(st, a, s);
  return delta_step_v<T, 1>(st, a, s);
}

bool delta_ok(const pace_step_t* st, const pace_delta_args_t* a) {
  if (!step_ok(st) || !a || !a->qkv || !a->a_raw || !a->b_raw || !a->dt_bias || !a->neg_a || !a->s_state || !a->out) return false;
  if (a->heads < 1 || a->kv_heads < 1 || a->heads % a->kv_heads || a->dim < 1 || a->vdim < 1) return false;
  const int64_t channels = 2 * (int64_t)a->kv_heads * a->dim + (int64_t)a->heads * a->vdim;
  return a->qkv_stride >= channels && a->a_stride >= (int64_t)a->heads * a->dim && a->b_stride >= a->heads &&
         a->out_stride >= (int64_t)a->heads * a->vdim && (a->dtype == PACE_DTYPE_BF16 || a->dtype == PACE_DTYPE_FP32);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_delta_prefill(const pace_step_t* st, const pace_delta_args_t* a, void* stream) {
  if (!delta_ok(st, a)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("delta_prefill", stream, "entries=%d tokens=%d heads=%d", st->n_entries, st->n_tokens, a->heads);
  if (delta_chunked_fits(*a)) return delta_chunked(*st, *a, (cudaStream_t)stream);
  return a->dtype == PACE_DTYPE_BF16 ? delta_seq<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : delta_seq<float>(*st, *a, (cudaStream_t)stream);
}

int pace_delta_step(const pace_step_t* st, const pace_delta_args_t* a, void* stream) {
  if (!delta_ok(st, a) || st->n_tokens != st->n_entries || !a->taps || !a->ring || a->n_taps < 1 || a->ring_rows < a->n_taps ||
      a->ring_stride < 2 * a->kv_heads * a->dim + a->heads * a->vdim)
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("delta_step", stream, "entries=%d heads=%d", st->n_entries, a->heads);
  return a->dtype == PACE_DTYPE_BF16 ? delta_step_t<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : delta_step_t<float>(*st, *a, (cudaStream_t)stream);
}

}  // extern "C"
