// Recurrent layers: short causal convolution, the real-gated linear recurrence (RG-LRU) and linear attention
// with a fixed decay per head.  States are fp32 and live in per-slot arrays; a sequence that starts at
// position 0 begins from zeros whatever its slot holds, so slots are reused without clearing them.
#include "hybrid.cuh"

namespace pace {
namespace {

// ---------------------------------------------------------------------------
// causal depthwise convolution
// ---------------------------------------------------------------------------
// Input of channel c at `back` tokens in front of local token l of an entry: from the step's rows, from the
// slot's ring of newest inputs, or zero in front of the sequence.
template <typename T>
__device__ __forceinline__ float conv_input(const T* __restrict__ in, int64_t in_stride, const float* __restrict__ ring,
                                            int n_taps, int channels, int t, int l, int pos, int back, int c) {
  if (l >= back) return to_f<T>(in[(size_t)(t - back) * in_stride + c]);
  if (pos < back) return 0.f;
  return ring[(size_t)((pos - back) % n_taps) * channels + c];
}

template <typename T, int V>
__global__ void causal_conv_kernel(pace_step_t st, const T* __restrict__ in, int64_t in_stride, const float* __restrict__ taps,
                                   const float* __restrict__ bias, int n_taps, const float* __restrict__ conv_state,
                                   T* __restrict__ out, int channels) {
  const int per = channels / V;
  const size_t total = (size_t)st.n_tokens * per;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i % per) * V;
    const int e = st.tok_entry[t], l = t - st.cu[e], pos = st.tok_pos[t];
    float acc[V];
    Vec<float, V>::load(bias + c, acc);
    for (int j = 0; j < n_taps; ++j) {
      const int back = n_taps - 1 - j;
      float x[V];
      if (l >= back) {
        Vec<T, V>::load(in + (size_t)(t - back) * in_stride + c, x);
      } else if (pos >= back) {
        Vec<float, V>::load(conv_state + ((size_t)st.slot[e] * n_taps + (pos - back) % n_taps) * channels + c, x);
      } else {
        continue;
      }
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = fmaf(taps[(size_t)(c + v) * n_taps + j], x[v], acc[v]);
    }
    Vec<T, V>::store(out + (size_t)t * channels + c, acc);
  }
}

// ---------------------------------------------------------------------------
// RG-LRU over any number of tokens: gates and convolution come from launches in front
// ---------------------------------------------------------------------------
constexpr int kSegs = 16, kSegTokens = 8, kTile = kSegs * kSegTokens;

// coefficients of S_t = a S_(t-1) + b for pre-activations of the two gates
template <typename T>
__device__ __forceinline__ void rglru_coefficients(float r_pre, float i_pre, float u, float decay_base, float& a, float& b) {
  const float log_a = decay_base * sigmoid_t<T>(r_pre);
  a = exp_t<T>(log_a);
  b = sqrtf(one_minus_exp<T>(2.0f * log_a, a * a)) * sigmoid_t<T>(i_pre) * u;
}

// A block walks 32 channels of one entry in tiles of 128 tokens: warp = a segment of 8 tokens, lane = a
// channel.  A thread composes its 8 steps into one affine map, the 16 maps of a channel meet in shared
// memory, every thread then replays its 8 steps from the state in front of them.  The next tile's operands
// are on their way meanwhile.
template <typename T>
__global__ void __launch_bounds__(512)
    rglru_scan_kernel(pace_step_t st, pace_rglru_args_t a) {
  __shared__ float2 maps[2][kSegs][32];
  const int e = blockIdx.y, lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int W = a.width, c = blockIdx.x * 32 + lane;
  const bool live = c < W;
  const int cc = live ? c : 0;
  const int bs = W / a.blocks, blk = cc / bs, in_blk = cc - blk * bs;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0, start = st.start[e], slot = st.slot[e];
  const T* u = static_cast<const T*>(a.u) + cc;
  const T* yx = static_cast<const T*>(a.yx) + cc;
  const float* gr = a.gates + (size_t)blk * st.n_tokens * 2 * bs + in_blk;
  T* out = static_cast<T*>(a.out) + cc;
  const float rb = a.ra_bias[cc], ib = a.ri_bias[cc], base = a.decay_base[cc];
  float* state = a.state + (size_t)slot * W + cc;
  float carry = start == 0 ? 0.f : *state;

  float g0[kSegTokens], g1[kSegTokens], uu[kSegTokens], yy[kSegTokens];
  auto fetch = [&](int tile) {
#pragma unroll
    for (int j = 0; j < kSegTokens; ++j) {
      const int l = tile * kTile + seg * kSegTokens + j;
      if (l < count) {
        const size_t t = (size_t)(t0 + l);
        g0[j] = gr[t * 2 * bs];
        g1[j] = gr[t * 2 * bs + bs];
        uu[j] = to_f<T>(u[t * W]);
        yy[j] = to_f<T>(yx[t * a.yx_stride]);
      }
    }
  };
  fetch(0);
  const int tiles = (count + kTile - 1) / kTile;
  for (int tile = 0; tile < tiles; ++tile) {
    float ca[kSegTokens], cb[kSegTokens], y[kSegTokens], A = 1.f, B = 0.f;
    const int l0 = tile * kTile + seg * kSegTokens;
#pragma unroll
    for (int j = 0; j < kSegTokens; ++j) {
      if (l0 + j < count) {
        rglru_coefficients<T>(g0[j] + rb, g1[j] + ib, uu[j], base, ca[j], cb[j]);
        y[j] = yy[j];
        A *= ca[j];
        B = fmaf(ca[j], B, cb[j]);
      }
    }
    if (tile + 1 < tiles) fetch(tile + 1);
    maps[tile & 1][seg][lane] = make_float2(A, B);
    __syncthreads();
    float s = carry, mine = 0.f;
#pragma unroll
    for (int k = 0; k < kSegs; ++k) {
      if (k == seg) mine = s;
      const float2 m = maps[tile & 1][k][lane];
      s = fmaf(m.x, s, m.y);
    }
    carry = s;
#pragma unroll
    for (int j = 0; j < kSegTokens; ++j) {
      if (l0 + j < count) {
        mine = fmaf(ca[j], mine, cb[j]);
        if (live) out[(size_t)(t0 + l0 + j) * W] = from_f<T>(mine * gelu_tanh_t<T>(y[j]));
      }
    }
  }
  if (!live) return;
  if (seg == 0) *state = carry;
  for (int j = seg; j < a.n_taps && j < count; j += kSegs) {
    const int l = count - 1 - j;
    a.conv_state[((size_t)slot * a.n_taps + (start + l) % a.n_taps) * W + c] =
        to_f<T>(yx[(size_t)(t0 + l) * a.yx_stride + W]);
  }
}

// ---------------------------------------------------------------------------
// RG-LRU, one token per entry: convolution, block-diagonal gates, state update and branch product
// ---------------------------------------------------------------------------
constexpr int kStepEntries = 32, kStepChannels = 32;

__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// two consecutive weights of a row of `n`, zero behind its end; rows of odd length are not word aligned
__device__ __forceinline__ uint32_t load_pair(const __nv_bfloat16* row, int k, int n, bool even) {
  if (even) return k < n ? *reinterpret_cast<const uint32_t*>(row + k) : 0u;
  uint32_t lo = 0, hi = 0;
  if (k < n) lo = *reinterpret_cast<const uint16_t*>(row + k);
  if (k + 1 < n) hi = *reinterpret_cast<const uint16_t*>(row + k + 1);
  return lo | (hi << 16);
}

template <typename T>
__device__ __forceinline__ void rglru_finish(const pace_step_t& st, const pace_rglru_args_t& a, int e, int c, float r_pre,
                                             float i_pre, float u) {
  const int W = a.width, slot = st.slot[e], pos = st.start[e];
  float ca, cb;
  rglru_coefficients<T>(r_pre + a.ra_bias[c], i_pre + a.ri_bias[c], u, a.decay_base[c], ca, cb);
  float* s = a.state + (size_t)slot * W + c;
  const float S = pos == 0 ? cb : fmaf(ca, *s, cb);
  *s = S;
  const T* row = static_cast<const T*>(a.yx) + (size_t)st.cu[e] * a.yx_stride;
  a.conv_state[((size_t)slot * a.n_taps + pos % a.n_taps) * W + c] = to_f<T>(row[W + c]);
  static_cast<T*>(a.out)[(size_t)st.cu[e] * W + c] = from_f<T>(S * gelu_tanh_t<T>(to_f<T>(row[c])));
}

// Block (slice, batch tile): 32 output channels of one gate block for 32 entries.  bf16: warp w multiplies
// entries [16 (w / 4), +16) with channels [8 (w % 4), +8) of both gates on the tensor cores (fp32
// accumulators are the pre-activations); fp32: one thread per (entry, channel).
template <typename T>
__global__ void __launch_bounds__(256)
    rglru_step_kernel(pace_step_t st, pace_rglru_args_t a, int slices, int ld) {
  extern __shared__ __align__(16) char smem_raw[];
  T* us = reinterpret_cast<T*>(smem_raw);  // [kStepEntries][ld]
  const int W = a.width, bs = W / a.blocks;
  const int blk = blockIdx.x / slices, o0 = (blockIdx.x % slices) * kStepChannels;
  const int e0 = blockIdx.y * kStepEntries, E = st.n_entries;
  const T* x0 = static_cast<const T*>(a.yx) + W;
  for (int i = threadIdx.x; i < kStepEntries * ld; i += 256) {
    const int r = i / ld, k = i - r * ld, e = e0 + r, c = blk * bs + k;
    float acc = 0.f;
    if (e < E && k < bs) {
      acc = a.conv_bias[c];
      const int pos = st.start[e], t = st.cu[e];
      const float* ring = a.conv_state + (size_t)st.slot[e] * a.n_taps * W;
      for (int j = 0; j < a.n_taps; ++j)
        acc = fmaf(a.taps[(size_t)c * a.n_taps + j],
                   conv_input<T>(x0, a.yx_stride, ring, a.n_taps, W, t, 0, pos, a.n_taps - 1 - j, c), acc);
    }
    us[i] = from_f<T>(acc);
  }
  __syncthreads();
  const T* wr = static_cast<const T*>(a.gate_w) + (size_t)blk * 2 * bs * bs;
  const T* wi = wr + (size_t)bs * bs;
  if constexpr (sizeof(T) == 2) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int m0 = (warp >> 2) * 16;
    if (e0 + m0 >= E) return;
    const int n = o0 + (warp & 3) * 8 + gid;  // the channel whose weights this lane feeds
    const bool even = (bs & 1) == 0;
    const __nv_bfloat16* rr = reinterpret_cast<const __nv_bfloat16*>(wr) + (size_t)(n < bs ? n : 0) * bs;
    const __nv_bfloat16* ri = reinterpret_cast<const __nv_bfloat16*>(wi) + (size_t)(n < bs ? n : 0) * bs;
    const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(us) + (m0 + gid) * ld + tig * 2;
    float cr[4] = {0.f, 0.f, 0.f, 0.f}, ci[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int k = 0; k < bs; k += 16) {
      uint32_t A[4];
      A[0] = *reinterpret_cast<const uint32_t*>(up + k);
      A[1] = *reinterpret_cast<const uint32_t*>(up + 8 * ld + k);
      A[2] = *reinterpret_cast<const uint32_t*>(up + k + 8);
      A[3] = *reinterpret_cast<const uint32_t*>(up + 8 * ld + k + 8);
      const int kk = k + tig * 2;
      mma_bf16(cr, A, load_pair(rr, kk, bs, even), load_pair(rr, kk + 8, bs, even));
      mma_bf16(ci, A, load_pair(ri, kk, bs, even), load_pair(ri, kk + 8, bs, even));
    }
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int r = m0 + gid + (q >> 1) * 8, o = o0 + (warp & 3) * 8 + tig * 2 + (q & 1);
      if (e0 + r < E && o < bs) rglru_finish<T>(st, a, e0 + r, blk * bs + o, cr[q], ci[q], to_f<T>(us[r * ld + o]));
    }
  } else {
    for (int i = threadIdx.x; i < kStepEntries * kStepChannels; i += 256) {
      const int r = i / kStepChannels, o = o0 + i % kStepChannels;
      if (e0 + r >= E || o >= bs) continue;
      float sr = 0.f, si = 0.f;
      for (int k = 0; k < bs; ++k) {
        const float x = to_f<T>(us[r * ld + k]);
        sr = fmaf(to_f<T>(wr[(size_t)o * bs + k]), x, sr);
        si = fmaf(to_f<T>(wi[(size_t)o * bs + k]), x, si);
      }
      rglru_finish<T>(st, a, e0 + r, blk * bs + o, sr, si, to_f<T>(us[r * ld + o]));
    }
  }
}

// ---------------------------------------------------------------------------
// Linear attention with decay
// ---------------------------------------------------------------------------
// Token by token, the state in registers: a block owns 32 value columns of one (entry, head); warp w holds
// rows [w DR, (w + 1) DR) of the state.  The form for fp32 and for shapes the chunked kernel does not take.
constexpr int kSeqTokens = 16;

template <typename T, int DR>
__global__ void __launch_bounds__(256)
    lightning_seq_kernel(pace_step_t st, pace_lightning_args_t a) {
  extern __shared__ float smem[];
  const int d = a.dim, vd = a.vdim, H = a.heads, dp = 8 * DR;
  float* qs = smem;                       // [kSeqTokens][dp]
  float* ks = qs + kSeqTokens * dp;       // [kSeqTokens][dp]
  float* vs = ks + kSeqTokens * dp;       // [kSeqTokens][32]
  float* part = vs + kSeqTokens * 32;     // [kSeqTokens][8][32]
  const int e = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * 32;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, col = v0 + lane;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0;
  float* state = a.state + ((size_t)st.slot[e] * H + h) * d * vd;
  const float decay = a.decay[h];
  float S[DR];
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = warp * DR + i;
    S[i] = (st.start[e] != 0 && r < d && col < vd) ? state[(size_t)r * vd + col] : 0.f;
  }
  for (int l0 = 0; l0 < count; l0 += kSeqTokens) {
    const int n = min(kSeqTokens, count - l0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * dp; i += 256) {
      const int j = i / dp, r = i - j * dp;
      const T* row = static_cast<const T*>(a.qkv) + (size_t)(t0 + l0 + j) * a.qkv_stride + h * d;
      qs[i] = r < d ? round_to<T>(silu_t<T>(to_f<T>(row[r]))) : 0.f;
      ks[i] = r < d ? round_to<T>(silu_t<T>(to_f<T>(row[(size_t)H * d + r]))) : 0.f;
    }
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int j = i >> 5, c = v0 + (i & 31);
      const T* row = static_cast<const T*>(a.qkv) + (size_t)(t0 + l0 + j) * a.qkv_stride + 2 * (size_t)H * d + (size_t)h * vd;
      vs[i] = c < vd ? round_to<T>(silu_t<T>(to_f<T>(row[c]))) : 0.f;
    }
    __syncthreads();
    for (int j = 0; j < n; ++j) {
      const float v = vs[j * 32 + lane];
      const float *kr = ks + j * dp + warp * DR, *qr = qs + j * dp + warp * DR;
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DR; ++i) {
        S[i] = fmaf(decay, S[i], kr[i] * v);
        o = fmaf(S[i], qr[i], o);
      }
      part[(j * 8 + warp) * 32 + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int j = i >> 5, c = i & 31;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += part[(j * 8 + w) * 32 + c];
      if (v0 + c < vd) static_cast<T*>(a.out)[(size_t)(t0 + l0 + j) * H * vd + (size_t)h * vd + v0 + c] = from_f<T>(o);
    }
  }
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = warp * DR + i;
    if (r < d && col < vd) state[(size_t)r * vd + col] = S[i];
  }
}

// One token per entry: the state is read and written once.  A block owns 32 V value columns of one (entry,
// head); warp w takes rows w, w + 8, ...
template <typename T, int V>
__global__ void __launch_bounds__(256)
    lightning_step_kernel(pace_step_t st, pace_lightning_args_t a) {
  __shared__ float qs[512], ks[512];
  __shared__ float part[8][32 * V];
  const int e = blockIdx.z, h = blockIdx.y, d = a.dim, vd = a.vdim, H = a.heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, col = (blockIdx.x * 32 + lane) * V;
  const T* row = static_cast<const T*>(a.qkv) + (size_t)st.cu[e] * a.qkv_stride;
  const bool fresh = st.start[e] == 0;
  float* state = a.state + ((size_t)st.slot[e] * H + h) * d * vd;
  for (int i = threadIdx.x; i < d; i += 256) {
    qs[i] = round_to<T>(silu_t<T>(to_f<T>(row[(size_t)h * d + i])));
    ks[i] = round_to<T>(silu_t<T>(to_f<T>(row[(size_t)(H + h) * d + i])));
  }
  float v[V], o[V];
#pragma unroll
  for (int j = 0; j < V; ++j) {
    v[j] = col + j < vd ? round_to<T>(silu_t<T>(to_f<T>(row[2 * (size_t)H * d + (size_t)h * vd + col + j]))) : 0.f;
    o[j] = 0.f;
  }
  __syncthreads();
  const float decay = a.decay[h];
  if (col < vd) {
#pragma unroll 8
    for (int r = warp; r < d; r += 8) {
      float s[V];
      if (fresh) {
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] = 0.f;
      } else {
        Vec<float, V>::load(state + (size_t)r * vd + col, s);
      }
      const float k = ks[r], q = qs[r];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        s[j] = fmaf(decay, s[j], k * v[j]);
        o[j] = fmaf(s[j], q, o[j]);
      }
      Vec<float, V>::store(state + (size_t)r * vd + col, s);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) part[warp][lane * V + j] = o[j];
  __syncthreads();
  for (int i = threadIdx.x; i < 32 * V; i += 256) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += part[w][i];
    const int c = blockIdx.x * 32 * V + i;
    if (c < vd) static_cast<T*>(a.out)[(size_t)st.cu[e] * H * vd + (size_t)h * vd + c] = from_f<T>(s);
  }
}

template <typename T, int DR>
int launch_lightning_seq(const pace_step_t& st, const pace_lightning_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (2 * kSeqTokens * 8 * DR + kSeqTokens * 32 + kSeqTokens * 8 * 32);
  PACE_CUDA_TRY(cudaFuncSetAttribute(lightning_seq_kernel<T, DR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)((a.vdim + 31) / 32), (unsigned)a.heads, (unsigned)st.n_entries);
  lightning_seq_kernel<T, DR><<<grid, 256, smem, s>>>(st, a);
  PACE_LAUNCH_CHECK("lightning_seq_kernel");
  return PACE_OK;
}

template <typename T>
int lightning_seq(const pace_step_t& st, const pace_lightning_args_t& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_lightning_seq<T, 4>(st, a, s);
  if (a.dim <= 64) return launch_lightning_seq<T, 8>(st, a, s);
  if (a.dim <= 128) return launch_lightning_seq<T, 16>(st, a, s);
  if (a.dim <= 256) return launch_lightning_seq<T, 32>(st, a, s);
  return launch_lightning_seq<T, 64>(st, a, s);
}

template <typename T, int V>
int launch_lightning_step(const pace_step_t& st, const pace_lightning_args_t& a, cudaStream_t s) {
  const dim3 grid((unsigned)((a.vdim + 32 * V - 1) / (32 * V)), (unsigned)a.heads, (unsigned)st.n_entries);
  lightning_step_kernel<T, V><<<grid, 256, 0, s>>>(st, a);
  PACE_LAUNCH_CHECK("lightning_step_kernel");
  return PACE_OK;
}

template <typename T>
int lightning_step_t(const pace_step_t& st, const pace_lightning_args_t& a, cudaStream_t s) {
  if (a.vdim % 4 == 0 && a.vdim >= 128 && aligned16(a.state)) return launch_lightning_step<T, 4>(st, a, s);
  if (a.vdim % 2 == 0 && a.vdim >= 64 && aligned16(a.state)) return launch_lightning_step<T, 2>(st, a, s);
  return launch_lightning_step<T, 1>(st, a, s);
}

template <typename T>
int causal_conv_t(const pace_step_t& st, const void* in, int64_t is, const float* taps, const float* bias, int n_taps,
                  const float* cs, void* out, int channels, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = channels % V == 0 && is % V == 0 && aligned16(in) && aligned16(out) && aligned16(bias) && aligned16(cs);
  const size_t groups = (size_t)st.n_tokens * (channels / (vec ? V : 1));
  size_t blocks = (groups + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (vec)
    causal_conv_kernel<T, V><<<(unsigned)blocks, 256, 0, s>>>(st, (const T*)in, is, taps, bias, n_taps, cs, (T*)out, channels);
  else
    causal_conv_kernel<T, 1><<<(unsigned)blocks, 256, 0, s>>>(st, (const T*)in, is, taps, bias, n_taps, cs, (T*)out, channels);
  PACE_LAUNCH_CHECK("causal_conv_kernel");
  return PACE_OK;
}

template <typename T>
int rglru_step_t(const pace_step_t& st, const pace_rglru_args_t& a, cudaStream_t s) {
  const int bs = a.width / a.blocks, slices = (bs + kStepChannels - 1) / kStepChannels;
  const int ld = sizeof(T) == 2 ? (bs + 15) / 16 * 16 + 8 : bs;
  const size_t smem = (size_t)kStepEntries * ld * sizeof(T);
  if (smem > 200 * 1024) return PACE_ERR_UNSUPPORTED;
  PACE_CUDA_TRY(cudaFuncSetAttribute(rglru_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)(a.blocks * slices), (unsigned)((st.n_entries + kStepEntries - 1) / kStepEntries));
  rglru_step_kernel<T><<<grid, 256, smem, s>>>(st, a, slices, ld);
  PACE_LAUNCH_CHECK("rglru_step_kernel");
  return PACE_OK;
}

bool dtype_ok(int dtype) { return dtype == PACE_DTYPE_BF16 || dtype == PACE_DTYPE_FP32; }
bool rglru_ok(const pace_step_t* st, const pace_rglru_args_t* a) {
  return step_ok(st) && a && a->yx && a->ra_bias && a->ri_bias && a->decay_base && a->state && a->conv_state && a->out &&
         a->width > 0 && a->blocks > 0 && a->width % a->blocks == 0 && a->n_taps > 0 && a->yx_stride >= 2 * (int64_t)a->width &&
         dtype_ok(a->dtype);
}
bool lightning_ok(const pace_step_t* st, const pace_lightning_args_t* a) {
  return step_ok(st) && a && a->qkv && a->decay && a->state && a->out && a->heads > 0 && a->dim > 0 && a->vdim > 0 &&
         dtype_ok(a->dtype);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_causal_conv(const pace_step_t* st, const void* in, int64_t is, const float* taps, const float* bias, int32_t n_taps,
                     const float* cs, void* out, int32_t channels, int32_t dtype, void* stream) {
  if (!step_ok(st) || !in || !taps || !bias || !cs || !out || n_taps < 1 || channels < 1 || !dtype_ok(dtype))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("causal_conv", stream, "tokens=%d channels=%d", st->n_tokens, channels);
  return dtype == PACE_DTYPE_BF16
             ? causal_conv_t<__nv_bfloat16>(*st, in, is, taps, bias, n_taps, cs, out, channels, (cudaStream_t)stream)
             : causal_conv_t<float>(*st, in, is, taps, bias, n_taps, cs, out, channels, (cudaStream_t)stream);
}

int pace_rglru_scan(const pace_step_t* st, const pace_rglru_args_t* a, void* stream) {
  if (!rglru_ok(st, a) || !a->u || !a->gates) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("rglru_scan", stream, "entries=%d tokens=%d width=%d", st->n_entries, st->n_tokens, a->width);
  const dim3 grid((unsigned)((a->width + 31) / 32), (unsigned)st->n_entries);
  if (a->dtype == PACE_DTYPE_BF16)
    rglru_scan_kernel<__nv_bfloat16><<<grid, 32 * kSegs, 0, (cudaStream_t)stream>>>(*st, *a);
  else
    rglru_scan_kernel<float><<<grid, 32 * kSegs, 0, (cudaStream_t)stream>>>(*st, *a);
  PACE_LAUNCH_CHECK("rglru_scan_kernel");
  return PACE_OK;
}

int pace_rglru_step(const pace_step_t* st, const pace_rglru_args_t* a, void* stream) {
  if (!rglru_ok(st, a) || !a->gate_w || !a->taps || !a->conv_bias || st->n_tokens != st->n_entries) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("rglru_step", stream, "entries=%d width=%d", st->n_entries, a->width);
  return a->dtype == PACE_DTYPE_BF16 ? rglru_step_t<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : rglru_step_t<float>(*st, *a, (cudaStream_t)stream);
}

int pace_lightning_prefill(const pace_step_t* st, const pace_lightning_args_t* a, void* stream) {
  if (!lightning_ok(st, a)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("lightning_prefill", stream, "entries=%d tokens=%d heads=%d", st->n_entries, st->n_tokens, a->heads);
  return a->dtype == PACE_DTYPE_BF16 ? lightning_seq<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : lightning_seq<float>(*st, *a, (cudaStream_t)stream);
}

int pace_lightning_step(const pace_step_t* st, const pace_lightning_args_t* a, void* stream) {
  if (!lightning_ok(st, a) || st->n_tokens != st->n_entries) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (a->dim > 512 || a->heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("lightning_step", stream, "entries=%d heads=%d", st->n_entries, a->heads);
  return a->dtype == PACE_DTYPE_BF16 ? lightning_step_t<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : lightning_step_t<float>(*st, *a, (cudaStream_t)stream);
}

}  // extern "C"
