// Recurrent layers: short causal convolution, the real-gated linear recurrence (RG-LRU) and linear attention
// with a fixed decay per head.  States are fp32 and live in per-slot arrays; a sequence that starts at
// position 0 begins from zeros whatever its slot holds, so slots are reused without clearing them.
#include "hybrid.cuh"

namespace pace {
bool lightning_chunked_fits(const pace_lightning_args_t& a);   // lightning.cu
int lightning_chunked(const pace_step_t& st, const pace_lightning_args_t& a, cudaStream_t s);

namespace {

// ---------------------------------------------------------------------------
// causal depthwise convolution
// ---------------------------------------------------------------------------
// A thread takes V channels of kConvTokens consecutive rows: the taps are read once for all of them, a row's
// inputs come from the cache after their first use.
constexpr int kConvTokens = 4;

template <typename T, int V, int NT, bool SILU>   // NT: number of taps where it is known at compile time, else 0
__global__ void __launch_bounds__(256) causal_conv_kernel(pace_step_t st, pace_causal_conv_args_t a) {
  const T* __restrict__ in = static_cast<const T*>(a.in);
  const float *__restrict__ taps = a.taps, *__restrict__ conv_state = a.conv_state;
  T* __restrict__ out = static_cast<T*>(a.out);
  const int channels = a.channels, n_taps = a.n_taps;
  const int64_t in_stride = a.in_stride;
  auto start_from = [&](int c, float* v) {
    if (a.bias) Vec<float, V>::load(a.bias + c, v);
    else
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = 0.f;
  };
  auto finish = [&](float* v, T* dst) {
    if constexpr (SILU) {
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = silu_t<T>(v[j]);
    }
    Vec<T, V>::store(dst, v);
  };
  const int per = channels / V;
  const size_t total = (size_t)((st.n_tokens + kConvTokens - 1) / kConvTokens) * per;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const int t0 = (int)(i / per) * kConvTokens, c = (int)(i % per) * V;
    float acc[kConvTokens][V];
    if constexpr (NT > 0) {
      // the usual place: four tokens of one entry with all their inputs among the step's rows
      const int tl = min(t0 + kConvTokens, st.n_tokens) - 1, e = st.tok_entry[tl];
      if (tl - t0 == kConvTokens - 1 && t0 - (NT - 1) >= st.cu[e]) {
        float x[kConvTokens + NT - 1][V];
        const T* row = in + (size_t)(t0 - (NT - 1)) * in_stride + c;
#pragma unroll
        for (int r = 0; r < kConvTokens + NT - 1; ++r, row += in_stride) Vec<T, V>::load(row, x[r]);
        float b[V];
        start_from(c, b);
#pragma unroll
        for (int r = 0; r < kConvTokens; ++r)
#pragma unroll
          for (int v = 0; v < V; ++v) acc[r][v] = b[v];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          float w[V];
          Vec<float, V>::load(taps + (size_t)j * channels + c, w);
#pragma unroll
          for (int r = 0; r < kConvTokens; ++r)
#pragma unroll
            for (int v = 0; v < V; ++v) acc[r][v] = fmaf(w[v], x[r + j][v], acc[r][v]);
        }
#pragma unroll
        for (int r = 0; r < kConvTokens; ++r) finish(acc[r], out + (size_t)(t0 + r) * a.out_stride + c);
        continue;
      }
    }
    int local[kConvTokens], pos[kConvTokens];
    const float* ring[kConvTokens];
#pragma unroll
    for (int r = 0; r < kConvTokens; ++r) {
      const int t = min(t0 + r, st.n_tokens - 1), e = st.tok_entry[t];
      local[r] = t - st.cu[e];
      pos[r] = st.tok_pos[t];
      ring[r] = conv_state + (size_t)st.slot[e] * a.ring_rows * a.ring_stride + c;
      start_from(c, acc[r]);
    }
    for (int j = 0; j < n_taps; ++j) {
      const int back = n_taps - 1 - j;
      float w[V];
      Vec<float, V>::load(taps + (size_t)j * channels + c, w);
#pragma unroll
      for (int r = 0; r < kConvTokens; ++r) {
        const int t = min(t0 + r, st.n_tokens - 1);
        float x[V];
        if (local[r] >= back) Vec<T, V>::load(in + (size_t)(t - back) * in_stride + c, x);
        else if (pos[r] >= back) Vec<float, V>::load(ring[r] + (size_t)((pos[r] - back) % a.ring_rows) * a.ring_stride, x);
        else continue;                                     // in front of the sequence
#pragma unroll
        for (int v = 0; v < V; ++v) acc[r][v] = fmaf(w[v], x[v], acc[r][v]);
      }
    }
#pragma unroll
    for (int r = 0; r < kConvTokens; ++r)
      if (t0 + r < st.n_tokens) finish(acc[r], out + (size_t)(t0 + r) * a.out_stride + c);
  }
}

// The newest inputs of every entry into its ring, behind the kernels that still read the older ones.
template <typename T>
__global__ void conv_store_kernel(pace_step_t st, const T* __restrict__ in, int64_t in_stride, float* __restrict__ ring, int rows,
                                  int ring_stride, int channels) {
  const int e = blockIdx.y, count = st.cu[e + 1] - st.cu[e], n = min(count, rows);
  float* dst = ring + (size_t)st.slot[e] * rows * ring_stride;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n * channels; i += gridDim.x * blockDim.x) {
    const int j = i / channels, c = i - j * channels, l = count - 1 - j;
    dst[(size_t)((st.start[e] + l) % rows) * ring_stride + c] = to_f<T>(in[(size_t)(st.cu[e] + l) * in_stride + c]);
  }
}

// ---------------------------------------------------------------------------
// RG-LRU over any number of tokens: gates and convolution come from launches in front
// ---------------------------------------------------------------------------
constexpr int kSegs = 8, kSegTokens = 8, kTile = kSegs * kSegTokens;

// coefficients of S_t = a S_(t-1) + b for pre-activations of the two gates
template <typename T>
__device__ __forceinline__ void rglru_coefficients(float r_pre, float i_pre, float u, float decay_base, float& a, float& b) {
  const float log_a = decay_base * sigmoid_t<T>(r_pre);
  a = exp_t<T>(log_a);
  b = sqrt_one_minus_exp<T>(2.0f * log_a, a * a) * sigmoid_t<T>(i_pre) * u;
}

// The blocks of a cluster walk 32 channels of one entry together: tiles of 64 tokens go round the cluster, in a
// block warp = a segment of 8 tokens, lane = a channel.  A thread composes its 8 steps into one affine map; the
// maps of a tile meet in shared memory, their products in the shared memory of every block of the cluster; then
// each thread replays its 8 steps from the state in front of them.  The next tile's operands are on their way
// meanwhile.  All blocks of a cluster take the same number of rounds.
constexpr int kMaxCluster = 4;

template <typename T>
__global__ void __launch_bounds__(32 * kSegs, 2)
    rglru_scan_kernel(pace_step_t st, pace_rglru_args_t a) {
  __shared__ float2 maps[2][kSegs][32];
  __shared__ float2 tiles_map[2][kMaxCluster][32];   // the round's tiles, written by the cluster's blocks
  uint32_t rank, n_rank;
  asm("mov.u32 %0, %%cluster_ctarank;" : "=r"(rank));
  asm("mov.u32 %0, %%cluster_nctarank;" : "=r"(n_rank));
  const int e = blockIdx.z, lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int W = a.width, c = blockIdx.y * 32 + lane;
  const bool live = c < W;
  const int cc = live ? c : 0;
  const int bs = W / a.blocks, blk = cc / bs, in_blk = cc - blk * bs;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0, start = st.start[e], slot = st.slot[e];
  const T* u = static_cast<const T*>(a.u) + (size_t)t0 * W + cc;
  const T* yx = static_cast<const T*>(a.yx) + (size_t)t0 * a.yx_stride + cc;
  const float* gr = a.gates + ((size_t)blk * st.n_tokens + t0) * 2 * bs + in_blk;
  T* out = static_cast<T*>(a.out) + (size_t)t0 * W + cc;
  const float rb = a.ra_bias[cc], ib = a.ri_bias[cc], base = a.decay_base[cc];
  float* state = a.state + (size_t)slot * W + cc;
  float carry = start == 0 ? 0.f : *state;

  float g0[kSegTokens], g1[kSegTokens];
  T uu[kSegTokens], yy[kSegTokens];
  auto fetch = [&](int l0) {
    // (rows behind the end are read from its last row and not used)
    const int from = min(l0, count - 1);
    const float* gp = gr + (size_t)from * 2 * bs;
    const T *up = u + (size_t)from * W, *yp = yx + (size_t)from * a.yx_stride;
    if (l0 + kSegTokens <= count) {
#pragma unroll
      for (int j = 0; j < kSegTokens; ++j) {
        g0[j] = gp[0];
        g1[j] = gp[bs];
        uu[j] = *up;
        yy[j] = *yp;
        gp += 2 * bs;
        up += W;
        yp += a.yx_stride;
      }
    } else {
#pragma unroll
      for (int j = 0; j < kSegTokens; ++j) {
        const int l = min(l0 + j, count - 1);
        g0[j] = gr[(size_t)l * 2 * bs];
        g1[j] = gr[(size_t)l * 2 * bs + bs];
        uu[j] = u[(size_t)l * W];
        yy[j] = yx[(size_t)l * a.yx_stride];
      }
    }
  };
  const int stride = kTile * (int)n_rank;
  int l0 = (int)rank * kTile + seg * kSegTokens;
  fetch(l0);
  const int rounds = (count + stride - 1) / stride;
  if (n_rank > 1) {                                  // every block of the cluster runs before anyone writes into it
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  }
  for (int round = 0; round < rounds; ++round, l0 += stride) {
    float ca[kSegTokens], cb[kSegTokens], A = 1.f, B = 0.f;
    T y[kSegTokens];
#pragma unroll
    for (int j = 0; j < kSegTokens; ++j) {
      rglru_coefficients<T>(g0[j] + rb, g1[j] + ib, to_f<T>(uu[j]), base, ca[j], cb[j]);
      if (l0 + j >= count) ca[j] = 1.f, cb[j] = 0.f;
      y[j] = yy[j];
      A *= ca[j];
      B = fmaf(ca[j], B, cb[j]);
    }
    if (round + 1 < rounds) fetch(l0 + stride);
    const int buf = round & 1;
    maps[buf][seg][lane] = make_float2(A, B);
    __syncthreads();
    // the map of the segments in front, and the tile's
    float fa = 1.f, fb = 0.f, ma = 1.f, mb = 0.f;
#pragma unroll
    for (int k = 0; k < kSegs; ++k) {
      if (k == seg) ma = fa, mb = fb;
      const float2 m = maps[buf][k][lane];
      fb = fmaf(m.x, fb, m.y);
      fa *= m.x;
    }
    float mine;
    if (n_rank == 1) {
      mine = fmaf(ma, carry, mb);
      carry = fmaf(fa, carry, fb);
    } else {
      if (seg < (int)n_rank) {                       // warp k sends the tile's map to block k
        uint32_t addr;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;"
                     : "=r"(addr) : "r"(smem_u32(&tiles_map[buf][rank][lane])), "r"((uint32_t)seg));
        asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(addr), "f"(fa), "f"(fb) : "memory");
      }
      asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
      asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      float s = carry;
      for (int k = 0; k < (int)n_rank; ++k) {
        if (k == (int)rank) mine = fmaf(ma, s, mb);
        const float2 m = tiles_map[buf][k][lane];
        s = fmaf(m.x, s, m.y);
      }
      carry = s;
    }
    if (live) {
      T* o = out + (size_t)l0 * W;
      if (l0 + kSegTokens <= count) {
#pragma unroll
        for (int j = 0; j < kSegTokens; ++j, o += W) {
          mine = fmaf(ca[j], mine, cb[j]);
          *o = from_f<T>(mine * gelu_tanh_t<T>(to_f<T>(y[j])));
        }
      } else {
#pragma unroll
        for (int j = 0; j < kSegTokens; ++j, o += W) {
          mine = fmaf(ca[j], mine, cb[j]);
          if (l0 + j < count) *o = from_f<T>(mine * gelu_tanh_t<T>(to_f<T>(y[j])));
        }
      }
    }
  }
  // (a block's last sends were received in front of the last barrier: nobody writes into a block that has left)
  if (!live || rank != 0) return;
  if (seg == 0) *state = carry;
  for (int j = seg; j < a.n_taps && j < count; j += kSegs) {
    const int l = count - 1 - j;
    a.conv_state[((size_t)slot * a.n_taps + (start + l) % a.n_taps) * W + c] = to_f<T>(yx[(size_t)l * a.yx_stride + W]);
  }
}

template <typename T>
int launch_rglru_scan(const pace_step_t& st, const pace_rglru_args_t& a, cudaStream_t s) {
  const int groups = (a.width + 31) / 32;
  int cluster = 1;                                   // blocks that share an entry's tiles, while the GPU has room for them
  while (cluster < kMaxCluster && cluster * 2 * kTile <= st.max_count && (int64_t)groups * st.n_entries * cluster * 2 <= 296)
    cluster *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)cluster, (unsigned)groups, (unsigned)st.n_entries);
  cfg.blockDim = dim3(32 * kSegs);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)cluster;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  PACE_CUDA_TRY(cudaLaunchKernelEx(&cfg, rglru_scan_kernel<T>, st, a));
  PACE_LAUNCH_CHECK("rglru_scan_kernel");
  return PACE_OK;
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

// The operands of one (entry, channel) besides the gates' sums, fetched before they are needed.
struct StepOperands {
  float y, x, state, ra, ri, base;
};
template <typename T>
__device__ __forceinline__ StepOperands rglru_operands(const pace_rglru_args_t& a, int row, int pos, int slot, int c) {
  const T* in = static_cast<const T*>(a.yx) + (size_t)row * a.yx_stride + c;
  StepOperands o;
  o.y = to_f<T>(in[0]);
  o.x = to_f<T>(in[a.width]);
  o.state = pos == 0 ? 0.f : a.state[(size_t)slot * a.width + c];
  o.ra = a.ra_bias[c];
  o.ri = a.ri_bias[c];
  o.base = a.decay_base[c];
  return o;
}
template <typename T>
__device__ __forceinline__ void rglru_finish(const pace_rglru_args_t& a, const StepOperands& o, int row, int pos, int slot, int c,
                                             float r_pre, float i_pre, float u) {
  float ca, cb;
  rglru_coefficients<T>(r_pre + o.ra, i_pre + o.ri, u, o.base, ca, cb);
  const float S = fmaf(ca, o.state, cb);
  a.state[(size_t)slot * a.width + c] = S;
  a.conv_state[((size_t)slot * a.n_taps + pos % a.n_taps) * a.width + c] = o.x;
  static_cast<T*>(a.out)[(size_t)row * a.width + c] = from_f<T>(S * gelu_tanh_t<T>(o.y));
}

// Block (slice, batch tile): 32 output channels of one gate block for 32 entries.  The slice's gate weights and the
// convolved inputs of the whole gate block go to shared memory (V elements per access), then bf16: warp w multiplies
// entries [16 (w / 4), +16) with channels [8 (w % 4), +8) of both gates on the tensor cores (fp32 accumulators
// are the pre-activations); fp32: one thread per (entry, channel).
constexpr int kStepThreads = 512;

template <typename T, int V, int NT>   // NT: taps known at compile time (their inputs are fetched together), else 0
__global__ void __launch_bounds__(kStepThreads)
    rglru_step_kernel(pace_step_t st, pace_rglru_args_t a, int slices, int ld) {
  extern __shared__ __align__(16) char smem_raw[];
  __shared__ int row_of[kStepEntries], pos_of[kStepEntries], slot_of[kStepEntries];
  T* us = reinterpret_cast<T*>(smem_raw);  // [kStepEntries][ld]
  T* ws = us + kStepEntries * ld;          // [2][kStepChannels][ld]
  const int W = a.width, bs = W / a.blocks, tid = threadIdx.x;
  const int blk = blockIdx.x / slices, o0 = (blockIdx.x % slices) * kStepChannels;
  const int e0 = blockIdx.y * kStepEntries, n_e = min(kStepEntries, st.n_entries - e0);
  const int lv = ld / V;                   // vectors of a shared row
  const T* wg = static_cast<const T*>(a.gate_w) + (size_t)blk * 2 * bs * bs;
  for (int i = tid; i < 2 * kStepChannels * lv; i += kStepThreads) {
    const int r = i / lv, k = (i - r * lv) * V, o = o0 + (r & (kStepChannels - 1));
    const bool in = o < bs && k < bs;
    const T* src = wg + (in ? ((size_t)(r / kStepChannels) * bs + o) * bs + k : 0);
    if constexpr (V * sizeof(T) == 16) {
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(ws + r * ld + k)), "l"(src), "r"(in ? 16 : 0)
                   : "memory");
    } else {
      ws[r * ld + k] = in ? *src : from_f<T>(0.f);
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (tid < n_e) {
    row_of[tid] = st.cu[e0 + tid];
    pos_of[tid] = st.start[e0 + tid];
    slot_of[tid] = st.slot[e0 + tid];
  }
  __syncthreads();
  // bf16: the outputs of a multiplying lane, their operands on the way while the inputs are convolved
  const int warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3, m0 = ((warp >> 2) & 1) * 16;
  StepOperands ops[4];
  if constexpr (sizeof(T) == 2) {
    if (warp < 8) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int r = m0 + gid + (q >> 1) * 8, o = o0 + (warp & 3) * 8 + tig * 2 + (q & 1);
        if (r < n_e && o < bs) ops[q] = rglru_operands<T>(a, row_of[r], pos_of[r], slot_of[r], blk * bs + o);
      }
    }
  }
  const T* x0 = static_cast<const T*>(a.yx) + W;
  for (int i = tid; i < kStepEntries * lv; i += kStepThreads) {
    const int r = i / lv, k = (i - r * lv) * V, c = blk * bs + k;
    float acc[V];
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = 0.f;
    if (r < n_e && k < bs) {
      const int pos = pos_of[r];
      const T* now = x0 + (size_t)row_of[r] * a.yx_stride + c;
      const float* ring = a.conv_state + (size_t)slot_of[r] * a.n_taps * W + c;
      if constexpr (NT > 0) {
        float x[NT][V];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int back = NT - 1 - j;
          if (back == 0) Vec<T, V>::load(now, x[j]);
          else if (pos >= back) Vec<float, V>::load(ring + (size_t)((pos - back) % NT) * W, x[j]);
          else
#pragma unroll
            for (int v = 0; v < V; ++v) x[j][v] = 0.f;
        }
        Vec<float, V>::load(a.conv_bias + c, acc);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          float w[V];
          Vec<float, V>::load(a.taps + (size_t)j * W + c, w);
#pragma unroll
          for (int v = 0; v < V; ++v) acc[v] = fmaf(w[v], x[j][v], acc[v]);
        }
      } else {
        Vec<float, V>::load(a.conv_bias + c, acc);
        for (int j = 0; j < a.n_taps; ++j) {
          const int back = a.n_taps - 1 - j;
          if (pos < back) continue;
          float x[V], w[V];
          if (back == 0) Vec<T, V>::load(now, x);
          else Vec<float, V>::load(ring + (size_t)((pos - back) % a.n_taps) * W, x);
          Vec<float, V>::load(a.taps + (size_t)j * W + c, w);
#pragma unroll
          for (int v = 0; v < V; ++v) acc[v] = fmaf(w[v], x[v], acc[v]);
        }
      }
    }
    Vec<T, V>::store(us + r * ld + k, acc);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if constexpr (sizeof(T) == 2) {
    if (warp >= 8 || m0 >= n_e) return;
    const __nv_bfloat16* up = reinterpret_cast<const __nv_bfloat16*>(us) + (m0 + gid) * ld + tig * 2;
    const __nv_bfloat16* rp = reinterpret_cast<const __nv_bfloat16*>(ws) + ((warp & 3) * 8 + gid) * ld + tig * 2;
    const __nv_bfloat16* ip = rp + kStepChannels * ld;
    auto pair = [](const __nv_bfloat16* p) { return *reinterpret_cast<const uint32_t*>(p); };
    float cr[4] = {0.f, 0.f, 0.f, 0.f}, ci[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int k = 0; k < bs; k += 16) {
      const uint32_t A[4] = {pair(up + k), pair(up + 8 * ld + k), pair(up + k + 8), pair(up + 8 * ld + k + 8)};
      mma_bf16(cr, A, pair(rp + k), pair(rp + k + 8));
      mma_bf16(ci, A, pair(ip + k), pair(ip + k + 8));
    }
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int r = m0 + gid + (q >> 1) * 8, o = o0 + (warp & 3) * 8 + tig * 2 + (q & 1);
      if (r < n_e && o < bs)
        rglru_finish<T>(a, ops[q], row_of[r], pos_of[r], slot_of[r], blk * bs + o, cr[q], ci[q], to_f<T>(us[r * ld + o]));
    }
  } else {
    for (int i = tid; i < kStepEntries * kStepChannels; i += kStepThreads) {
      const int r = i / kStepChannels, oo = i % kStepChannels, o = o0 + oo, c = blk * bs + o;
      if (r >= n_e || o >= bs) continue;
      float sr = 0.f, si = 0.f;
      for (int k = 0; k < bs; ++k) {
        const float x = to_f<T>(us[r * ld + k]);
        sr = fmaf(to_f<T>(ws[oo * ld + k]), x, sr);
        si = fmaf(to_f<T>(ws[(kStepChannels + oo) * ld + k]), x, si);
      }
      rglru_finish<T>(a, rglru_operands<T>(a, row_of[r], pos_of[r], slot_of[r], c), row_of[r], pos_of[r], slot_of[r], c, sr, si,
                      to_f<T>(us[r * ld + o]));
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

template <typename T, bool SILU>
int causal_conv_t(const pace_step_t& st, const pace_causal_conv_args_t& a, cudaStream_t s) {
  constexpr int V = 8 / sizeof(T);      // (four bf16 or two fp32 channels: the window of rows stays in registers)
  const bool vec = a.channels % V == 0 && a.in_stride % V == 0 && a.out_stride % V == 0 && a.ring_stride % V == 0 &&
                   aligned16(a.in) && aligned16(a.out) && aligned16(a.bias) && aligned16(a.conv_state) && aligned16(a.taps);
  const size_t groups = (size_t)((st.n_tokens + kConvTokens - 1) / kConvTokens) * (a.channels / (vec ? V : 1));
  size_t blocks = (groups + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (vec && a.n_taps == 4) causal_conv_kernel<T, V, 4, SILU><<<(unsigned)blocks, 256, 0, s>>>(st, a);
  else if (vec) causal_conv_kernel<T, V, 0, SILU><<<(unsigned)blocks, 256, 0, s>>>(st, a);
  else causal_conv_kernel<T, 1, 0, SILU><<<(unsigned)blocks, 256, 0, s>>>(st, a);
  PACE_LAUNCH_CHECK("causal_conv_kernel");
  return PACE_OK;
}

template <typename T, int V, int NT>
int launch_rglru_step(const pace_step_t& st, const pace_rglru_args_t& a, int slices, int ld, size_t smem, cudaStream_t s) {
  PACE_CUDA_TRY(cudaFuncSetAttribute(rglru_step_kernel<T, V, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)(a.blocks * slices), (unsigned)((st.n_entries + kStepEntries - 1) / kStepEntries));
  rglru_step_kernel<T, V, NT><<<grid, kStepThreads, smem, s>>>(st, a, slices, ld);
  PACE_LAUNCH_CHECK("rglru_step_kernel");
  return PACE_OK;
}

template <typename T>
int rglru_step_t(const pace_step_t& st, const pace_rglru_args_t& a, cudaStream_t s) {
  const int bs = a.width / a.blocks, slices = (bs + kStepChannels - 1) / kStepChannels;
  const int ld = (bs + 15) / 16 * 16 + 16 / (int)sizeof(T);   // whole k steps of the tensor cores, rows 16 bytes apart
  const size_t smem = (size_t)(kStepEntries + 2 * kStepChannels) * ld * sizeof(T);
  if (smem > 200 * 1024) return PACE_ERR_UNSUPPORTED;
  constexpr int V = 16 / sizeof(T);
  const bool vec = bs % V == 0 && a.yx_stride % V == 0 && aligned16(a.yx) && aligned16(a.gate_w) && aligned16(a.taps) &&
                   aligned16(a.conv_bias) && aligned16(a.conv_state);
  if (vec && a.n_taps == 4) return launch_rglru_step<T, V, 4>(st, a, slices, ld, smem, s);
  return vec ? launch_rglru_step<T, V, 0>(st, a, slices, ld, smem, s) : launch_rglru_step<T, 1, 0>(st, a, slices, ld, smem, s);
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

int pace_causal_conv(const pace_step_t* st, const pace_causal_conv_args_t* a, void* stream) {
  if (!step_ok(st) || !a || !a->in || !a->taps || !a->conv_state || !a->out || a->n_taps < 1 || a->channels < 1 ||
      a->ring_rows < a->n_taps - 1 || a->ring_rows < 1 || a->ring_stride < a->channels || a->in_stride < a->channels ||
      a->out_stride < a->channels || !dtype_ok(a->dtype))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("causal_conv", stream, "tokens=%d channels=%d", st->n_tokens, a->channels);
  const cudaStream_t s = (cudaStream_t)stream;
  if (a->dtype == PACE_DTYPE_BF16)
    return a->silu ? causal_conv_t<__nv_bfloat16, true>(*st, *a, s) : causal_conv_t<__nv_bfloat16, false>(*st, *a, s);
  return a->silu ? causal_conv_t<float, true>(*st, *a, s) : causal_conv_t<float, false>(*st, *a, s);
}

int pace_conv_store(const pace_step_t* st, const void* in, int64_t in_stride, float* ring, int32_t ring_rows, int32_t ring_stride,
                    int32_t channels, int32_t dtype, void* stream) {
  if (!step_ok(st) || !in || !ring || ring_rows < 1 || channels < 1 || ring_stride < channels || in_stride < channels ||
      !dtype_ok(dtype))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  const int64_t n = (int64_t)(st->max_count < ring_rows ? st->max_count : ring_rows) * channels;
  const dim3 grid((unsigned)((n + 255) / 256 < 64 ? (n + 255) / 256 : 64), (unsigned)st->n_entries);
  if (dtype == PACE_DTYPE_BF16)
    conv_store_kernel<<<grid, 256, 0, (cudaStream_t)stream>>>(*st, (const __nv_bfloat16*)in, in_stride, ring, ring_rows, ring_stride, channels);
  else
    conv_store_kernel<<<grid, 256, 0, (cudaStream_t)stream>>>(*st, (const float*)in, in_stride, ring, ring_rows, ring_stride, channels);
  PACE_LAUNCH_CHECK("conv_store_kernel");
  return PACE_OK;
}

int pace_rglru_scan(const pace_step_t* st, const pace_rglru_args_t* a, void* stream) {
  if (!rglru_ok(st, a) || !a->u || !a->gates) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (st->n_entries > 65535 || a->width > 32 * 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("rglru_scan", stream, "entries=%d tokens=%d width=%d", st->n_entries, st->n_tokens, a->width);
  return a->dtype == PACE_DTYPE_BF16 ? launch_rglru_scan<__nv_bfloat16>(*st, *a, (cudaStream_t)stream)
                                     : launch_rglru_scan<float>(*st, *a, (cudaStream_t)stream);
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
  if (lightning_chunked_fits(*a)) return lightning_chunked(*st, *a, (cudaStream_t)stream);
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
