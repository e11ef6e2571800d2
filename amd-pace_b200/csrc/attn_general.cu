// Causal softmax attention over the paged pool on the CUDA cores, for rows the tensor-core kernels do not
// take: fp32 caches, head sizes beyond 128, any pair of key and value sizes up to 512.
//
// A thread block owns 32 query rows (token, grouped head) of one (sequence, KV head); its eight warps hold
// four rows each.  Keys and values pass through shared memory 32 at a time: a lane scores one key for its
// warp's rows, then owns value columns while the weights are passed round by shuffles.  Online softmax,
// everything in fp32.
#include "hybrid.cuh"

namespace pace {
namespace {

constexpr int kRows = 32, kKeys = 32, kRowsPerWarp = 4, kThreads = 256;

template <typename T, int VI>  // VI: value columns per lane
__global__ void __launch_bounds__(kThreads)
    attn_general_kernel(KVView kv, pace_step_t st, const T* __restrict__ q, T* __restrict__ out, int H, int d, int vd, int row,
                        float scale) {
  extern __shared__ float smem[];
  const int e = blockIdx.z, g = blockIdx.y;
  const int Gq = H / kv.n_kv_heads;
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0, start = st.start[e];
  const int r0 = blockIdx.x * kRows;
  if (r0 >= count * Gq) return;
  const int slot = st.slot[e];
  if (slot < 0 || slot >= kv.max_seqs) {
    if (threadIdx.x == 0) raise_status(kv.status, PACE_DEV_BAD_INDEX);
    return;
  }
  const int ks_ld = d | 1;
  float* qs = smem;                      // [kRows][d]
  float* ks = qs + kRows * d;            // [kKeys][ks_ld]
  float* vs = ks + kKeys * ks_ld;        // [kKeys][vd]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;

  for (int i = tid; i < kRows * d; i += kThreads) {
    const int r = i / d, c = i - r * d;
    float v = 0.f;
    if (r0 + r < count * Gq) {
      const int tok = (r0 + r) / Gq, hh = g * Gq + (r0 + r) % Gq;
      v = to_f<T>(q[((size_t)st.q_row[t0 + tok] * H + hh) * row + c]);
    }
    qs[i] = v;
  }
  int last[kRowsPerWarp];  // last visible position of the warp's rows, -1 for rows that do not exist
  float m[kRowsPerWarp], l[kRowsPerWarp], acc[kRowsPerWarp][VI];
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) {
    const int rr = r0 + warp * kRowsPerWarp + r;
    last[r] = rr < count * Gq ? start + rr / Gq : -1;
    m[r] = -INFINITY;
    l[r] = 0.f;
#pragma unroll
    for (int i = 0; i < VI; ++i) acc[r][i] = 0.f;
  }
  const int r_end = min(r0 + kRows, count * Gq) - 1;
  const int n_keys = start + r_end / Gq + 1;
  for (int k0 = 0; k0 < n_keys; k0 += kKeys) {
    __syncthreads();
    for (int i = tid; i < kKeys * (d + vd); i += kThreads) {
      const bool is_v = i >= kKeys * d;
      const int w = is_v ? vd : d, o = is_v ? i - kKeys * d : i;
      const int j = o / w, c = o - j * w, pos = k0 + j;
      float v = 0.f;
      if (pos < n_keys) {
        const int lp = pos / kv.page_tokens;
        const int pg = view_page(kv, slot, lp);
        if (pg >= 0)
          v = to_f<T>((reinterpret_cast<const T*>(is_v ? kv.v : kv.k))[(((size_t)pg * kv.n_kv_heads + g) * kv.page_tokens +
                                                                       (pos - lp * kv.page_tokens)) * row + c]);
        else
          raise_status(kv.status, PACE_DEV_BAD_INDEX);
      }
      if (is_v) vs[j * vd + c] = v; else ks[j * ks_ld + c] = v;
    }
    __syncthreads();
    float s[kRowsPerWarp] = {0.f, 0.f, 0.f, 0.f};
    const float* kr = ks + lane * ks_ld;
    const float* qr = qs + warp * kRowsPerWarp * d;
    for (int c = 0; c < d; ++c) {
      const float x = kr[c];
#pragma unroll
      for (int r = 0; r < kRowsPerWarp; ++r) s[r] = fmaf(qr[r * d + c], x, s[r]);
    }
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; ++r) {
      if (last[r] < k0) continue;  // (the warp's rows agree: lanes differ in the key only)
      float x = k0 + lane <= last[r] ? s[r] * scale : -INFINITY;
      float mx = x;
#pragma unroll
      for (int o = 16; o; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      mx = fmaxf(mx, m[r]);
      const float p = expf(x - mx);
      float sum = p;
#pragma unroll
      for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      const float f = expf(m[r] - mx);
      m[r] = mx;
      l[r] = l[r] * f + sum;
#pragma unroll
      for (int i = 0; i < VI; ++i) acc[r][i] *= f;
      for (int j = 0; j < kKeys; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
#pragma unroll
        for (int i = 0; i < VI; ++i) {
          const int c = lane + 32 * i;
          if (c < vd) acc[r][i] = fmaf(pj, vs[j * vd + c], acc[r][i]);
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) {
    const int rr = r0 + warp * kRowsPerWarp + r;
    if (last[r] < 0) continue;
    const int tok = rr / Gq, hh = g * Gq + rr % Gq;
    T* o = out + ((size_t)st.q_row[t0 + tok] * H + hh) * row;
#pragma unroll
    for (int i = 0; i < VI; ++i) {
      const int c = lane + 32 * i;
      if (c < vd) o[c] = from_f<T>(acc[r][i] / l[r]);
    }
  }
}

template <typename T, int VI>
int launch_general(const KVView& kv, const pace_step_t& st, const void* q, void* out, int H, int d, int vd, int row,
                   float scale, cudaStream_t s) {
  const size_t smem = sizeof(float) * ((size_t)kRows * d + (size_t)kKeys * (d | 1) + (size_t)kKeys * vd);
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_general_kernel<T, VI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const int Gq = H / kv.n_kv_heads;
  const dim3 grid((unsigned)((st.max_count * Gq + kRows - 1) / kRows), (unsigned)kv.n_kv_heads, (unsigned)st.n_entries);
  attn_general_kernel<T, VI><<<grid, kThreads, smem, s>>>(kv, st, (const T*)q, (T*)out, H, d, vd, row, scale);
  PACE_LAUNCH_CHECK("attn_general_kernel");
  return PACE_OK;
}

template <typename T>
int general_t(const KVView& kv, const pace_step_t& st, const void* q, void* out, int H, int d, int vd, int row, float scale,
              cudaStream_t s) {
  if (vd <= 32) return launch_general<T, 1>(kv, st, q, out, H, d, vd, row, scale, s);
  if (vd <= 64) return launch_general<T, 2>(kv, st, q, out, H, d, vd, row, scale, s);
  if (vd <= 128) return launch_general<T, 4>(kv, st, q, out, H, d, vd, row, scale, s);
  if (vd <= 256) return launch_general<T, 8>(kv, st, q, out, H, d, vd, row, scale, s);
  return launch_general<T, 16>(kv, st, q, out, H, d, vd, row, scale, s);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" int pace_attn_general(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const void* q, void* out,
                                 int32_t H, int32_t d, int32_t vd, float scale, int32_t dtype, void* stream) {
  if (!p || !p->pages || !step_ok(st) || !q || !out || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (H < 1 || H % p->n_kv_heads || d < 1 || vd < 1 || st->max_count < 0) return PACE_ERR_INVALID;
  if (dtype != PACE_DTYPE_BF16 && dtype != PACE_DTYPE_FP32) return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_BF16 && dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  const int row = dtype == PACE_DTYPE_BF16 ? p->head_dim : p->head_dim / 2;
  if (d > row || vd > row) return PACE_ERR_INVALID;
  if (d > 512 || vd > 512 || p->n_kv_heads > 65535 || st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("attn_general", stream, "layer=%d entries=%d tokens=%d", layer, st->n_entries, st->n_tokens);
  const KVView kv = make_view(p, layer, nullptr);
  return dtype == PACE_DTYPE_BF16 ? general_t<__nv_bfloat16>(kv, *st, q, out, H, d, vd, row, scale, (cudaStream_t)stream)
                                  : general_t<float>(kv, *st, q, out, H, d, vd, row, scale, (cudaStream_t)stream);
}
