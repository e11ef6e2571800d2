// Causal softmax attention over the paged pool on the CUDA cores, for rows the tensor-core kernels do not
// take: fp32 caches, head sizes beyond 128, any pair of key and value sizes up to 640 and 512; with or without a span,
// a distance bias and a sink.
//
// A thread block owns 32 query rows (token, grouped head) of one (sequence, KV head); its eight warps hold
// four rows each.  Keys and values pass through shared memory 32 at a time: a lane scores one key for its
// warp's rows, then owns value columns while the weights are passed round by shuffles.  Online softmax,
// everything in fp32.
#include "span.cuh"

namespace pace {
namespace {

struct GeneralArgs {
  const void* q;
  void* out;
  const int32_t* rows;   // row of q and out of a token, nullptr: the token itself
  const float* slopes;
  const float* sinks;
  int H, d, vd, q_row, o_row, row;   // elements of a row of q, out and the pool
  int entry0, span, span_size;
  float scale, softcap;
  int64_t o_tok;         // elements between the rows of out
};

constexpr int kRows = 32, kKeys = 32, kRowsPerWarp = 4, kThreads = 256;

template <typename T, int VI>  // VI: value columns per lane
__global__ void __launch_bounds__(kThreads)
    attn_general_kernel(KVView kv, pace_step_t st, GeneralArgs a) {
  extern __shared__ float smem[];
  const T* __restrict__ q = static_cast<const T*>(a.q);
  T* __restrict__ out = static_cast<T*>(a.out);
  const int H = a.H, d = a.d, vd = a.vd, row = a.row;
  const int e = a.entry0 + blockIdx.z, g = blockIdx.y;
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
      v = to_f<T>(q[((size_t)(a.rows ? a.rows[t0 + tok] : t0 + tok) * H + hh) * a.q_row + c]);
    }
    qs[i] = v;
  }
  int last[kRowsPerWarp];   // last visible position of the warp's rows, -1 for rows that do not exist
  int first[kRowsPerWarp];  // first one
  float slope[kRowsPerWarp];
  float m[kRowsPerWarp], l[kRowsPerWarp], acc[kRowsPerWarp][VI];
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) {
    const int rr = r0 + warp * kRowsPerWarp + r;
    last[r] = rr < count * Gq ? start + rr / Gq : -1;
    first[r] = last[r] < 0 ? 0 : span_first(a.span, a.span_size, last[r]);
    slope[r] = (a.slopes && last[r] >= 0) ? a.slopes[g * Gq + rr % Gq] : 0.f;
    m[r] = -INFINITY;
    l[r] = 0.f;
#pragma unroll
    for (int i = 0; i < VI; ++i) acc[r][i] = 0.f;
  }
  const int r_end = min(r0 + kRows, count * Gq) - 1;
  const int n_keys = start + r_end / Gq + 1;
  for (int k0 = span_first(a.span, a.span_size, start + r0 / Gq) / kKeys * kKeys; k0 < n_keys; k0 += kKeys) {
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
      if (last[r] < k0 || first[r] >= k0 + kKeys) continue;  // (the warp's rows agree: lanes differ in the key only)
      const int pos = k0 + lane;
      float x = -INFINITY;
      if (pos <= last[r] && pos >= first[r]) {
        x = s[r] * a.scale;
        if (a.softcap > 0.f) x = a.softcap * tanhf(x / a.softcap);
        x += slope[r] * (float)(pos - last[r]);
      }
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
    if (a.sinks) {  // one more term of the denominator
      const float sink = a.sinks[hh], mx = fmaxf(m[r], sink), f = expf(m[r] - mx);
      l[r] = l[r] * f + expf(sink - mx);
#pragma unroll
      for (int i = 0; i < VI; ++i) acc[r][i] *= f;
    }
    T* o = out + (a.rows ? a.rows[t0 + tok] : t0 + tok) * a.o_tok + (int64_t)hh * a.o_row;
#pragma unroll
    for (int i = 0; i < VI; ++i) {
      const int c = lane + 32 * i;
      if (c < vd) o[c] = from_f<T>(acc[r][i] / l[r]);
    }
  }
}

template <typename T, int VI>
int launch_general(const KVView& kv, const pace_step_t& st, const GeneralArgs& a, int entries, int max_tokens, cudaStream_t s) {
  const size_t smem = sizeof(float) * ((size_t)kRows * a.d + (size_t)kKeys * (a.d | 1) + (size_t)kKeys * a.vd);
  if (smem > 227 * 1024) return PACE_ERR_UNSUPPORTED;
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_general_kernel<T, VI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const int Gq = a.H / kv.n_kv_heads;
  const dim3 grid((unsigned)(((size_t)max_tokens * Gq + kRows - 1) / kRows), (unsigned)kv.n_kv_heads, (unsigned)entries);
  attn_general_kernel<T, VI><<<grid, kThreads, smem, s>>>(kv, st, a);
  PACE_LAUNCH_CHECK("attn_general_kernel");
  return PACE_OK;
}

template <typename T>
int general_t(const KVView& kv, const pace_step_t& st, const GeneralArgs& a, int entries, int max_tokens, cudaStream_t s) {
  if (a.vd <= 32) return launch_general<T, 1>(kv, st, a, entries, max_tokens, s);
  if (a.vd <= 64) return launch_general<T, 2>(kv, st, a, entries, max_tokens, s);
  if (a.vd <= 128) return launch_general<T, 4>(kv, st, a, entries, max_tokens, s);
  if (a.vd <= 256) return launch_general<T, 8>(kv, st, a, entries, max_tokens, s);
  return launch_general<T, 16>(kv, st, a, entries, max_tokens, s);
}

int general(const KVView& kv, const pace_step_t& st, const GeneralArgs& a, int entries, int max_tokens, int dtype, cudaStream_t s) {
  if (a.d > 640 || a.vd > 512 || kv.n_kv_heads > 65535 || entries > 65535) return PACE_ERR_UNSUPPORTED;
  return dtype == PACE_DTYPE_BF16 ? general_t<__nv_bfloat16>(kv, st, a, entries, max_tokens, s)
                                  : general_t<float>(kv, st, a, entries, max_tokens, s);
}

}  // namespace

int attn_general_span(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_attn_span_args_t& a,
                      cudaStream_t s) {
  GeneralArgs ga;
  ga.q = a.q;
  ga.out = a.out;
  ga.rows = nullptr;
  ga.slopes = a.slopes;
  ga.sinks = a.sinks;
  ga.H = a.n_q_heads;
  ga.d = a.dim;
  ga.vd = a.vdim;
  ga.q_row = a.q_elems;
  ga.o_row = a.out_elems;
  ga.row = a.dtype == PACE_DTYPE_BF16 ? p->head_dim : p->head_dim / 2;
  ga.entry0 = a.entry_begin;
  ga.span = a.span;
  ga.span_size = a.span_size;
  ga.scale = a.scale;
  ga.softcap = a.softcap;
  ga.o_tok = span_out_row(a);
  return general(make_view(p, layer, nullptr), st, ga, a.entry_end - a.entry_begin, a.max_tokens, a.dtype, s);
}

}  // namespace pace

using namespace pace;

extern "C" int pace_attn_general(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const void* q, void* out,
                                 int32_t H, int32_t d, int32_t vd, float scale, int32_t dtype, void* stream) {
  if (!p || !p->pages || !step_ok(st) || !q || !out || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (H < 1 || H % p->n_kv_heads || d < 1 || vd < 1 || st->max_count < 0) return PACE_ERR_INVALID;
  if (dtype != PACE_DTYPE_BF16 && dtype != PACE_DTYPE_FP32) return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_BF16 && dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  GeneralArgs ga;
  ga.row = ga.q_row = ga.o_row = dtype == PACE_DTYPE_BF16 ? p->head_dim : p->head_dim / 2;
  if (d > ga.row || vd > ga.row) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("attn_general", stream, "layer=%d entries=%d tokens=%d", layer, st->n_entries, st->n_tokens);
  ga.q = q;
  ga.out = out;
  ga.rows = st->q_row;
  ga.slopes = ga.sinks = nullptr;
  ga.H = H;
  ga.d = d;
  ga.vd = vd;
  ga.entry0 = 0;
  ga.span = PACE_SPAN_ALL;
  ga.span_size = 0;
  ga.scale = scale;
  ga.softcap = 0.f;
  ga.o_tok = (int64_t)H * ga.o_row;
  return general(make_view(p, layer, nullptr), *st, ga, st->n_entries, st->max_count, dtype, (cudaStream_t)stream);
}
