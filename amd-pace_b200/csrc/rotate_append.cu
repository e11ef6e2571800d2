// Projections on their way to attention without norms: rotation of queries and keys (pairs of neighbours or of the two halves),
// queries to the staging rows, keys and values to their pages, and the means of whole blocks of cached rows to the pages of a pool
// of blocks.  fp32 arithmetic, a thread per vector of a head row.
#include "hybrid.cuh"

namespace pace {
namespace {

constexpr int kThreads = 256;

// the row of block `b` of a sequence: keys (plane 0) or values (plane 1) of KV head g, vector at c; null without a page
template <typename T>
__device__ __forceinline__ T* view_row(const KVView& kv, int slot, int index, bool is_v, int g, int row) {
  const int lp = index / kv.page_tokens, pg = slot >= 0 && slot < kv.max_seqs ? view_page(kv, slot, lp) : -1;
  if (pg < 0) {
    raise_status(kv.status, PACE_DEV_BAD_INDEX);
    return nullptr;
  }
  T* base = const_cast<T*>(reinterpret_cast<const T*>(is_v ? kv.v : kv.k));
  return base + (((size_t)pg * kv.n_kv_heads + g) * kv.page_tokens + (index - lp * kv.page_tokens)) * row;
}

// sum[] += the vectors at c of cached rows [first, first + n)
template <typename T, int V>
__device__ __forceinline__ void add_rows(const KVView& kv, int slot, int first, int n, bool is_v, int g, int row, int c, float* sum) {
  for (int i = 0; i < n;) {
    const T* r = view_row<T>(kv, slot, first + i, is_v, g, row);
    const int run = min(n - i, kv.page_tokens - (first + i) % kv.page_tokens);   // rows of one page
#pragma unroll 8
    for (int j = 0; j < run; ++j) {
      if (!r) break;
      float x[V];
      Vec<T, V>::load(r + (size_t)j * row + c, x);
#pragma unroll
      for (int k = 0; k < V; ++k) sum[k] += x[k];
    }
    i += run;
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(kThreads) append_rotate_kernel(pace_step_t st, KVView kv, KVView blocks, pace_append_rotate_args_t a, int row) {
  const int H = a.n_q_heads, G = kv.n_kv_heads, d = a.dim, vd = a.vdim, per = row / V, heads = H + 2 * G, half = a.rot_pairs;
  const size_t total = (size_t)st.n_tokens * heads * per;
  for (size_t i = blockIdx.x * (size_t)kThreads + threadIdx.x; i < total; i += (size_t)gridDim.x * kThreads) {
    const int c = (int)(i % per) * V, hh = (int)(i / per % heads), t = (int)(i / ((size_t)per * heads));
    const bool is_q = hh < H, is_v = hh >= H + G;
    const int g = is_q ? 0 : is_v ? hh - H - G : hh - H, n = is_v ? vd : d, pos = st.tok_pos[t];
    const T* src = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride + (is_q ? hh * d : is_v ? (H + G) * d + g * vd : H * d + g * d);
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = 0.f;
    if (c < n) Vec<T, V>::load(src + c, x);
    if (!is_v && c < 2 * half) {
      if (pos >= a.table_rows) {
        raise_status(kv.status, PACE_DEV_BAD_INDEX);
      } else if (a.halves) {                     // (V divides the number of pairs: a vector lies in one half)
        const bool second = c >= half;
        const int p = second ? c - half : c;
        float y[V], cs[V], sn[V];
        Vec<T, V>::load(src + (second ? p : p + half), y);
        Vec<float, V>::load(a.cos_table + (size_t)pos * half + p, cs);
        Vec<float, V>::load(a.sin_table + (size_t)pos * half + p, sn);
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] = second ? x[j] * cs[j] + y[j] * sn[j] : x[j] * cs[j] - y[j] * sn[j];
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const int p = (c + j) >> 1;
          const float y = to_f<T>(src[(c + j) ^ 1]), cs = a.cos_table[(size_t)pos * half + p], sn = a.sin_table[(size_t)pos * half + p];
          x[j] = (c + j) & 1 ? x[j] * cs + y * sn : x[j] * cs - y * sn;
        }
      }
    }
    if (is_q) {
      Vec<T, V>::store(static_cast<T*>(a.q_out) + ((size_t)t * H + hh) * row + c, x);
      continue;
    }
    const int slot = st.slot[st.tok_entry[t]];
    T* dst = view_row<T>(kv, slot, pos, is_v, g, row);
    if (!dst) continue;
    Vec<T, V>::store(dst + c, x);
    if (a.block_now && (pos + 1) % a.block == 0) {      // the token completes a block, whose other rows are cached already
      float sum[V];
#pragma unroll
      for (int j = 0; j < V; ++j) sum[j] = 0.f;
      add_rows<T, V>(kv, slot, pos + 1 - a.block, a.block - 1, is_v, g, row, c, sum);
#pragma unroll
      for (int j = 0; j < V; ++j) sum[j] = (sum[j] + round_to<T>(x[j])) / (float)a.block;
      T* b = view_row<T>(blocks, slot, pos / a.block, is_v, g, row);
      if (b) Vec<T, V>::store(b + c, sum);
    }
  }
}

// Blocks whose last token belongs to the step: thread per (vector, KV head, plane), a grid row per (entry, block).
template <typename T, int V>
__global__ void __launch_bounds__(kThreads) block_means_kernel(pace_step_t st, KVView kv, KVView blocks, int block, int row) {
  const int e = blockIdx.y, start = st.start[e], end = start + st.cu[e + 1] - st.cu[e], b = start / block + blockIdx.x;
  if (b >= end / block) return;
  const int per = row / V, slot = st.slot[e];
  for (int i = threadIdx.x; i < 2 * kv.n_kv_heads * per; i += kThreads) {
    const int c = i % per * V, g = i / per % kv.n_kv_heads;
    const bool is_v = i >= kv.n_kv_heads * per;
    float sum[V];
#pragma unroll
    for (int j = 0; j < V; ++j) sum[j] = 0.f;
    add_rows<T, V>(kv, slot, b * block, block, is_v, g, row, c, sum);
#pragma unroll
    for (int j = 0; j < V; ++j) sum[j] /= (float)block;
    T* dst = view_row<T>(blocks, slot, b, is_v, g, row);
    if (dst) Vec<T, V>::store(dst + c, sum);
  }
}

template <typename T>
int append_rotate_t(const KVView& kv, const KVView& blocks, const pace_step_t& st, const pace_append_rotate_args_t& a, cudaStream_t s) {
  const int row = kv.head_dim * 2 / (int)sizeof(T);
  if (a.dim > row || a.vdim > row) return PACE_ERR_INVALID;
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.dim % V == 0 && a.vdim % V == 0 && row % V == 0 && a.qkv_stride % V == 0 && aligned16(a.qkv) && aligned16(a.q_out) &&
                   a.rot_pairs % V == 0 && aligned16(a.cos_table) && aligned16(a.sin_table);
  const size_t n = (size_t)st.n_tokens * (a.n_q_heads + 2 * kv.n_kv_heads) * (row / (vec ? V : 1));
  const unsigned grid = (unsigned)((n + kThreads - 1) / kThreads < 148 * 32 ? (n + kThreads - 1) / kThreads : 148 * 32);
  if (vec) append_rotate_kernel<T, V><<<grid, kThreads, 0, s>>>(st, kv, blocks, a, row);
  else append_rotate_kernel<T, 1><<<grid, kThreads, 0, s>>>(st, kv, blocks, a, row);
  PACE_LAUNCH_CHECK("append_rotate_kernel");
  if (a.block > 0 && !a.block_now) {
    const dim3 g2((unsigned)(st.max_count / a.block + 1), (unsigned)st.n_entries);
    if (row % V == 0) block_means_kernel<T, V><<<g2, kThreads, 0, s>>>(st, kv, blocks, a.block, row);
    else block_means_kernel<T, 1><<<g2, kThreads, 0, s>>>(st, kv, blocks, a.block, row);
    PACE_LAUNCH_CHECK("block_means_kernel");
  }
  note_pool_write(s);
  return PACE_OK;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" int pace_kv_append_rotate(const pace_kv_pool_t* p, int32_t layer, const pace_kv_pool_t* bp, int32_t block_layer,
                                     const pace_step_t* st, const pace_append_rotate_args_t* a, void* stream) {
  if (!p || !p->pages || !p->block_table || !step_ok(st) || !a || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (!a->qkv || !a->q_out || a->n_q_heads < 1 || a->dim < 1 || a->vdim < 1 || a->n_q_heads % p->n_kv_heads || a->rot_pairs < 0 ||
      2 * a->rot_pairs > a->dim || (a->rot_pairs > 0 && (!a->cos_table || !a->sin_table || a->table_rows < 1)) || a->block < 0 ||
      (a->dtype != PACE_DTYPE_BF16 && a->dtype != PACE_DTYPE_FP32) || (a->block_now && st->n_tokens != st->n_entries))
    return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_SHARED || row_tokens(*p) != 1) return PACE_ERR_UNSUPPORTED;
  if (p->row_format == PACE_ROWS_BF16 && a->dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  if (a->block > 0 && (!bp || !bp->pages || !bp->block_table || block_layer < 0 || block_layer >= bp->n_layers || row_tokens(*bp) != a->block ||
                       bp->n_kv_heads != p->n_kv_heads || bp->head_dim != p->head_dim || bp->row_format != p->row_format))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  if (st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  PACE_PROFILE("kv_append_rotate", stream, "layer=%d tokens=%d", layer, st->n_tokens);
  const KVView kv = make_view(p, layer, nullptr), blocks = a->block > 0 ? make_view(bp, block_layer, nullptr) : kv;
  return a->dtype == PACE_DTYPE_BF16 ? append_rotate_t<__nv_bfloat16>(kv, blocks, *st, *a, (cudaStream_t)stream)
                                     : append_rotate_t<float>(kv, blocks, *st, *a, (cudaStream_t)stream);
}
