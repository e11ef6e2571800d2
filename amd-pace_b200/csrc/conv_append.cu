// Short causal convolutions of the query, key and value projections on their way to attention: per token and head the
// convolution over the last tokens, the norm over the head, the rotation, then the staging row (queries) or the page (keys,
// values).  Inputs in front of the step come from the sequence's ring of newest projections.  fp32 arithmetic.
#include "hybrid.cuh"

namespace pace {
namespace {

struct PageRows {
  const int32_t* block_table;
  int32_t* status;
  char *k, *v;       // this layer's K and V regions
  int page_tokens, n_kv_heads, max_pages_per_seq, max_seqs, n_pages;
};

constexpr int kTokens = 4, kThreads = 256;

// LH lanes per head row, ITEMS vectors of V elements per lane; a block takes `per` tokens, whose rows the convolution
// reads again out of the cache.  NT: taps where known at compile time (and held in registers), else 0.
template <typename T, int V, int LH, int ITEMS, int NT>
__global__ void __launch_bounds__(kThreads) append_conv_kernel(pace_step_t st, PageRows pg, pace_append_conv_args_t a, int row, int per) {
  const int lane = threadIdx.x % LH, groups = blockDim.x / LH, t0 = blockIdx.x * per;
  const int n_tok = min(per, st.n_tokens - t0);
  const int H = a.n_q_heads, G = pg.n_kv_heads, d = a.dim, vd = a.vdim, channels = (H + G) * d + G * vd;
  const int taps = NT ? NT : a.n_taps;
  const T* in = static_cast<const T*>(a.qkv);
  // blocks of one token spread the heads over the grid's y extent, so that a decode step fills the GPU
  const int rounds = (H + 2 * G + groups * gridDim.y - 1) / (groups * gridDim.y);   // (the same for every thread)
  for (int it = 0; it < rounds; ++it) {
    const int hh = (it * gridDim.y + blockIdx.y) * groups + threadIdx.x / LH;
    const bool exists = hh < H + 2 * G, is_q = hh < H, is_v = hh >= H + G;
    const int g = is_v ? hh - H - G : hh - H, n = exists ? (is_v ? vd : d) : 0;
    const int ch0 = is_q ? hh * d : is_v ? (H + G) * d + g * vd : H * d + g * d;   // first channel of the head
    float w[NT ? NT : 1][V];   // (ITEMS is 1 where NT is not 0)
    if constexpr (NT > 0) {
      if (lane * V < n) {
#pragma unroll
        for (int j = 0; j < NT; ++j) Vec<float, V>::load(a.taps + (size_t)j * channels + ch0 + lane * V, w[j]);
      }
    }
    for (int r = 0; r < n_tok; ++r) {
      const int t = t0 + r, e = st.tok_entry[t], local = t - st.cu[e], pos = st.tok_pos[t], slot = st.slot[e];
      float* ring = a.ring + (size_t)slot * a.ring_rows * a.ring_stride + ch0;
      const T* now = in + (size_t)t * a.qkv_stride + ch0;
      float y[ITEMS][V], ss = 0.f;
#pragma unroll
      for (int i = 0; i < ITEMS; ++i) {
        const int c = (i * LH + lane) * V;
#pragma unroll
        for (int v = 0; v < V; ++v) y[i][v] = 0.f;
        if (c >= n) continue;
        auto tap = [&](int j, const float* wj) {
          const int back = taps - 1 - j;
          float x[V];
          if (back <= local) Vec<T, V>::load(now - (int64_t)back * a.qkv_stride + c, x);
          else if (back <= pos) Vec<float, V>::load(ring + (size_t)((pos - back) % a.ring_rows) * a.ring_stride + c, x);
          else return;                                     // in front of the sequence
#pragma unroll
          for (int v = 0; v < V; ++v) y[i][v] = fmaf(wj[v], x[v], y[i][v]);
          if (a.store_ring && back == 0) Vec<float, V>::store(ring + (size_t)(pos % a.ring_rows) * a.ring_stride + c, x);
        };
        if constexpr (NT > 0) {
#pragma unroll
          for (int j = 0; j < NT; ++j) tap(j, w[j]);
        } else {
          for (int j = 0; j < taps; ++j) {
            float wj[V];
            Vec<float, V>::load(a.taps + (size_t)j * channels + ch0 + c, wj);
            tap(j, wj);
          }
        }
#pragma unroll
        for (int v = 0; v < V; ++v) ss = fmaf(y[i][v], y[i][v], ss);
      }
#pragma unroll
      for (int o = LH / 2; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float f = is_v ? a.v_mul : 1.0f / sqrtf(ss / (float)n + a.eps);
      const float* nw = is_q ? a.q_norm : a.k_norm;
      T* dst = nullptr;
      if (exists && is_q) {
        dst = static_cast<T*>(a.q_out) + ((size_t)t * H + hh) * row;
      } else if (exists) {
        const int lp = pos / pg.page_tokens;
        int page = -1;
        if (slot >= 0 && slot < pg.max_seqs && lp < pg.max_pages_per_seq)
          page = pg.block_table[(size_t)slot * pg.max_pages_per_seq + lp];
        if (page >= 0 && page < pg.n_pages)
          dst = reinterpret_cast<T*>(is_v ? pg.v : pg.k) + (((size_t)page * G + g) * pg.page_tokens + (pos - lp * pg.page_tokens)) * row;
        else if (lane == 0)
          raise_status(pg.status, PACE_DEV_BAD_INDEX);
      }
      const bool turns = !is_v && a.rot_pairs > 0;
      if (turns && pos >= a.table_rows && lane == 0) raise_status(pg.status, PACE_DEV_BAD_INDEX);
#pragma unroll
      for (int i = 0; i < ITEMS; ++i) {
        const int c = (i * LH + lane) * V;
        if (!is_v && c < n) {
          float wv[V];
          Vec<float, V>::load(nw + c, wv);
#pragma unroll
          for (int v = 0; v < V; ++v) y[i][v] *= f * wv[v];
        } else {
#pragma unroll
          for (int v = 0; v < V; ++v) y[i][v] *= f;
        }
        // the partner of an element lies in the same vector, or (V = 1) in the neighbouring lane
        if constexpr (V == 1) {
          const float other = __shfl_xor_sync(0xffffffffu, y[i][0], 1);
          if (turns && (c >> 1) < a.rot_pairs && pos < a.table_rows) {
            const float cs = a.cos_table[(size_t)pos * a.rot_pairs + (c >> 1)], sn = a.sin_table[(size_t)pos * a.rot_pairs + (c >> 1)];
            y[i][0] = (c & 1) ? y[i][0] * cs + other * sn : y[i][0] * cs - other * sn;
          }
        } else if (turns && pos < a.table_rows) {
#pragma unroll
          for (int v = 0; v < V; v += 2) {
            const int pr = (c + v) >> 1;
            if (pr < a.rot_pairs) {
              const float cs = a.cos_table[(size_t)pos * a.rot_pairs + pr], sn = a.sin_table[(size_t)pos * a.rot_pairs + pr];
              const float u = y[i][v] * cs - y[i][v + 1] * sn;
              y[i][v + 1] = y[i][v + 1] * cs + y[i][v] * sn;
              y[i][v] = u;
            }
          }
        }
        if (dst && c < n) Vec<T, V>::store(dst + c, y[i]);
      }
      if (dst) {                                           // what a row has beyond its head size
        float zero[V];
#pragma unroll
        for (int v = 0; v < V; ++v) zero[v] = 0.f;
        for (int c = n + lane * V; c < row; c += LH * V) Vec<T, V>::store(dst + c, zero);
      }
    }
  }
}

template <typename T, int V, int LH, int ITEMS, int NT>
int launch(const pace_step_t& st, const PageRows& pg, const pace_append_conv_args_t& a, int row, cudaStream_t s) {
  const int heads = a.n_q_heads + 2 * pg.n_kv_heads, per = st.n_tokens >= 148 * kTokens ? kTokens : 1,
            blocks = (st.n_tokens + per - 1) / per;
  int threads = (heads * LH + 31) / 32 * 32;
  if (threads > kThreads) threads = kThreads;
  int split = 1;                                            // few tokens: several blocks share their heads
  while (blocks * split < 296 && split * threads < heads * LH && split < 64) split *= 2;
  append_conv_kernel<T, V, LH, ITEMS, NT><<<dim3((unsigned)blocks, (unsigned)split), threads, 0, s>>>(st, pg, a, row, per);
  PACE_LAUNCH_CHECK("append_conv_kernel");
  return PACE_OK;
}

template <typename T, int V, int LH>
int launch_taps(const pace_step_t& st, const PageRows& pg, const pace_append_conv_args_t& a, int row, cudaStream_t s) {
  if (a.n_taps == 4) return launch<T, V, LH, 1, 4>(st, pg, a, row, s);
  if (a.n_taps == 3) return launch<T, V, LH, 1, 3>(st, pg, a, row, s);
  if (a.n_taps == 2) return launch<T, V, LH, 1, 2>(st, pg, a, row, s);
  return launch<T, V, LH, 1, 0>(st, pg, a, row, s);
}

template <typename T>
int append_conv_t(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_append_conv_args_t& a, cudaStream_t s) {
  const int row = p->head_dim * 2 / (int)sizeof(T), widest = a.dim > a.vdim ? a.dim : a.vdim;
  if (widest > row) return PACE_ERR_INVALID;
  const size_t region = (size_t)p->n_pages * p->n_kv_heads * p->page_tokens * p->head_dim * 2;  // bytes
  PageRows pg;
  pg.block_table = p->block_table;
  pg.status = p->status;
  pg.k = static_cast<char*>(p->pages) + (size_t)layer * 2 * region;
  pg.v = pg.k + region;
  pg.page_tokens = p->page_tokens;
  pg.n_kv_heads = p->n_kv_heads;
  pg.max_pages_per_seq = p->max_pages_per_seq;
  pg.max_seqs = p->max_seqs;
  pg.n_pages = p->n_pages;
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.dim % V == 0 && a.vdim % V == 0 && row % V == 0 && a.qkv_stride % V == 0 && a.ring_stride % V == 0 &&
                   aligned16(a.qkv) && aligned16(a.q_out) && aligned16(a.q_norm) && aligned16(a.k_norm) && aligned16(a.taps) &&
                   aligned16(a.ring);
  int rc;
  if (vec && widest <= 8 * V) rc = launch_taps<T, V, 8>(st, pg, a, row, s);
  else if (vec && widest <= 16 * V) rc = launch_taps<T, V, 16>(st, pg, a, row, s);
  else if (vec && widest <= 32 * V) rc = launch_taps<T, V, 32>(st, pg, a, row, s);
  else if (widest <= 128) rc = launch<T, 1, 32, 4, 0>(st, pg, a, row, s);
  else if (widest <= 640) rc = launch<T, 1, 32, 20, 0>(st, pg, a, row, s);
  else return PACE_ERR_UNSUPPORTED;
  if (rc == PACE_OK) note_pool_write(s);
  return rc;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" int pace_kv_append_conv(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const pace_append_conv_args_t* a,
                                   void* stream) {
  if (!p || !p->pages || !p->block_table || !step_ok(st) || !a || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (!a->qkv || !a->taps || !a->ring || !a->q_norm || !a->k_norm || !a->q_out || a->n_q_heads < 1 || a->n_q_heads % p->n_kv_heads ||
      a->dim < 1 || a->vdim < 1 || a->n_taps < 1 || a->ring_rows < 1 || a->ring_rows < a->n_taps - 1 || a->rot_pairs < 0 ||
      2 * a->rot_pairs > a->dim || (a->rot_pairs > 0 && (!a->cos_table || !a->sin_table || a->table_rows < 1)))
    return PACE_ERR_INVALID;
  const int64_t channels = (int64_t)(a->n_q_heads + p->n_kv_heads) * a->dim + (int64_t)p->n_kv_heads * a->vdim;
  if (a->qkv_stride < channels || a->ring_stride < channels) return PACE_ERR_INVALID;
  if (a->store_ring && (st->n_tokens != st->n_entries || a->ring_rows < a->n_taps)) return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_SHARED) return PACE_ERR_UNSUPPORTED;
  if (p->row_format == PACE_ROWS_BF16 && a->dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("kv_append_conv", stream, "layer=%d tokens=%d", layer, st->n_tokens);
  if (a->dtype == PACE_DTYPE_BF16) return append_conv_t<__nv_bfloat16>(p, layer, *st, *a, (cudaStream_t)stream);
  if (a->dtype == PACE_DTYPE_FP32) return append_conv_t<float>(p, layer, *st, *a, (cudaStream_t)stream);
  return PACE_ERR_INVALID;
}
