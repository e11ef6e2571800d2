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

constexpr int kTokens = 8, kThreads = 256;

struct Token {
  int pos, local, slot;
  int64_t page_row;    // row of the layer's pages for KV head 0, -1: none
};

// A block takes `per` tokens of the heads of one round: LH lanes per head row, ITEMS vectors of V elements per lane.  NT: taps
// where known at compile time (ITEMS is then 1, and the usual tokens - one sequence, all inputs among the step's rows - keep their
// window of rows in registers), else 0.
template <typename T, int V, int LH, int ITEMS, int NT>
__global__ void __launch_bounds__(kThreads, ITEMS == 1 ? 2 : 1) append_conv_kernel(pace_step_t st, PageRows pg, pace_append_conv_args_t a, int row, int per) {
  __shared__ Token info[kTokens];
  extern __shared__ float turn_by[];       // [per][cosines, sines][rot_pairs] of the block's tokens
  const int lane = threadIdx.x % LH, groups = blockDim.x / LH, t0 = blockIdx.x * per, n_tok = min(per, st.n_tokens - t0);
  const int H = a.n_q_heads, G = pg.n_kv_heads, d = a.dim, vd = a.vdim, channels = (H + G) * d + G * vd;
  const int taps = NT ? NT : a.n_taps;
  const T* in = static_cast<const T*>(a.qkv);
  const int hh = blockIdx.y * groups + threadIdx.x / LH;
  const bool exists = hh < H + 2 * G, is_q = hh < H, is_v = hh >= H + G;
  const int g = is_v ? hh - H - G : hh - H, n = exists ? (is_v ? vd : d) : 0;
  const int ch0 = is_q ? hh * d : is_v ? (H + G) * d + g * vd : H * d + g * d;   // first channel of the head
  if (threadIdx.x < n_tok) {
    const int t = t0 + threadIdx.x, e = st.tok_entry[t], pos = st.tok_pos[t], slot = st.slot[e], lp = pos / pg.page_tokens;
    Token k;
    k.pos = pos;
    k.local = t - st.cu[e];
    k.slot = slot;
    int page = -1;
    if (slot >= 0 && slot < pg.max_seqs && lp < pg.max_pages_per_seq) page = pg.block_table[(size_t)slot * pg.max_pages_per_seq + lp];
    if (page < 0 || page >= pg.n_pages || (a.rot_pairs > 0 && pos >= a.table_rows)) raise_status(pg.status, PACE_DEV_BAD_INDEX);
    k.page_row = page >= 0 && page < pg.n_pages ? (int64_t)page * G * pg.page_tokens + (pos - lp * pg.page_tokens) : -1;
    info[threadIdx.x] = k;
  }
  for (int i = threadIdx.x; i < n_tok * 2 * a.rot_pairs; i += blockDim.x) {
    const int r = i / (2 * a.rot_pairs), c = i - r * 2 * a.rot_pairs, pos = min(st.tok_pos[t0 + r], a.table_rows - 1);
    turn_by[i] = c < a.rot_pairs ? a.cos_table[(size_t)pos * a.rot_pairs + c] : a.sin_table[(size_t)pos * a.rot_pairs + c - a.rot_pairs];
  }
  float nw[ITEMS][V];      // norm weights
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * LH + lane) * V;
    if (!is_v && c < n) Vec<float, V>::load((is_q ? a.q_norm : a.k_norm) + c, nw[i]);
    else
#pragma unroll
      for (int v = 0; v < V; ++v) nw[i][v] = 1.f;
  }

  // norm, rotation and store of a token's convolved head row
  auto finish = [&](int r, float (*y)[V]) {
    const Token& k = info[r];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) ss = fmaf(y[i][v], y[i][v], ss);
#pragma unroll
    for (int o = LH / 2; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float f = is_v ? a.v_mul : 1.0f / sqrtf(ss / (float)n + a.eps);
    T* dst = nullptr;
    if (is_q) dst = static_cast<T*>(a.q_out) + ((size_t)(t0 + r) * H + hh) * row;
    else if (exists && k.page_row >= 0) dst = reinterpret_cast<T*>(is_v ? pg.v : pg.k) + (k.page_row + (int64_t)g * pg.page_tokens) * row;
    const bool turns = !is_v;
    const float *cs = turn_by + r * 2 * a.rot_pairs, *sn = cs + a.rot_pairs;
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * LH + lane) * V;
#pragma unroll
      for (int v = 0; v < V; ++v) y[i][v] *= f * nw[i][v];
      // the partner of an element lies in the same vector, or (V = 1) in the neighbouring lane
      if constexpr (V == 1) {
        const float other = __shfl_xor_sync(0xffffffffu, y[i][0], 1);
        if (turns && (c >> 1) < a.rot_pairs)
          y[i][0] = (c & 1) ? y[i][0] * cs[c >> 1] + other * sn[c >> 1] : y[i][0] * cs[c >> 1] - other * sn[c >> 1];
      } else if (turns && c < 2 * a.rot_pairs) {
#pragma unroll
        for (int v = 0; v < V; v += 2) {
          const int pr = (c + v) >> 1;
          if (pr < a.rot_pairs) {
            const float u = y[i][v] * cs[pr] - y[i][v + 1] * sn[pr];
            y[i][v + 1] = y[i][v + 1] * cs[pr] + y[i][v] * sn[pr];
            y[i][v] = u;
          }
        }
      }
      if (dst && c < n) Vec<T, V>::store(dst + c, y[i]);
    }
    if (dst) {                                             // what a row has beyond its head size
      float zero[V];
#pragma unroll
      for (int v = 0; v < V; ++v) zero[v] = 0.f;
      for (int c = n + lane * V; c < row; c += LH * V) Vec<T, V>::store(dst + c, zero);
    }
  };

  float w[NT ? NT : 1][V];
  if constexpr (NT > 0) {
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (lane * V < n) Vec<float, V>::load(a.taps + (size_t)j * channels + ch0 + lane * V, w[j]);
      else
#pragma unroll
        for (int v = 0; v < V; ++v) w[j][v] = 0.f;
    }
  }
  if constexpr (NT > 0 && V * sizeof(T) == 16) {
    // (a first look without the barrier: the rows may be on their way while the tokens' places are looked up)
    const int e0 = st.tok_entry[t0];
    if (per > 1 && t0 - (NT - 1) >= st.cu[e0] && t0 + n_tok <= st.cu[e0 + 1]) {
      uint4 raw[kTokens + NT - 1];
      const T* src = in + (int64_t)(t0 - (NT - 1)) * a.qkv_stride + ch0 + (lane * V < n ? lane * V : 0);
#pragma unroll
      for (int r = 0; r < kTokens + NT - 1; ++r)
        raw[r] = lane * V < n && r < n_tok + NT - 1 ? *reinterpret_cast<const uint4*>(src + r * a.qkv_stride) : make_uint4(0, 0, 0, 0);
      __syncthreads();
#pragma unroll
      for (int r = 0; r < kTokens; ++r) {
        if (r >= n_tok) break;
        float y[1][V];
#pragma unroll
        for (int v = 0; v < V; ++v) y[0][v] = 0.f;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          float x[V];
          Vec<T, V>::load(reinterpret_cast<const T*>(&raw[r + j]), x);
#pragma unroll
          for (int v = 0; v < V; ++v) y[0][v] = fmaf(w[j][v], x[v], y[0][v]);
        }
        finish(r, y);
      }
      return;
    }
  }
  __syncthreads();
  for (int r = 0; r < n_tok; ++r) {
    const Token& k = info[r];
    float* ring = a.ring + (size_t)k.slot * a.ring_rows * a.ring_stride + ch0;
    const T* now = in + (size_t)(t0 + r) * a.qkv_stride + ch0;
    float y[ITEMS][V];
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * LH + lane) * V;
#pragma unroll
      for (int v = 0; v < V; ++v) y[i][v] = 0.f;
      if (c >= n) continue;
      auto tap = [&](int j, const float* wj) {
        const int back = taps - 1 - j;
        float x[V];
        if (back <= k.local) Vec<T, V>::load(now - (int64_t)back * a.qkv_stride + c, x);
        else if (back <= k.pos) Vec<float, V>::load(ring + (size_t)((k.pos - back) % a.ring_rows) * a.ring_stride + c, x);
        else return;                                       // in front of the sequence
#pragma unroll
        for (int v = 0; v < V; ++v) y[i][v] = fmaf(wj[v], x[v], y[i][v]);
        if (a.store_ring && back == 0) Vec<float, V>::store(ring + (size_t)(k.pos % a.ring_rows) * a.ring_stride + c, x);
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
    }
    finish(r, y);
  }
}

template <typename T, int V, int LH, int ITEMS, int NT>
int launch(const pace_step_t& st, const PageRows& pg, const pace_append_conv_args_t& a, int row, cudaStream_t s) {
  const int heads = a.n_q_heads + 2 * pg.n_kv_heads, per = st.n_tokens >= 148 * kTokens ? kTokens : st.n_tokens >= 148 ? 2 : 1;
  int threads = (heads * LH + 31) / 32 * 32;
  if (threads > kThreads) threads = kThreads;
  const int groups = threads / LH, rounds = (heads + groups - 1) / groups;
  if (rounds > 65535) return PACE_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * per * 2 * a.rot_pairs;
  append_conv_kernel<T, V, LH, ITEMS, NT><<<dim3((unsigned)((st.n_tokens + per - 1) / per), (unsigned)rounds), threads, smem, s>>>(st, pg, a, row, per);
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
