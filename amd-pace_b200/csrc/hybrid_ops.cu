// Token-wise kernels of hybrid decoders: residual + norms, the append of normalised keys, output gates,
// squared ReLU.  One thread block per token row where a row has to be summed over; fp32 arithmetic.
#include "hybrid.cuh"

namespace pace {
namespace {

// ---------------------------------------------------------------------------
// x' = x + rms(y) w_post (+ embedding row);  h = rms(x') w_next, or x' itself
// MOE: y is the weighted sum of the rows of the token's experts
// ---------------------------------------------------------------------------
constexpr int kMaxTop = 64;

template <typename T, int V, int ITEMS, bool MOE>
__global__ void __launch_bounds__(512) residual_norm_kernel(pace_step_t st, pace_residual_norm_args_t a) {
  __shared__ float red[32];
  __shared__ int e_row[MOE ? kMaxTop : 1];
  __shared__ float e_w[MOE ? kMaxTop : 1];
  const int t = blockIdx.x, W = a.width;
  if constexpr (MOE) {
    // one warp per chosen expert: the expert's first row is the number of tokens of all experts in front of it
    for (int k = threadIdx.x >> 5; k < a.top; k += blockDim.x >> 5) {
      const int e = a.slot_expert[(size_t)t * a.top + k];
      int n = 0;
      for (int i = threadIdx.x & 31; i < e && e < a.n_experts; i += 32) n += a.expert_count[i];
#pragma unroll
      for (int o = 16; o; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
      if ((threadIdx.x & 31) == 0) {
        e_row[k] = e < a.n_experts ? n + a.slot_rank[(size_t)t * a.top + k] : -1;   // -1: an identity expert
        e_w[k] = a.slot_weight[(size_t)t * a.top + k];
      }
    }
    __syncthreads();
  }
  float xv[ITEMS][V], yv[ITEMS][V];
  float* x = a.x + (size_t)t * W;
  const T* y = a.y ? static_cast<const T*>(a.y) + (size_t)t * a.y_stride : nullptr;
  const T* em = nullptr;
  if (a.embed) {
    const int tok = st.token[t];
    if (tok >= 0 && tok < a.vocab) em = static_cast<const T*>(a.embed) + (size_t)tok * W;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
    if (c < W) {
      if (!a.restart) Vec<float, V>::load(x + c, xv[i]);
      else
#pragma unroll
        for (int j = 0; j < V; ++j) xv[i][j] = 0.f;
      if (MOE) {
#pragma unroll
        for (int j = 0; j < V; ++j) yv[i][j] = 0.f;
        for (int k = 0; k < a.top; ++k) {
          float r[V];
          Vec<T, V>::load(e_row[k] >= 0 ? static_cast<const T*>(a.y) + (size_t)e_row[k] * a.y_stride + c
                                        : static_cast<const T*>(a.identity) + (size_t)t * W + c, r);
#pragma unroll
          for (int j = 0; j < V; ++j) yv[i][j] = fmaf(e_w[k], r[j], yv[i][j]);
        }
      } else if (y) {
        Vec<T, V>::load(y + c, yv[i]);
      }
      if (a.add) {
        float r[V];
        Vec<T, V>::load(static_cast<const T*>(a.add) + (size_t)t * a.add_stride + c, r);
#pragma unroll
        for (int j = 0; j < V; ++j) yv[i][j] += r[j];
      }
      if (a.y_bias) {
        float r[V];
        Vec<float, V>::load(a.y_bias + c, r);
#pragma unroll
        for (int j = 0; j < V; ++j) yv[i][j] += r[j];
      }
      if (y) {
#pragma unroll
        for (int j = 0; j < V; ++j) ss += yv[i][j] * yv[i][j];
      }
    }
  }
  if (y) {
    float r = 1.f;
    if (a.w_post) r = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) {
        float w[V];
        if (a.w_post) Vec<float, V>::load(a.w_post + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j) xv[i][j] += a.w_post ? yv[i][j] * r * (a.weight_offset + w[j]) : yv[i][j] * a.y_mul;
      }
    }
  }
  float em_r = 1.f;
  if (a.embed_norm) {
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W && em) {
        float e[V];
        Vec<T, V>::load(em + c, e);
#pragma unroll
        for (int j = 0; j < V; ++j) ss += e[j] * e[j];
      }
    }
    em_r = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
  }
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
    if (c < W) {
      if (em) {
        float e[V], w[V];
        Vec<T, V>::load(em + c, e);
        if (a.embed_norm) Vec<float, V>::load(a.embed_norm + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j)
          xv[i][j] = fmaf(e[j], a.embed_norm ? em_r * (a.weight_offset + w[j]) : a.embed_scale, xv[i][j]);
      }
      Vec<float, V>::store(x + c, xv[i]);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += xv[i][j] * xv[i][j];
    }
  }
  if (!a.h) return;
  T* h = static_cast<T*>(a.h) + (size_t)t * W;
  if (!a.w_next) {
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) Vec<T, V>::store(h + c, xv[i]);
    }
    return;
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
    if (c < W) {
      float w[V];
      Vec<float, V>::load(a.w_next + c, w);
#pragma unroll
      for (int j = 0; j < V; ++j) w[j] = xv[i][j] * r * (a.weight_offset + w[j]);
      Vec<T, V>::store(h + c, w);
      if (a.h2) {
        Vec<float, V>::load(a.w_next2 + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j) w[j] = xv[i][j] * r * (a.weight_offset + w[j]);
        Vec<T, V>::store(static_cast<T*>(a.h2) + (size_t)t * W + c, w);
      }
    }
  }
}

// Threads for a row of `groups` vectors and how many vectors each of them takes (1, 2, 4, 8 or 16), 0 = too wide.
int row_items(int groups, int* threads) {
  int th = (groups + 31) / 32 * 32;
  if (th > 512) th = 512;
  *threads = th;
  const int need = (groups + th - 1) / th;
  for (int i = 1; i <= 16; i *= 2)
    if (need <= i) return i;
  return 0;
}

template <typename T, int V>
int launch_residual_norm(const pace_step_t& st, const pace_residual_norm_args_t& a, cudaStream_t s) {
  int threads = 0;
  const int items = row_items((a.width + V - 1) / V, &threads);
#define PACE_NORM_CASE(n)                                                                          \
  case n:                                                                                          \
    if (a.top > 0) residual_norm_kernel<T, V, n, true><<<st.n_tokens, threads, 0, s>>>(st, a);     \
    else residual_norm_kernel<T, V, n, false><<<st.n_tokens, threads, 0, s>>>(st, a);              \
    break;
  switch (items) {
    PACE_NORM_CASE(1)
    PACE_NORM_CASE(2)
    PACE_NORM_CASE(4)
    PACE_NORM_CASE(8)
    PACE_NORM_CASE(16)
    default: return PACE_ERR_UNSUPPORTED;
  }
#undef PACE_NORM_CASE
  PACE_LAUNCH_CHECK("residual_norm_kernel");
  return PACE_OK;
}

// ---------------------------------------------------------------------------
// q / k norms over the whole projections, query temperature, rows to the staging buffer and to the pages
// ---------------------------------------------------------------------------
struct PageRows {
  const int32_t* block_table;
  int32_t* status;
  char *k, *v;       // this layer's K and V regions
  int page_tokens, n_kv_heads, max_pages_per_seq, max_seqs, n_pages;
};

template <typename T, int V>
__global__ void append_norm_kernel(pace_step_t st, PageRows pg, pace_append_norm_args_t a, int row) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const int H = a.n_q_heads, G = pg.n_kv_heads, d = a.dim, vd = a.vdim;
  const int nq = H * d, nk = G * d;
  const T* src = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride;
  const T *qs = src, *ks = src + nq, *vs = ks + nk;
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * V; c < nq + nk; c += blockDim.x * V) {  // (V divides dim: a vector never straddles)
    float x[V];
    Vec<T, V>::load(src + c, x);
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) s += x[j] * x[j];
    if (c < nq) sq += s; else sk += s;
  }
  const float rq0 = a.q_norm ? 1.0f / sqrtf(block_sum(sq, red) / (float)nq + a.eps) : 1.f;
  const float rk = a.k_norm ? 1.0f / sqrtf(block_sum(sk, red) / (float)nk + a.eps) : 1.f;
  const int pos = st.tok_pos[t];
  float temp = a.q_mul;
  if (a.temp_coef != 0.f) temp *= 1.0f + a.temp_coef * logf((float)(floor((double)(pos + 1) / a.temp_every) + 1.0));
  const int slot = st.slot[st.tok_entry[t]];
  const int lp = pos / pg.page_tokens;
  int page = -1;
  if (slot >= 0 && slot < pg.max_seqs && lp < pg.max_pages_per_seq)
    page = pg.block_table[(size_t)slot * pg.max_pages_per_seq + lp];
  if (page < 0 || page >= pg.n_pages) {
    if (threadIdx.x == 0) raise_status(pg.status, PACE_DEV_BAD_INDEX);
    page = -1;
  }
  const int per_row = row / V;  // vectors of one padded row
  T* qo = static_cast<T*>(a.q_out) + (size_t)st.q_row[t] * H * row;
  for (int i = threadIdx.x; i < (H + 2 * G) * per_row; i += blockDim.x) {
    const int hh = i / per_row, c = (i - hh * per_row) * V;
    float x[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = 0.f;
    if (hh < H) {
      if (c < d) {
        Vec<T, V>::load(qs + hh * d + c, x);
        if (a.q_norm) {
          float w[V];
          Vec<float, V>::load(a.q_norm + hh * d + c, w);
#pragma unroll
          for (int j = 0; j < V; ++j) x[j] *= rq0 * w[j];
        }
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] *= temp;
      }
      Vec<T, V>::store(qo + (size_t)hh * row + c, x);
      continue;
    }
    const int g = hh < H + G ? hh - H : hh - H - G;
    const bool is_v = hh >= H + G;
    if (is_v) {
      if (c < vd) Vec<T, V>::load(vs + g * vd + c, x);
    } else if (c < d) {
      Vec<T, V>::load(ks + g * d + c, x);
      if (a.k_norm) {
        float w[V];
        Vec<float, V>::load(a.k_norm + g * d + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] *= rk * w[j];
      }
    }
    if (page >= 0) {
      const size_t off = (((size_t)page * G + g) * pg.page_tokens + (pos - lp * pg.page_tokens)) * row + c;
      Vec<T, V>::store(reinterpret_cast<T*>(is_v ? pg.v : pg.k) + off, x);
    }
  }
}

// The same for rows that fit in registers (ITEMS vectors of V elements per thread): one pass over the projection row,
// one reduction for both sums.
template <typename T, int V, int ITEMS>
__global__ void __launch_bounds__(512) append_norm_regs_kernel(pace_step_t st, PageRows pg, pace_append_norm_args_t a, int row) {
  __shared__ float2 red[16];
  const int t = blockIdx.x, tid = threadIdx.x;
  const int H = a.n_q_heads, G = pg.n_kv_heads, d = a.dim, vd = a.vdim;
  const int nq = H * d, nk = G * d, n = nq + nk + G * vd;
  const T* src = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride;
  uint4 raw[ITEMS];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + tid) * V;
    if (c < n) raw[i] = *reinterpret_cast<const uint4*>(src + c);
  }
  const int pos = st.tok_pos[t], slot = st.slot[st.tok_entry[t]];
  const size_t q_row = (size_t)st.q_row[t];
  const int lp = pos / pg.page_tokens;
  int page = -1;
  if (slot >= 0 && slot < pg.max_seqs && lp < pg.max_pages_per_seq)
    page = pg.block_table[(size_t)slot * pg.max_pages_per_seq + lp];
  float2 ss = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + tid) * V;
    if (c < nq + nk) {
      float x[V], s = 0.f;
      Vec<T, V>::load(reinterpret_cast<const T*>(&raw[i]), x);
#pragma unroll
      for (int j = 0; j < V; ++j) s = fmaf(x[j], x[j], s);
      if (c < nq) ss.x += s; else ss.y += s;
    }
  }
#pragma unroll
  for (int o = 16; o; o >>= 1) {
    ss.x += __shfl_xor_sync(0xffffffffu, ss.x, o);
    ss.y += __shfl_xor_sync(0xffffffffu, ss.y, o);
  }
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = make_float2(0.f, 0.f);
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
    ss.x += red[w].x;
    ss.y += red[w].y;
  }
  float temp = a.q_mul;
  if (a.temp_coef != 0.f) temp *= 1.0f + a.temp_coef * logf((float)(floor((double)(pos + 1) / a.temp_every) + 1.0));
  const float fq = (a.q_norm ? 1.0f / sqrtf(ss.x / (float)nq + a.eps) : 1.f) * temp;
  const float fk = a.k_norm ? 1.0f / sqrtf(ss.y / (float)nk + a.eps) : 1.f;
  if (page < 0 || page >= pg.n_pages) {
    if (tid == 0) raise_status(pg.status, PACE_DEV_BAD_INDEX);
    page = -1;
  }
  T* qo = static_cast<T*>(a.q_out) + q_row * H * row;
  const size_t in_page = (size_t)pos - (size_t)lp * pg.page_tokens;
  auto page_row = [&](bool is_v, int g) {
    return reinterpret_cast<T*>(is_v ? pg.v : pg.k) + (((size_t)page * G + g) * pg.page_tokens + in_page) * row;
  };
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + tid) * V;
    if (c >= n) continue;
    if (c >= nq + nk) {                                    // values go as they are
      const int o = c - nq - nk, g = o / vd;
      if (page >= 0) *reinterpret_cast<uint4*>(page_row(true, g) + (o - g * vd)) = raw[i];
      continue;
    }
    const bool is_q = c < nq;
    const float* w = is_q ? (a.q_norm ? a.q_norm + c : nullptr) : (a.k_norm ? a.k_norm + c - nq : nullptr);
    const float f = is_q ? fq : fk;
    float x[V];
    Vec<T, V>::load(reinterpret_cast<const T*>(&raw[i]), x);
    if (w) {
      float wv[V];
      Vec<float, V>::load(w, wv);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= f * wv[j];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= f;
    }
    const int o = is_q ? c : c - nq, h = o / d;
    if (is_q) Vec<T, V>::store(qo + (size_t)h * row + (o - h * d), x);
    else if (page >= 0) Vec<T, V>::store(page_row(false, h) + (o - h * d), x);
  }
  // what a row has beyond its head size
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const int pd = (row - d) / V, pv = (row - vd) / V, heads_d = H + (page >= 0 ? G : 0);
  for (int i = tid; i < heads_d * pd; i += blockDim.x) {
    const int h = i / pd, c = d + (i - h * pd) * V;
    *reinterpret_cast<uint4*>((h < H ? qo + (size_t)h * row : page_row(false, h - H)) + c) = zero;
  }
  if (page >= 0)
    for (int i = tid; i < G * pv; i += blockDim.x) {
      const int g = i / pv;
      *reinterpret_cast<uint4*>(page_row(true, g) + vd + (i - g * pv) * V) = zero;
    }
}

// Per-head norms without weights: LH lanes per head row of (queries, keys, values), V elements an access.
template <typename T, int V, int LH>
__global__ void append_heads_kernel(pace_step_t st, PageRows pg, pace_append_norm_args_t a, int row) {
  const int t = blockIdx.x, lane = threadIdx.x % LH, groups = blockDim.x / LH;
  const int H = a.n_q_heads, G = pg.n_kv_heads, d = a.dim, vd = a.vdim;
  const T* src = static_cast<const T*>(a.qkv) + (size_t)t * a.qkv_stride;
  const int pos = st.tok_pos[t], slot = st.slot[st.tok_entry[t]], lp = pos / pg.page_tokens;
  int page = -1;
  if (slot >= 0 && slot < pg.max_seqs && lp < pg.max_pages_per_seq)
    page = pg.block_table[(size_t)slot * pg.max_pages_per_seq + lp];
  float temp = a.q_mul;
  if (a.temp_coef != 0.f) temp *= 1.0f + a.temp_coef * logf((float)(floor((double)(pos + 1) / a.temp_every) + 1.0));
  const int rounds = (H + 2 * G + groups - 1) / groups;   // (the same for every thread: shuffles need whole warps)
  for (int it = 0; it < rounds; ++it) {
    const int hh = it * groups + threadIdx.x / LH;
    const bool exists = hh < H + 2 * G, is_q = hh < H, is_v = hh >= H + G;
    const int g = is_v ? hh - H - G : hh - H, n = is_v ? vd : d;
    const T* x = src + (is_q ? hh * d : is_v ? H * d + G * d + g * vd : H * d + g * d);
    float f = 1.f, first[V], ss = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) first[j] = 0.f;
    for (int c = lane * V; c < n && exists; c += LH * V) {
      float v[V];
      Vec<T, V>::load(x + c, v);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        ss = fmaf(v[j], v[j], ss);
        if (c == lane * V) first[j] = v[j];
      }
    }
#pragma unroll
    for (int o = LH / 2; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!is_v) f = 1.0f / sqrtf(ss / (float)n + a.eps) * (is_q ? temp : 1.f);
    if (!exists) continue;
    T* dst;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + ((size_t)t * H + hh) * row;
    } else {
      if (page < 0 || page >= pg.n_pages) {
        if (lane == 0) raise_status(pg.status, PACE_DEV_BAD_INDEX);
        continue;
      }
      dst = reinterpret_cast<T*>(is_v ? pg.v : pg.k) + (((size_t)page * G + g) * pg.page_tokens + (pos - lp * pg.page_tokens)) * row;
    }
    for (int c = lane * V; c < row; c += LH * V) {
      float v[V];
      if (c == lane * V) {
#pragma unroll
        for (int j = 0; j < V; ++j) v[j] = first[j];
      } else if (c < n) {
        Vec<T, V>::load(x + c, v);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] = c < n ? v[j] * f : 0.f;
      Vec<T, V>::store(dst + c, v);
    }
  }
}

template <typename T, int V>
void launch_append_heads(const pace_step_t& st, const PageRows& pg, const pace_append_norm_args_t& a, int row, cudaStream_t s) {
  const int heads = a.n_q_heads + 2 * pg.n_kv_heads, lanes = (row + V - 1) / V;
  auto threads = [&](int lh) {
    const int n = (heads * lh + 31) / 32 * 32;
    return n < 256 ? n : 256;
  };
  if (lanes <= 8) append_heads_kernel<T, V, 8><<<st.n_tokens, threads(8), 0, s>>>(st, pg, a, row);
  else if (lanes <= 16) append_heads_kernel<T, V, 16><<<st.n_tokens, threads(16), 0, s>>>(st, pg, a, row);
  else append_heads_kernel<T, V, 32><<<st.n_tokens, threads(32), 0, s>>>(st, pg, a, row);
}

template <typename T>
int launch_append_norm(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_append_norm_args_t& a,
                       cudaStream_t s) {
  const int row = p->head_dim * 2 / (int)sizeof(T);  // elements of a pool row
  if (a.dim > row || a.vdim > row) return PACE_ERR_INVALID;
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
  const bool vec = a.dim % V == 0 && a.vdim % V == 0 && row % V == 0 && a.qkv_stride % V == 0 && aligned16(a.qkv) &&
                   aligned16(a.q_out) && (!a.q_norm || aligned16(a.q_norm)) && (!a.k_norm || aligned16(a.k_norm));
  if (a.per_head) {
    if (vec) launch_append_heads<T, V>(st, pg, a, row, s);
    else launch_append_heads<T, 1>(st, pg, a, row, s);
    PACE_LAUNCH_CHECK("append_heads_kernel");
    note_pool_write(s);
    return PACE_OK;
  }
  const int groups = (a.n_q_heads + 2 * p->n_kv_heads) * row / (vec ? V : 1);
  const int threads = groups < 512 ? (groups + 31) / 32 * 32 : 512;
  const int n_vec = (a.n_q_heads * a.dim + p->n_kv_heads * (a.dim + a.vdim)) / V;
  int per = n_vec <= 4 * 128 ? 2 : n_vec <= 4 * 512 ? 4 : 8;   // vectors a thread holds
  const int nt = ((n_vec + per - 1) / per + 31) / 32 * 32;
  if (vec && nt <= 512) {
    if (per == 2) append_norm_regs_kernel<T, V, 2><<<st.n_tokens, nt, 0, s>>>(st, pg, a, row);
    else if (per == 4) append_norm_regs_kernel<T, V, 4><<<st.n_tokens, nt, 0, s>>>(st, pg, a, row);
    else append_norm_regs_kernel<T, V, 8><<<st.n_tokens, nt, 0, s>>>(st, pg, a, row);
  } else if (vec) {
    append_norm_kernel<T, V><<<st.n_tokens, threads, 0, s>>>(st, pg, a, row);
  } else {
    append_norm_kernel<T, 1><<<st.n_tokens, threads, 0, s>>>(st, pg, a, row);
  }
  PACE_LAUNCH_CHECK("append_norm_kernel");
  note_pool_write(s);
  return PACE_OK;
}

// ---------------------------------------------------------------------------
// gates and activation
// ---------------------------------------------------------------------------
template <typename T, int V>
__global__ void gate_heads_kernel(pace_step_t st, const T* __restrict__ attn, const T* __restrict__ gate, int64_t gs,
                                  T* __restrict__ out, int H, int vd, int row) {
  const int n = H * vd, per = n / V;
  const size_t total = (size_t)st.n_tokens * per;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i % per) * V;
    const int h = c / vd;
    float o[V], g[V];
    Vec<T, V>::load(attn + ((size_t)st.q_row[t] * H + h) * row + (c - h * vd), o);
    Vec<T, V>::load(gate + (size_t)t * gs + c, g);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] *= sigmoid_t<T>(g[j]);
    Vec<T, V>::store(out + (size_t)t * n + c, o);
  }
}

template <typename T, int V>
__global__ void norm_gate_kernel(const T* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate,
                                 int64_t gs, T* __restrict__ out, int n, float eps) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const T* src = o + (size_t)t * n;
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
    float x[V];
    Vec<T, V>::load(src + c, x);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += x[j] * x[j];
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
  for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
    float x[V], g[V], wv[V];
    Vec<T, V>::load(src + c, x);
    Vec<T, V>::load(gate + (size_t)t * gs + c, g);
    Vec<float, V>::load(w + c, wv);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = x[j] * r * wv[j] * sigmoid_t<T>(g[j]);
    Vec<T, V>::store(out + (size_t)t * n + c, x);
  }
}

template <typename T, int V>
__global__ void relu_squared_kernel(T* __restrict__ x, int64_t n) {
  for (int64_t i = (blockIdx.x * (int64_t)blockDim.x + threadIdx.x) * V; i < n; i += (int64_t)gridDim.x * blockDim.x * V) {
    float v[V];
    Vec<T, V>::load(x + i, v);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float p = fmaxf(v[j], 0.f);
      v[j] = p * p;
    }
    Vec<T, V>::store(x + i, v);
  }
}

template <typename T, int V, int ACT, bool GATED>
__global__ void glu_kernel(const T* __restrict__ x, int64_t xs, T* __restrict__ out, int64_t os, int n_tokens, int n) {
  const int per = n / V;
  const size_t total = (size_t)n_tokens * per;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i % per) * V;
    float g[V], u[V];
    Vec<T, V>::load(x + (size_t)t * xs + c, g);
    if constexpr (GATED) Vec<T, V>::load(x + (size_t)t * xs + n + c, u);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float f = act_t<T>(ACT, g[j]);
      u[j] = GATED ? u[j] * f : f;
    }
    Vec<T, V>::store(out + (size_t)t * os + c, u);
  }
}

template <typename T, int V>
__global__ void gate_per_head_kernel(T* __restrict__ x, const T* __restrict__ gate, int64_t gs, int n_tokens, int heads, int vd) {
  const int per = vd / V;
  const size_t total = (size_t)n_tokens * heads * per;
  for (size_t i = blockIdx.x * (size_t)blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t th = i / per;
    const float f = sigmoid_t<T>(to_f<T>(gate[th / heads * gs + th % heads]));
    float v[V];
    Vec<T, V>::load(x + i * V, v);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] *= f;
    Vec<T, V>::store(x + i * V, v);
  }
}

__global__ void soft_cap_kernel(float* x, int64_t n, float cap) {
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x)
    x[i] = cap * tanhf(x[i] / cap);
}

// Norms over parts of a row: LP lanes (a divisor of 32) per part, or (LP = 0) a block per part.
template <typename T, int V, int LP>
__global__ void part_norm_gate_kernel(pace_part_norm_gate_args_t a) {
  __shared__ float red[32];
  const int parts = a.n / a.part, per_block = LP ? blockDim.x / LP : 1;
  const int64_t total = (int64_t)a.n_tokens * parts;
  const int lane = LP ? threadIdx.x % LP : threadIdx.x, step = (LP ? LP : blockDim.x) * V;
  int64_t i = (int64_t)blockIdx.x * per_block + (LP ? threadIdx.x / LP : 0);
  const bool live = i < total;                 // (shuffles need whole warps)
  if (!live) i = total - 1;
  const int t = (int)(i / parts), c0 = (int)(i % parts) * a.part;
  const T* o = static_cast<const T*>(a.o) + (size_t)t * a.o_stride + c0;
  const T* gate = static_cast<const T*>(a.gate) + (size_t)t * a.gate_stride + c0;
  T* out = static_cast<T*>(a.out) + (size_t)t * a.out_stride + c0;
  auto value = [&](int c, float* x) {
    Vec<T, V>::load(o + c, x);
    if (a.gate_mode == PACE_GATE_SILU_FIRST) {
      float g[V];
      Vec<T, V>::load(gate + c, g);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= silu_t<T>(g[j]);
    }
  };
  float ss = 0.f, first[V];
#pragma unroll
  for (int j = 0; j < V; ++j) first[j] = 0.f;
  for (int c = lane * V; c < a.part; c += step) {
    float x[V];
    value(c, x);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      ss = fmaf(x[j], x[j], ss);
      if (c == lane * V) first[j] = x[j];
    }
  }
  if constexpr (LP > 0) {
#pragma unroll
    for (int w = LP / 2; w; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
  } else {
    ss = block_sum(ss, red);
  }
  if (!live) return;
  const float r = 1.0f / sqrtf(ss / (float)a.part + a.eps);
  for (int c = lane * V; c < a.part; c += step) {
    float x[V], w[V];
    if (c == lane * V) {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] = first[j];
    } else {
      value(c, x);
    }
    Vec<float, V>::load(a.w + (c0 + c) % a.w_period, w);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= r * w[j];
    if (a.gate_mode != PACE_GATE_SILU_FIRST) {
      float g[V];
      Vec<T, V>::load(gate + c, g);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= a.gate_mode == PACE_GATE_SILU ? silu_t<T>(g[j]) : sigmoid_t<T>(g[j]);
    }
    Vec<T, V>::store(out + c, x);
  }
}

template <typename T, int V>
void launch_part_norm_gate(const pace_part_norm_gate_args_t& a, cudaStream_t s) {
  const int vecs = (a.part + V - 1) / V;
  const int64_t total = (int64_t)a.n_tokens * (a.n / a.part);
  auto blocks = [&](int lp) { return (unsigned)((total * lp + 127) / 128); };
  if (vecs <= 8) part_norm_gate_kernel<T, V, 8><<<blocks(8), 128, 0, s>>>(a);
  else if (vecs <= 16) part_norm_gate_kernel<T, V, 16><<<blocks(16), 128, 0, s>>>(a);
  else if (vecs <= 64) part_norm_gate_kernel<T, V, 32><<<blocks(32), 128, 0, s>>>(a);
  else part_norm_gate_kernel<T, V, 0><<<(unsigned)total, vecs < 512 ? (vecs + 31) / 32 * 32 : 512, 0, s>>>(a);
}

template <typename T>
int part_norm_gate_t(const pace_part_norm_gate_args_t& a, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.part % V == 0 && a.w_period % V == 0 && (a.o_stride | a.gate_stride | a.out_stride) % V == 0 && aligned16(a.o) &&
                   aligned16(a.gate) && aligned16(a.out) && aligned16(a.w);
  if (vec) launch_part_norm_gate<T, V>(a, s);
  else launch_part_norm_gate<T, 1>(a, s);
  PACE_LAUNCH_CHECK("part_norm_gate_kernel");
  return PACE_OK;
}

unsigned elementwise_blocks(size_t threads_wanted) {
  size_t b = (threads_wanted + 255) / 256;
  return (unsigned)(b < 1 ? 1 : b > 148 * 16 ? 148 * 16 : b);
}

__global__ void step_decode_kernel(int32_t* token, int32_t* tok_pos, int32_t* start, const int64_t* next, const int64_t* pos,
                                   int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  token[i] = (int32_t)next[i];
  tok_pos[i] = start[i] = (int32_t)pos[i];
}

template <typename T>
int gate_heads_t(const pace_step_t& st, const void* attn, const void* gate, int64_t gs, void* out, int H, int vd, int row,
                 cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = vd % V == 0 && row % V == 0 && gs % V == 0 && aligned16(attn) && aligned16(gate) && aligned16(out);
  const size_t n = (size_t)st.n_tokens * H * vd;
  if (vec)
    gate_heads_kernel<T, V><<<elementwise_blocks(n / V), 256, 0, s>>>(st, (const T*)attn, (const T*)gate, gs, (T*)out, H, vd, row);
  else
    gate_heads_kernel<T, 1><<<elementwise_blocks(n), 256, 0, s>>>(st, (const T*)attn, (const T*)gate, gs, (T*)out, H, vd, row);
  PACE_LAUNCH_CHECK("gate_heads_kernel");
  return PACE_OK;
}

template <typename T>
int norm_gate_t(const void* o, const float* w, const void* gate, int64_t gs, void* out, int n_tokens, int n, float eps,
                cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = n % V == 0 && gs % V == 0 && aligned16(o) && aligned16(gate) && aligned16(out) && aligned16(w);
  const int groups = vec ? n / V : n;
  const int threads = groups < 512 ? (groups + 31) / 32 * 32 : 512;
  if (vec)
    norm_gate_kernel<T, V><<<n_tokens, threads, 0, s>>>((const T*)o, w, (const T*)gate, gs, (T*)out, n, eps);
  else
    norm_gate_kernel<T, 1><<<n_tokens, threads, 0, s>>>((const T*)o, w, (const T*)gate, gs, (T*)out, n, eps);
  PACE_LAUNCH_CHECK("norm_gate_kernel");
  return PACE_OK;
}

template <typename T>
int relu_squared_t(void* x, int64_t n, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  if (n % V == 0 && aligned16(x))
    relu_squared_kernel<T, V><<<elementwise_blocks((size_t)n / V), 256, 0, s>>>((T*)x, n);
  else
    relu_squared_kernel<T, 1><<<elementwise_blocks((size_t)n), 256, 0, s>>>((T*)x, n);
  PACE_LAUNCH_CHECK("relu_squared_kernel");
  return PACE_OK;
}

template <typename T>
int gate_per_head_t(void* x, const void* gate, int64_t gs, int n_tokens, int heads, int vd, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const size_t n = (size_t)n_tokens * heads * vd;
  if (vd % V == 0 && aligned16(x))
    gate_per_head_kernel<T, V><<<elementwise_blocks(n / V), 256, 0, s>>>((T*)x, (const T*)gate, gs, n_tokens, heads, vd);
  else
    gate_per_head_kernel<T, 1><<<elementwise_blocks(n), 256, 0, s>>>((T*)x, (const T*)gate, gs, n_tokens, heads, vd);
  PACE_LAUNCH_CHECK("gate_per_head_kernel");
  return PACE_OK;
}

template <typename T, int ACT, bool GATED>
int glu_t(const void* x, int64_t xs, void* out, int64_t os, int n_tokens, int n, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const size_t total = (size_t)n_tokens * n;
  if (n % V == 0 && xs % V == 0 && os % V == 0 && aligned16(x) && aligned16(out))
    glu_kernel<T, V, ACT, GATED><<<elementwise_blocks(total / V), 256, 0, s>>>((const T*)x, xs, (T*)out, os, n_tokens, n);
  else
    glu_kernel<T, 1, ACT, GATED><<<elementwise_blocks(total), 256, 0, s>>>((const T*)x, xs, (T*)out, os, n_tokens, n);
  PACE_LAUNCH_CHECK("glu_kernel");
  return PACE_OK;
}

template <typename T, bool GATED>
int glu_act(const void* x, int64_t xs, void* out, int64_t os, int n_tokens, int n, int act, cudaStream_t s) {
  if (act == PACE_ACT_SILU) return glu_t<T, PACE_ACT_SILU, GATED>(x, xs, out, os, n_tokens, n, s);
  if (act == PACE_ACT_GELU_TANH) return glu_t<T, PACE_ACT_GELU_TANH, GATED>(x, xs, out, os, n_tokens, n, s);
  return glu_t<T, PACE_ACT_GELU_ERF, GATED>(x, xs, out, os, n_tokens, n, s);
}

bool dtype_ok(int dtype) { return dtype == PACE_DTYPE_BF16 || dtype == PACE_DTYPE_FP32; }

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_residual_norm(const pace_step_t* st, const pace_residual_norm_args_t* a, void* stream) {
  if (!step_ok(st) || !a || !a->x || a->width < 1 || !dtype_ok(a->dtype)) return PACE_ERR_INVALID;
  if ((a->w_next2 == nullptr) != (a->h2 == nullptr) || (a->h2 && !a->w_next) || ((a->add || a->y_bias) && !a->y) ||
      (a->add && a->add_stride < a->width) || (a->embed_norm && !a->embed))
    return PACE_ERR_INVALID;
  if ((a->w_next && !a->h) || (a->embed && a->vocab < 1) || (a->y && a->y_stride < a->width)) return PACE_ERR_INVALID;
  if (a->top < 0 || (a->top > 0 && (!a->y || a->top > kMaxTop || (a->n_experts < a->top && !a->identity) || !a->slot_expert || !a->slot_rank ||
                                    !a->slot_weight || !a->expert_count)))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("residual_norm", stream, "tokens=%d width=%d", st->n_tokens, a->width);
  const cudaStream_t s = (cudaStream_t)stream;
  // four elements per access: 16 bytes of fp32, 8 of bf16
  const bool vec = a->width % 4 == 0 && a->y_stride % 4 == 0 && aligned16(a->x) && aligned16(a->y) && aligned16(a->h) &&
                   aligned16(a->embed) && aligned16(a->w_post) && aligned16(a->w_next) && aligned16(a->w_next2) && aligned16(a->h2) &&
                   aligned16(a->identity) && aligned16(a->add) && a->add_stride % 4 == 0 && aligned16(a->y_bias) &&
                   aligned16(a->embed_norm);
  if (a->dtype == PACE_DTYPE_BF16)
    return vec ? launch_residual_norm<__nv_bfloat16, 4>(*st, *a, s) : launch_residual_norm<__nv_bfloat16, 1>(*st, *a, s);
  return vec ? launch_residual_norm<float, 4>(*st, *a, s) : launch_residual_norm<float, 1>(*st, *a, s);
}

int pace_kv_append_norm(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const pace_append_norm_args_t* a,
                        void* stream) {
  if (!p || !p->pages || !p->block_table || !step_ok(st) || !a || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (!a->qkv || !a->q_out || a->n_q_heads < 1 || a->dim < 1 || a->vdim < 1 || !dtype_ok(a->dtype)) return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_SHARED) return PACE_ERR_UNSUPPORTED;
  if (a->per_head && (a->q_norm || a->k_norm)) return PACE_ERR_INVALID;
  if (a->n_q_heads % p->n_kv_heads || (a->temp_coef != 0.f && !(a->temp_every > 0.0))) return PACE_ERR_INVALID;
  if (p->row_format == PACE_ROWS_BF16 && a->dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("kv_append_norm", stream, "layer=%d tokens=%d", layer, st->n_tokens);
  return a->dtype == PACE_DTYPE_BF16 ? launch_append_norm<__nv_bfloat16>(p, layer, *st, *a, (cudaStream_t)stream)
                                     : launch_append_norm<float>(p, layer, *st, *a, (cudaStream_t)stream);
}

int pace_gate_heads(const pace_step_t* st, const void* attn, const void* gate, int64_t gs, void* out, int32_t H, int32_t vd,
                    int32_t row, int32_t dtype, void* stream) {
  if (!step_ok(st) || !attn || !gate || !out || H < 1 || vd < 1 || row < vd || !dtype_ok(dtype)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  return dtype == PACE_DTYPE_BF16 ? gate_heads_t<__nv_bfloat16>(*st, attn, gate, gs, out, H, vd, row, (cudaStream_t)stream)
                                  : gate_heads_t<float>(*st, attn, gate, gs, out, H, vd, row, (cudaStream_t)stream);
}

int pace_norm_gate(const void* o, const float* w, const void* gate, int64_t gs, void* out, int32_t n_tokens, int32_t n,
                   float eps, int32_t dtype, void* stream) {
  if (!o || !w || !gate || !out || n_tokens < 0 || n < 1 || !dtype_ok(dtype)) return PACE_ERR_INVALID;
  if (n_tokens == 0) return PACE_OK;
  return dtype == PACE_DTYPE_BF16 ? norm_gate_t<__nv_bfloat16>(o, w, gate, gs, out, n_tokens, n, eps, (cudaStream_t)stream)
                                  : norm_gate_t<float>(o, w, gate, gs, out, n_tokens, n, eps, (cudaStream_t)stream);
}

int pace_gate_per_head(void* x, const void* gate, int64_t gs, int32_t n_tokens, int32_t heads, int32_t vd, int32_t dtype, void* stream) {
  if (!x || !gate || n_tokens < 0 || heads < 1 || vd < 1 || gs < heads || !dtype_ok(dtype)) return PACE_ERR_INVALID;
  if (n_tokens == 0) return PACE_OK;
  return dtype == PACE_DTYPE_BF16 ? gate_per_head_t<__nv_bfloat16>(x, gate, gs, n_tokens, heads, vd, (cudaStream_t)stream)
                                  : gate_per_head_t<float>(x, gate, gs, n_tokens, heads, vd, (cudaStream_t)stream);
}

int pace_relu_squared(void* x, int64_t n, int32_t dtype, void* stream) {
  if (!x || n < 0 || !dtype_ok(dtype)) return PACE_ERR_INVALID;
  if (n == 0) return PACE_OK;
  return dtype == PACE_DTYPE_BF16 ? relu_squared_t<__nv_bfloat16>(x, n, (cudaStream_t)stream)
                                  : relu_squared_t<float>(x, n, (cudaStream_t)stream);
}

int pace_glu(const void* x, int64_t x_stride, void* out, int64_t out_stride, int32_t n_tokens, int32_t n, int32_t act, int32_t gated,
             int32_t dtype, void* stream) {
  if (!x || !out || n_tokens < 0 || n < 1 || x_stride < (gated ? 2 : 1) * (int64_t)n || out_stride < n || !dtype_ok(dtype))
    return PACE_ERR_INVALID;
  if (act != PACE_ACT_SILU && act != PACE_ACT_GELU_TANH && act != PACE_ACT_GELU_ERF) return PACE_ERR_INVALID;
  if (n_tokens == 0) return PACE_OK;
  const cudaStream_t s = (cudaStream_t)stream;
  if (dtype == PACE_DTYPE_BF16)
    return gated ? glu_act<__nv_bfloat16, true>(x, x_stride, out, out_stride, n_tokens, n, act, s)
                 : glu_act<__nv_bfloat16, false>(x, x_stride, out, out_stride, n_tokens, n, act, s);
  return gated ? glu_act<float, true>(x, x_stride, out, out_stride, n_tokens, n, act, s)
               : glu_act<float, false>(x, x_stride, out, out_stride, n_tokens, n, act, s);
}

int pace_soft_cap(float* x, int64_t n, float cap, void* stream) {
  if (!x || n < 0 || !(cap > 0.f)) return PACE_ERR_INVALID;
  if (n == 0) return PACE_OK;
  soft_cap_kernel<<<elementwise_blocks((size_t)n), 256, 0, (cudaStream_t)stream>>>(x, n, cap);
  PACE_LAUNCH_CHECK("soft_cap_kernel");
  return PACE_OK;
}

int pace_part_norm_gate(const pace_part_norm_gate_args_t* a, void* stream) {
  if (!a || !a->o || !a->gate || !a->w || !a->out || a->n_tokens < 0 || a->part < 1 || a->n < a->part || a->n % a->part ||
      a->w_period < 1 || a->gate_mode < PACE_GATE_SIGMOID || a->gate_mode > PACE_GATE_SILU || a->o_stride < a->n || a->gate_stride < a->n || a->out_stride < a->n || !dtype_ok(a->dtype))
    return PACE_ERR_INVALID;
  if (a->n_tokens == 0) return PACE_OK;
  if ((int64_t)a->n_tokens * (a->n / a->part) > 0x3fffffff) return PACE_ERR_UNSUPPORTED;
  return a->dtype == PACE_DTYPE_BF16 ? part_norm_gate_t<__nv_bfloat16>(*a, (cudaStream_t)stream)
                                     : part_norm_gate_t<float>(*a, (cudaStream_t)stream);
}

int pace_step_decode(int32_t* token, int32_t* tok_pos, int32_t* start, const int64_t* next, const int64_t* pos, int32_t n,
                     void* stream) {
  if (!token || !tok_pos || !start || !next || !pos || n < 0) return PACE_ERR_INVALID;
  if (n == 0) return PACE_OK;
  step_decode_kernel<<<(n + 127) / 128, 128, 0, (cudaStream_t)stream>>>(token, tok_pos, start, next, pos, n);
  PACE_LAUNCH_CHECK("step_decode_kernel");
  return PACE_OK;
}

}  // extern "C"
