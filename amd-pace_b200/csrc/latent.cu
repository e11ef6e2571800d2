// What surrounds the products of latent attention: norms and rotation of one token's down projections on their way to
// the pages, rotation of query parts, gathering of page rows for the expanded form.  fp32 arithmetic.
#include "hybrid.cuh"

namespace pace {
namespace {

struct LatentRows {
  const int32_t* block_table;
  int32_t* status;
  char* rows;      // this layer's rows
  int page_tokens, max_pages_per_seq, max_seqs, n_pages;
};

LatentRows latent_rows(const pace_kv_pool_t* p, int layer) {
  LatentRows r;
  const size_t region = (size_t)p->n_pages * p->n_kv_heads * p->page_tokens * p->head_dim * 2;  // bytes
  r.block_table = p->block_table;
  r.status = p->status;
  r.rows = static_cast<char*>(p->pages) + (size_t)layer * region;
  r.page_tokens = p->page_tokens;
  r.max_pages_per_seq = p->max_pages_per_seq;
  r.max_seqs = p->max_seqs;
  r.n_pages = p->n_pages;
  return r;
}

__device__ __forceinline__ int latent_page(const LatentRows& r, int slot, int lp) {
  int page = -1;
  if (slot >= 0 && slot < r.max_seqs && lp >= 0 && lp < r.max_pages_per_seq)
    page = r.block_table[(size_t)slot * r.max_pages_per_seq + lp];
  return page < r.n_pages ? page : -1;
}

// (u, v) of a pair at angle (c, s) -> (u c - v s, v c + u s)
__device__ __forceinline__ void turn(float c, float s, float& u, float& v) {
  const float a = u * c - v * s;
  v = v * c + u * s;
  u = a;
}

// One block per token; threads 0 .. W - 1 (a whole number of warps) serve the query latent, the others the key/value
// latent, so that both norms are reduced at the same time.
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_append_kernel(pace_step_t st, LatentRows lr, pace_latent_append_args_t a, int row) {
  __shared__ float red[8];
  const int t = blockIdx.x, half = blockDim.x >> 1;
  const bool kv = (int)threadIdx.x >= half;
  const int tid = kv ? threadIdx.x - half : threadIdx.x;
  const int n = kv ? a.kv_rank : a.q_rank;
  const T* src = static_cast<const T*>(a.down) + (size_t)t * a.down_stride + (kv ? a.q_rank : 0);
  const int pos = st.tok_pos[t], lp = pos / lr.page_tokens;
  const int page = kv ? latent_page(lr, st.slot[st.tok_entry[t]], lp) : 0;   // (in flight while the norm is summed)
  float ss = 0.f;
  for (int c = tid * V; c < n; c += half * V) {
    float x[V];
    Vec<T, V>::load(src + c, x);
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(x[j], x[j], ss);
  }
#pragma unroll
  for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  const int warps = half >> 5;
  ss = 0.f;
  for (int w = 0; w < warps; ++w) ss += red[(kv ? warps : 0) + w];
  const float r = 1.0f / sqrtf(ss / (float)n + a.eps);
  T* dst = kv ? nullptr : static_cast<T*>(a.cq) + (size_t)t * n;
  const float* wt = kv ? a.kv_norm : a.q_norm;
  if (kv) {
    if (page < 0) {
      if (tid == 0) raise_status(lr.status, PACE_DEV_BAD_INDEX);
      return;
    }
    dst = reinterpret_cast<T*>(lr.rows) + ((size_t)page * lr.page_tokens + (pos - lp * lr.page_tokens)) * row;
  }
  for (int c = tid * V; c < n; c += half * V) {
    float x[V], w[V];
    Vec<T, V>::load(src + c, x);
    Vec<float, V>::load(wt + c, w);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= r * w[j];
    Vec<T, V>::store(dst + c, x);
  }
  if (!kv) return;
  if (a.rot_pairs > 0 && pos >= a.table_rows) {
    if (tid == 0) raise_status(lr.status, PACE_DEV_BAD_INDEX);
    return;
  }
  const float *cs = a.cos_table + (size_t)pos * a.rot_pairs, *sn = a.sin_table + (size_t)pos * a.rot_pairs;
  for (int i = tid; 2 * i < row - n; i += half) {
    const int c = 2 * i;
    float u = c < a.rot_dim ? to_f<T>(src[n + c]) : 0.f, v = c + 1 < a.rot_dim ? to_f<T>(src[n + c + 1]) : 0.f;
    if (i < a.rot_pairs) turn(cs[i], sn[i], u, v);
    dst[n + c] = from_f<T>(u);
    if (n + c + 1 < row) dst[n + c + 1] = from_f<T>(v);
  }
}

// a thread per pair of (token, head)
template <typename T>
__global__ void rotate_heads_kernel(pace_step_t st, pace_rotate_args_t a) {
  const int pairs = (a.pad_dim + 1) / 2;
  const size_t total = (size_t)(a.token_end - a.token_begin) * a.n_heads * pairs;
  for (size_t k = blockIdx.x * (size_t)blockDim.x + threadIdx.x; k < total; k += (size_t)gridDim.x * blockDim.x) {
    const int i = (int)(k % pairs), h = (int)(k / pairs % a.n_heads);
    const int t = a.token_begin + (int)(k / ((size_t)pairs * a.n_heads)), c = 2 * i;
    const T* src = static_cast<const T*>(a.src) + t * a.src_row + h * a.src_head;
    T* dst = static_cast<T*>(a.dst) + t * a.dst_row + h * a.dst_head;
    float u = c < a.rot_dim ? to_f<T>(src[c]) : 0.f, v = c + 1 < a.rot_dim ? to_f<T>(src[c + 1]) : 0.f;
    const int pos = st.tok_pos[t];
    if (i < a.rot_pairs && pos < a.table_rows)
      turn(a.cos_table[(size_t)pos * a.rot_pairs + i], a.sin_table[(size_t)pos * a.rot_pairs + i], u, v);
    dst[c] = from_f<T>(u);
    if (c + 1 < a.pad_dim) dst[c + 1] = from_f<T>(v);
  }
}

// the same, four pairs (16 bytes of bf16) a thread
__global__ void rotate_heads_vec_kernel(pace_step_t st, pace_rotate_args_t a) {
  const int per = a.pad_dim / 8;
  const size_t total = (size_t)(a.token_end - a.token_begin) * a.n_heads * per;
  for (size_t k = blockIdx.x * (size_t)blockDim.x + threadIdx.x; k < total; k += (size_t)gridDim.x * blockDim.x) {
    const int c = (int)(k % per) * 8, h = (int)(k / per % a.n_heads), t = a.token_begin + (int)(k / ((size_t)per * a.n_heads));
    float x[8];
    if (c < a.rot_dim) {
      Vec<__nv_bfloat16, 8>::load(static_cast<const __nv_bfloat16*>(a.src) + t * a.src_row + h * a.src_head + c, x);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = 0.f;
    }
    const int pos = st.tok_pos[t];
    if (c / 2 + 4 <= a.rot_pairs && pos < a.table_rows) {
      float cs[4], sn[4];
      Vec<float, 4>::load(a.cos_table + (size_t)pos * a.rot_pairs + c / 2, cs);
      Vec<float, 4>::load(a.sin_table + (size_t)pos * a.rot_pairs + c / 2, sn);
#pragma unroll
      for (int j = 0; j < 4; ++j) turn(cs[j], sn[j], x[2 * j], x[2 * j + 1]);
    }
    Vec<__nv_bfloat16, 8>::store(static_cast<__nv_bfloat16*>(a.dst) + t * a.dst_row + h * a.dst_head + c, x);
  }
}

// a thread per 16 bytes
__global__ void latent_gather_kernel(LatentRows lr, const int32_t* __restrict__ slot, const int32_t* __restrict__ pos, int n,
                                     uint4* __restrict__ out, int pieces) {
  const size_t total = (size_t)n * pieces;
  for (size_t k = blockIdx.x * (size_t)blockDim.x + threadIdx.x; k < total; k += (size_t)gridDim.x * blockDim.x) {
    const int i = (int)(k / pieces), c = (int)(k % pieces), p = pos[i], lp = p / lr.page_tokens;
    const int page = latent_page(lr, slot[i], lp);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (page >= 0)
      v = reinterpret_cast<const uint4*>(lr.rows)[((size_t)page * lr.page_tokens + (p - lp * lr.page_tokens)) * pieces + c];
    else
      raise_status(lr.status, PACE_DEV_BAD_INDEX);
    out[k] = v;
  }
}

unsigned blocks_for(size_t threads) {
  const size_t b = (threads + 255) / 256;
  return (unsigned)(b < 1 ? 1 : b > 148 * 16 ? 148 * 16 : b);
}

template <typename T>
int append_t(const pace_kv_pool_t* p, int layer, const pace_step_t& st, const pace_latent_append_args_t& a, cudaStream_t s) {
  const int row = p->head_dim * 2 / (int)sizeof(T);
  if (a.kv_rank + a.rot_dim > row) return PACE_ERR_INVALID;
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.q_rank % V == 0 && a.kv_rank % V == 0 && a.down_stride % V == 0 && aligned16(a.down) && aligned16(a.cq) &&
                   aligned16(a.q_norm) && aligned16(a.kv_norm) && row % V == 0;
  if (vec) latent_append_kernel<T, V><<<st.n_tokens, 128, 0, s>>>(st, latent_rows(p, layer), a, row);
  else latent_append_kernel<T, 1><<<st.n_tokens, 256, 0, s>>>(st, latent_rows(p, layer), a, row);
  PACE_LAUNCH_CHECK("latent_append_kernel");
  note_pool_write(s);
  return PACE_OK;
}

bool latent_pool_ok(const pace_kv_pool_t* p, int layer) {
  return p && p->pages && p->block_table && p->row_format == PACE_ROWS_SHARED && p->n_kv_heads == 1 && layer >= 0 &&
         layer < p->n_layers;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_latent_append(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const pace_latent_append_args_t* a,
                       void* stream) {
  if (!latent_pool_ok(p, layer) || !step_ok(st) || !a || !a->down || !a->kv_norm || a->kv_rank < 1 || a->q_rank < 0 ||
      a->rot_dim < 0 || a->rot_pairs < 0 || 2 * a->rot_pairs > a->rot_dim)
    return PACE_ERR_INVALID;
  if ((a->q_rank > 0 && (!a->cq || !a->q_norm)) || (a->rot_pairs > 0 && (!a->cos_table || !a->sin_table || a->table_rows < 1)))
    return PACE_ERR_INVALID;
  if (a->dtype != PACE_DTYPE_BF16 && a->dtype != PACE_DTYPE_FP32) return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("latent_append", stream, "layer=%d tokens=%d", layer, st->n_tokens);
  return a->dtype == PACE_DTYPE_BF16 ? append_t<__nv_bfloat16>(p, layer, *st, *a, (cudaStream_t)stream)
                                     : append_t<float>(p, layer, *st, *a, (cudaStream_t)stream);
}

int pace_rotate_heads(const pace_step_t* st, const pace_rotate_args_t* a, void* stream) {
  if (!step_ok(st) || !a || !a->src || !a->dst || a->token_begin < 0 || a->token_end > st->n_tokens || a->n_heads < 1 ||
      a->rot_dim < 0 || a->pad_dim < a->rot_dim || a->rot_pairs < 0 || 2 * a->rot_pairs > a->rot_dim)
    return PACE_ERR_INVALID;
  if (a->rot_pairs > 0 && (!a->cos_table || !a->sin_table)) return PACE_ERR_INVALID;
  if (a->token_begin >= a->token_end || a->pad_dim == 0) return PACE_OK;
  const size_t n = (size_t)(a->token_end - a->token_begin) * a->n_heads * ((a->pad_dim + 1) / 2);
  const bool vec = a->dtype == PACE_DTYPE_BF16 && a->rot_dim % 8 == 0 && a->pad_dim % 8 == 0 && a->rot_pairs % 4 == 0 &&
                   (a->src_row | a->src_head | a->dst_row | a->dst_head) % 8 == 0 && aligned16(a->src) && aligned16(a->dst) &&
                   aligned16(a->cos_table) && aligned16(a->sin_table);
  if (vec) rotate_heads_vec_kernel<<<blocks_for(n / 4), 256, 0, (cudaStream_t)stream>>>(*st, *a);
  else if (a->dtype == PACE_DTYPE_BF16) rotate_heads_kernel<__nv_bfloat16><<<blocks_for(n), 256, 0, (cudaStream_t)stream>>>(*st, *a);
  else if (a->dtype == PACE_DTYPE_FP32) rotate_heads_kernel<float><<<blocks_for(n), 256, 0, (cudaStream_t)stream>>>(*st, *a);
  else return PACE_ERR_INVALID;
  PACE_LAUNCH_CHECK("rotate_heads_kernel");
  return PACE_OK;
}

int pace_latent_gather(const pace_kv_pool_t* p, int32_t layer, const int32_t* slot, const int32_t* pos, int32_t n, void* out,
                       void* stream) {
  if (!latent_pool_ok(p, layer) || !slot || !pos || !out || n < 0 || !aligned16(out)) return PACE_ERR_INVALID;
  if (n == 0) return PACE_OK;
  const int pieces = p->head_dim / 8;
  latent_gather_kernel<<<blocks_for((size_t)n * pieces), 256, 0, (cudaStream_t)stream>>>(latent_rows(p, layer), slot, pos, n,
                                                                                        (uint4*)out, pieces);
  PACE_LAUNCH_CHECK("latent_gather_kernel");
  return PACE_OK;
}

}  // extern "C"
