// What lies between two layers whose mixers read shifted inputs: the residual stream takes up a sublayer's output and a vector, the
// sum is normalised, and every element is moved towards the previous token's; and the embedding of token pairs in front of
// the first layer.  The stream is read from one buffer and written to another, so that a block can make the norm of
// the token in front of its own once more instead of waiting for it.  fp32 arithmetic.
#include "hybrid.cuh"

namespace pace {
namespace {

template <typename T, int V, int ITEMS>
__global__ void __launch_bounds__(512) shift_norm_kernel(pace_step_t st, pace_shift_norm_args_t a, int per) {
  __shared__ float red[2][32];
  const int W = a.width, t0 = blockIdx.x * per, t1 = min(t0 + per, st.n_tokens);
  float prev[ITEMS][V], mix[ITEMS][V];
  int slot = -1;
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) mix[i][j] = prev[i][j] = 0.f;
    if (c < W) Vec<float, V>::load(a.shift + c, mix[i]);
  }
  // the token in front of the block's first one is made once more if it belongs to the same sequence; in a step of one token per
  // entry nothing has to be looked up
  const bool single = st.n_tokens == st.n_entries;
  for (int t = !single && t0 > st.cu[st.tok_entry[t0]] ? t0 - 1 : t0; t < t1; ++t) {
    const bool own = t >= t0;
    const int e = single ? t : st.tok_entry[t], start = st.start[e];
    slot = st.slot[e];
    float x[ITEMS][V], y[ITEMS][V];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) {
        Vec<float, V>::load(a.x_in + (size_t)t * W + c, x[i]);
        if (a.y) {
          Vec<T, V>::load(static_cast<const T*>(a.y) + (size_t)t * a.y_stride + c, y[i]);
          if (a.y_bias) {
            float b[V];
            Vec<float, V>::load(a.y_bias + c, b);
#pragma unroll
            for (int j = 0; j < V; ++j) y[i][j] += b[j];
          }
#pragma unroll
          for (int j = 0; j < V; ++j) ss = fmaf(y[i][j], y[i][j], ss);
        }
      }
    }
    if (single || t == st.cu[e]) {             // the previous token is the state's, or there is none
      const bool fresh = start == 0;
#pragma unroll
      for (int i = 0; i < ITEMS; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * V;
#pragma unroll
        for (int j = 0; j < V; ++j) prev[i][j] = 0.f;
        if (!fresh && c < W) Vec<float, V>::load(a.state + (size_t)slot * a.state_stride + c, prev[i]);
      }
    }
    if (a.y) {
      const float r = 1.0f / sqrtf(block_sum(ss, red[0]) / (float)W + a.eps);
#pragma unroll
      for (int i = 0; i < ITEMS; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * V;
        if (c < W) {
          float w[V];
          Vec<float, V>::load(a.w_post + c, w);
#pragma unroll
          for (int j = 0; j < V; ++j) x[i][j] += y[i][j] * r * w[j];
        }
      }
    }
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) {
        if (a.add) {
          float b[V];
          Vec<float, V>::load(a.add + c, b);
#pragma unroll
          for (int j = 0; j < V; ++j) x[i][j] += b[j];
        }
        if (own) Vec<float, V>::store(a.x_out + (size_t)t * W + c, x[i]);
#pragma unroll
        for (int j = 0; j < V; ++j) ss = fmaf(x[i][j], x[i][j], ss);
      }
    }
    const float r = 1.0f / sqrtf(block_sum(ss, red[1]) / (float)W + a.eps);
    const bool last = single || t + 1 == st.cu[e + 1];
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * V;
      if (c < W) {
        float w[V], h[V];
        Vec<float, V>::load(a.w_next + c, w);
#pragma unroll
        for (int j = 0; j < V; ++j) {
          w[j] *= x[i][j] * r;
          h[j] = fmaf(prev[i][j] - w[j], mix[i][j], w[j]);
          prev[i][j] = w[j];
        }
        if (own) {
          Vec<T, V>::store(static_cast<T*>(a.h) + (size_t)t * W + c, h);
          if (last) Vec<float, V>::store(a.state_out + (size_t)slot * a.state_stride + c, w);
        }
      }
    }
  }
}

// x = embed[token] * scale + pairs[(previous * mul_prev + token * mul_cur) mod buckets]
template <typename T, int V>
__global__ void __launch_bounds__(256) embed_pairs_kernel(pace_step_t st, pace_embed_pairs_args_t a) {
  const int t = blockIdx.x, e = st.tok_entry[t], tok = st.token[t], slot = st.slot[e];
  const bool first = t == st.cu[e];
  const T *em = nullptr, *pr = nullptr;
  int prev = -1;
  if (a.pairs) prev = !first ? st.token[t - 1] : st.start[e] > 0 ? a.last_token[slot] : -1;
  if (tok >= 0 && tok < a.vocab) em = static_cast<const T*>(a.embed) + (size_t)tok * a.width;
  if (a.pairs) {
    int64_t r = a.buckets;
    if (prev >= 0) {
      r = ((int64_t)prev * a.mul_prev + (int64_t)tok * a.mul_cur) % a.buckets;
      if (r < 0) r += a.buckets;
    }
    pr = static_cast<const T*>(a.pairs) + (size_t)r * a.width;
  }
  for (int c = threadIdx.x * V; c < a.width; c += blockDim.x * V) {
    float x[V], y[V];
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = 0.f;
    if (em) Vec<T, V>::load(em + c, x);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= a.scale;
    if (pr) {
      Vec<T, V>::load(pr + c, y);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += y[j];
    }
    Vec<float, V>::store(a.x + (size_t)t * a.width + c, x);
  }
  if (a.store_last) {                          // one token per entry: nobody else reads this slot's
    __syncthreads();
    if (threadIdx.x == 0) a.last_token[slot] = tok;
  }
}

// rows of the entries' slots, and their last tokens
__global__ void state_commit_kernel(pace_step_t st, const float* __restrict__ from, float* __restrict__ to, int64_t n, int64_t stride,
                                    int32_t* last_token) {
  const int e = blockIdx.y, slot = st.slot[e];
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x)
    to[(size_t)slot * stride + i] = from[(size_t)slot * stride + i];
  if (last_token && blockIdx.x == 0 && threadIdx.x == 0) last_token[slot] = st.token[st.cu[e + 1] - 1];
}

template <typename T, int V>
int launch_shift_norm(const pace_step_t& st, const pace_shift_norm_args_t& a, cudaStream_t s) {
  const int groups = (a.width + V - 1) / V;
  int threads = (groups + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int need = (groups + threads - 1) / threads;
  // tokens a block walks over: many tokens pay for one more per block
  const int per = st.n_tokens >= 148 * 16 ? 4 : st.n_tokens >= 148 * 4 ? 2 : 1;
  const unsigned grid = (unsigned)((st.n_tokens + per - 1) / per);
#define PACE_SHIFT_CASE(n) \
  if (need <= n) { shift_norm_kernel<T, V, n><<<grid, threads, 0, s>>>(st, a, per); PACE_LAUNCH_CHECK("shift_norm_kernel"); return PACE_OK; }
  PACE_SHIFT_CASE(1) PACE_SHIFT_CASE(2) PACE_SHIFT_CASE(4) PACE_SHIFT_CASE(8) PACE_SHIFT_CASE(16)
#undef PACE_SHIFT_CASE
  return PACE_ERR_UNSUPPORTED;
}

bool dtype_ok(int dtype) { return dtype == PACE_DTYPE_BF16 || dtype == PACE_DTYPE_FP32; }

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_shift_norm(const pace_step_t* st, const pace_shift_norm_args_t* a, void* stream) {
  if (!step_ok(st) || !a || !a->x_in || !a->x_out || !a->w_next || !a->shift || !a->h || !a->state || !a->state_out || a->width < 1 ||
      a->state_stride < a->width || !dtype_ok(a->dtype) || (a->y && (!a->w_post || a->y_stride < a->width)) || (a->y_bias && !a->y))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  // in place only where no block reads another one's tokens
  if ((a->x_in == a->x_out || a->state == a->state_out) && st->n_tokens != st->n_entries) return PACE_ERR_INVALID;
  PACE_PROFILE("shift_norm", stream, "tokens=%d width=%d", st->n_tokens, a->width);
  const cudaStream_t s = (cudaStream_t)stream;
  const bool vec = a->width % 4 == 0 && a->y_stride % 4 == 0 && a->state_stride % 4 == 0 && aligned16(a->x_in) && aligned16(a->x_out) &&
                   aligned16(a->y) && aligned16(a->y_bias) && aligned16(a->w_post) && aligned16(a->add) && aligned16(a->w_next) &&
                   aligned16(a->shift) && aligned16(a->state) && aligned16(a->state_out) && aligned16(a->h);
  if (a->dtype == PACE_DTYPE_BF16)
    return vec ? launch_shift_norm<__nv_bfloat16, 4>(*st, *a, s) : launch_shift_norm<__nv_bfloat16, 1>(*st, *a, s);
  return vec ? launch_shift_norm<float, 4>(*st, *a, s) : launch_shift_norm<float, 1>(*st, *a, s);
}

int pace_embed_pairs(const pace_step_t* st, const pace_embed_pairs_args_t* a, void* stream) {
  if (!step_ok(st) || !a || !a->x || !a->embed || a->width < 1 || a->vocab < 1 || !dtype_ok(a->dtype) ||
      (a->pairs && (!a->last_token || a->buckets < 1)) || (a->store_last && (!a->last_token || st->n_tokens != st->n_entries)))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0) return PACE_OK;
  const cudaStream_t s = (cudaStream_t)stream;
  const bool vec = a->width % 4 == 0 && aligned16(a->x) && aligned16(a->embed) && aligned16(a->pairs);
  if (a->dtype == PACE_DTYPE_BF16) {
    if (vec) embed_pairs_kernel<__nv_bfloat16, 4><<<st->n_tokens, 256, 0, s>>>(*st, *a);
    else embed_pairs_kernel<__nv_bfloat16, 1><<<st->n_tokens, 256, 0, s>>>(*st, *a);
  } else {
    if (vec) embed_pairs_kernel<float, 4><<<st->n_tokens, 256, 0, s>>>(*st, *a);
    else embed_pairs_kernel<float, 1><<<st->n_tokens, 256, 0, s>>>(*st, *a);
  }
  PACE_LAUNCH_CHECK("embed_pairs_kernel");
  return PACE_OK;
}

int pace_state_commit(const pace_step_t* st, const float* from, float* to, int64_t n, int64_t stride, int32_t* last_token, void* stream) {
  if (!step_ok(st) || !from || !to || n < 0 || stride < n) return PACE_ERR_INVALID;
  if (st->n_entries == 0 || (n == 0 && !last_token)) return PACE_OK;
  if (st->n_entries > 65535) return PACE_ERR_UNSUPPORTED;
  const int64_t blocks = (n + 1023) / 1024;
  state_commit_kernel<<<dim3((unsigned)(blocks < 1 ? 1 : blocks < 64 ? blocks : 64), (unsigned)st->n_entries), 256, 0, (cudaStream_t)stream>>>(
      *st, from, to, n, stride, last_token);
  PACE_LAUNCH_CHECK("state_commit_kernel");
  return PACE_OK;
}

}  // extern "C"
