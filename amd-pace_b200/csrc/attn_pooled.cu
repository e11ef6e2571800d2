// Attention over a window of tokens and pooled blocks whose softmax weights are mixed over the heads: decode, short portions of
// prompts, fp32.
//
// Mixing needs the weights of all heads of a (query, key) pair, finished: a head's share of the denominator is known once all
// its keys have been scored.  So a token is the unit of work, with all its heads.
//   attn_pooled_step_kernel     bf16 rows of 64 or 128: the blocks of a cluster share a token's keys; scores of all heads stay in shared
//                               memory, maxima and sums meet over the cluster, then weights, mixing and values; keys and values
//                               go from their pages to mma.sync fragments in registers and are read once
//   attn_pooled_general_kernel  everything else: scores twice, once for the sums, once for the weights; CUDA cores, fp32
// A query head's output is multiplied by sigmoid(gate) on its way out.
#include <cooperative_groups.h>

#include "pooled.cuh"

namespace cg = cooperative_groups;

namespace pace {
namespace {

// ---------------------------------------------------------------------------------------------------------------------
// any sizes, either format
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kTile = 32, kGenThreads = 256;

struct GeneralSmem {
  int q, tile, p, mixed, o, ml, total;   // floats
};
__host__ __device__ inline GeneralSmem general_smem(int H, int d, int vd) {
  GeneralSmem m;
  int off = 0;
  auto take = [&](int n) {
    const int o = off;
    off += (n + 3) / 4 * 4;
    return o;
  };
  m.q = take(H * d);
  m.tile = take(kTile * ((d > vd ? d : vd) | 1));
  m.p = take(H * kTile);
  m.mixed = take(H * kTile);
  m.o = take(H * vd);
  m.ml = take(2 * H);
  m.total = off;
  return m;
}

template <typename T>
__global__ void __launch_bounds__(kGenThreads) attn_pooled_general_kernel(KVView kv, KVView bk, pace_step_t st, pace_attn_pooled_args_t a) {
  extern __shared__ __align__(16) float smem_f[];
  const int H = a.n_q_heads, G = kv.n_kv_heads, Gq = H / G, d = a.dim, vd = a.vdim, row = a.q_elems;
  const GeneralSmem L = general_smem(H, d, vd);
  float *q = smem_f + L.q, *tile = smem_f + L.tile, *p = smem_f + L.p, *mixed = smem_f + L.mixed, *o = smem_f + L.o, *ml = smem_f + L.ml;
  const int t = a.token_begin + blockIdx.x, e = st.tok_entry[t], pos = st.tok_pos[t], slot = st.slot[e];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (slot < 0 || slot >= kv.max_seqs) {
    if (tid == 0) raise_status(kv.status, PACE_DEV_BAD_INDEX);
    return;
  }
  for (int i = tid; i < H * d; i += kGenThreads) q[i] = to_f<T>(static_cast<const T*>(a.q)[((size_t)t * H + i / d) * row + i % d]);
  for (int i = tid; i < H * vd; i += kGenThreads) o[i] = 0.f;
  for (int h = tid; h < H; h += kGenThreads) {
    ml[2 * h] = a.sinks ? a.sinks[h] : -INFINITY;        // a sink is one more term of the denominator
    ml[2 * h + 1] = a.sinks ? 1.f : 0.f;
  }
  const int nb = blocks_seen(pos, a.window, a.block), first = window_first(pos, a.window);
  const int b_tiles = (nb + kTile - 1) / kTile, tiles = b_tiles + (pos - first) / kTile + 1;
  // keys or values of a tile for KV head g
  auto fetch = [&](int it, int g, bool is_v) {
    const bool blk = it < b_tiles;
    const KVView& v = blk ? bk : kv;
    const int i0 = blk ? it * kTile : first + (it - b_tiles) * kTile, n = blk ? nb : pos + 1, w = is_v ? vd : d;
    __syncthreads();
    for (int i = tid; i < kTile * w; i += kGenThreads) {
      const int j = i / w, c = i - j * w, idx = i0 + j;
      float x = 0.f;
      if (idx < n) {
        const int pg = view_page(v, slot, idx / v.page_tokens);
        if (pg < 0) raise_status(v.status, PACE_DEV_BAD_INDEX);
        else x = to_f<T>(reinterpret_cast<const T*>(is_v ? v.v : v.k)[(((size_t)pg * G + g) * v.page_tokens + idx % v.page_tokens) * row + c]);
      }
      tile[j * (w | 1) + c] = x;
    }
    __syncthreads();
    return min(kTile, n - i0);
  };
  for (int pass = 0; pass < 2; ++pass)
    for (int it = 0; it < tiles; ++it) {
      for (int g = 0; g < G; ++g) {
        const int n = fetch(it, g, false);
        for (int hh = warp; hh < Gq; hh += kGenThreads / 32) {
          const int h = g * Gq + hh;
          float s = 0.f;
          for (int c = 0; c < d; ++c) s = fmaf(q[h * d + c], tile[lane * (d | 1) + c], s);
          s = lane < n ? s * a.scale : -INFINITY;
          const float m = ml[2 * h], l = ml[2 * h + 1];
          if (pass == 0) {
            float mx = s;
#pragma unroll
            for (int w = 16; w; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
            mx = fmaxf(mx, m);
            float sum = expf(s - mx);
#pragma unroll
            for (int w = 16; w; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
            __syncwarp();
            if (lane == 0) {
              ml[2 * h] = mx;
              ml[2 * h + 1] = l * expf(m - mx) + sum;
            }
          } else {
            p[h * kTile + lane] = expf(s - m) / l;
          }
        }
      }
      if (pass == 0) continue;
      __syncthreads();
      for (int i = tid; i < H * kTile; i += kGenThreads) {
        const int h = i / kTile, j = i % kTile;
        float w = p[i];
        if (a.mix) {
          w = 0.f;
          for (int g = 0; g < H; ++g) w = fmaf(a.mix[h * H + g], p[g * kTile + j], w);
        }
        mixed[i] = w;
      }
      for (int g = 0; g < G; ++g) {
        const int n = fetch(it, g, true);
        for (int i = tid; i < Gq * vd; i += kGenThreads) {
          const int hh = i / vd, c = i - hh * vd;
          float s = o[g * Gq * vd + i];
          for (int j = 0; j < n; ++j) s = fmaf(mixed[(g * Gq + hh) * kTile + j], tile[j * (vd | 1) + c], s);
          o[g * Gq * vd + i] = s;
        }
      }
    }
  __syncthreads();
  for (int i = tid; i < H * vd; i += kGenThreads) {
    float y = o[i];
    if (a.gate) y *= sigmoid_t<T>(to_f<T>(static_cast<const T*>(a.gate)[(size_t)t * a.gate_stride + i]));
    static_cast<T*>(a.out)[(size_t)t * a.out_stride + i] = from_f<T>(y);
  }
}

template <typename T>
int launch_general(const KVView& kv, const KVView& bk, const pace_step_t& st, const pace_attn_pooled_args_t& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (size_t)general_smem(a.n_q_heads, a.dim, a.vdim).total;
  if (smem > 227 * 1024) return PACE_ERR_UNSUPPORTED;
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_pooled_general_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  attn_pooled_general_kernel<T><<<a.token_end - a.token_begin, kGenThreads, smem, s>>>(kv, bk, st, a);
  PACE_LAUNCH_CHECK("attn_pooled_general_kernel");
  return PACE_OK;
}

// ---------------------------------------------------------------------------------------------------------------------
// bf16 rows of 64 or 128
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kWarps = 16, kThreads = 32 * kWarps, kMaxCluster = 8;

__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// A block's share is `cap` keys in groups of 16: row numbers, scores (then nothing), weights in two bf16 terms; later the
// warps' outputs take the scores' place.
struct StepSmem {
  int rows, scores, hi, lo, ml, mix, total;   // bytes
  int pitch_s, pitch_w, pitch_m;              // elements of a head's row
};
// warps that share a task's keys, each with outputs of its own
__host__ __device__ inline int step_sets(int tasks) { return kWarps / tasks > 1 ? kWarps / tasks : 1; }
__host__ __device__ inline StepSmem step_smem(int H, int cap, int dp, int o_sets) {
  StepSmem m;
  int off = 0;
  auto take = [&](int bytes) {
    const int o = off;
    off += (bytes + 15) / 16 * 16;
    return o;
  };
  m.pitch_s = cap + 4;
  m.pitch_w = cap + 8;                        // 4 words more than a multiple of 8: the lanes of a fragment hit different banks
  m.rows = take(cap * 4);
  const int sb = H * m.pitch_s * 4, ob = o_sets * H * dp * 4;
  m.scores = take(sb > ob ? sb : ob);
  m.hi = take(H * m.pitch_w * 2);
  m.lo = take(H * m.pitch_w * 2);
  m.ml = take(H * 16);
  m.pitch_m = (H + 7) / 8 * 8;                // (what lies behind the last head is multiplied and not stored)
  m.mix = take(H * m.pitch_m * 4);
  m.total = off;
  return m;
}

// DP: elements of a row; a token's keys are blocks [0, nb) in groups of 16, then tokens [first, pos] in groups of 16
template <int DP>
__global__ void __launch_bounds__(kThreads, 1) attn_pooled_step_kernel(KVView kv, KVView bk, pace_step_t st, pace_attn_pooled_args_t a, int cap, int o_sets) {
  extern __shared__ __align__(16) unsigned char sm[];
  cg::cluster_group cl = cg::this_cluster();
  const int ns = gridDim.x, share = blockIdx.x, t = a.token_begin + blockIdx.y;
  const int H = a.n_q_heads, G = kv.n_kv_heads, Gq = H / G;
  const StepSmem L = step_smem(H, cap, DP, o_sets);
  int* rows = reinterpret_cast<int*>(sm + L.rows);
  float* S = reinterpret_cast<float*>(sm + L.scores);
  __nv_bfloat16* w_hi = reinterpret_cast<__nv_bfloat16*>(sm + L.hi);
  __nv_bfloat16* w_lo = reinterpret_cast<__nv_bfloat16*>(sm + L.lo);
  float2* ml = reinterpret_cast<float2*>(sm + L.ml);         // this block's, then [H ..): the token's (reference, factor)
  float* mixer = reinterpret_cast<float*>(sm + L.mix);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int e = st.tok_entry[t], pos = st.tok_pos[t];
  int slot = st.slot[e];
  if (slot < 0 || slot >= kv.max_seqs) {                      // (nobody leaves before the cluster's barriers)
    if (tid == 0) raise_status(kv.status, PACE_DEV_BAD_INDEX);
    slot = 0;
  }
  const int nb = blocks_seen(pos, a.window, a.block), first = window_first(pos, a.window);
  const int b_groups = (nb + 15) / 16, groups = b_groups + (pos - first) / 16 + 1, per = (groups + ns - 1) / ns;
  const int ga = min(share * per, groups), gz = min(ga + per, groups), n_keys = (gz - ga) * 16;   // (at most cap)
  // ---- where the share's rows lie: (page x G) x page rows + row, of the blocks' or the tokens' pages ----
  for (int i = tid; i < n_keys; i += kThreads) {
    const int gi = ga + i / 16;
    const bool blk = gi < b_groups;
    const KVView& v = blk ? bk : kv;
    const int idx = blk ? min(gi * 16 + (i & 15), nb - 1) : min(first + (gi - b_groups) * 16 + (i & 15), pos);   // (a group's rest repeats a row)
    int pg = view_page(v, slot, idx / v.page_tokens);
    if (pg < 0) {
      raise_status(v.status, PACE_DEV_BAD_INDEX);
      pg = 0;
    }
    rows[i] = pg * G * v.page_tokens + idx % v.page_tokens;
  }
  if (a.mix)       // by key head, so that neighbouring heads lie side by side
    for (int i = tid; i < H * H; i += kThreads) mixer[i % H * L.pitch_m + i / H] = a.mix[i];
  __syncthreads();
  // the values are on their way to L2 while the keys are scored
  for (int i = tid; i < n_keys * G * (DP / 64); i += kThreads) {
    const int j = i / (G * (DP / 64)), r = i - j * (G * (DP / 64)), gi = ga + j / 16;
    const bool blk = gi < b_groups;
    const __nv_bfloat16* at = (blk ? bk.v : kv.v) + (size_t)(rows[j] + r / (DP / 64) * (blk ? bk.page_tokens : kv.page_tokens)) * DP + r % (DP / 64) * 64;
    asm volatile("prefetch.global.L2 [%0];" ::"l"(at));
  }

  // a task is up to eight heads of a KV head; warps of a task, the task this warp begins with
  const int tiles = (Gq + 7) / 8, tasks = G * tiles, wpg = step_sets(tasks), sub = warp % wpg, set = warp / wpg, n_sets = kWarps / wpg;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + (size_t)t * H * DP;
  // ---- scores: 16 keys are the row operand, up to 8 heads the columns; lane's 8 neighbouring columns per slab of 32 ----
  for (int task = set; task < tasks; task += n_sets) {
      const int gk = task / tiles, h0 = task % tiles * 8;
      uint4 qf[DP / 32];
#pragma unroll
      for (int s = 0; s < DP / 32; ++s)
        qf[s] = h0 + g < Gq ? *reinterpret_cast<const uint4*>(q + (size_t)(gk * Gq + h0 + g) * DP + 32 * s + 8 * tq) : make_uint4(0, 0, 0, 0);
#pragma unroll 2
      for (int gi = ga + sub; gi < gz; gi += wpg) {
        const bool blk = gi < b_groups;
        const __nv_bfloat16* base = blk ? bk.k : kv.k;
        const int page_rows = blk ? bk.page_tokens : kv.page_tokens, i0 = (gi - ga) * 16;
        const uint4* r0 = reinterpret_cast<const uint4*>(base + (size_t)(rows[i0 + g] + gk * page_rows) * DP + 8 * tq);
        const uint4* r1 = reinterpret_cast<const uint4*>(base + (size_t)(rows[i0 + g + 8] + gk * page_rows) * DP + 8 * tq);
        uint4 k0[DP / 32], k1[DP / 32];
#pragma unroll
        for (int s = 0; s < DP / 32; ++s) {
          k0[s] = __ldg(r0 + 4 * s);
          k1[s] = __ldg(r1 + 4 * s);
        }
        float c[4] = {0.f, 0.f, 0.f, 0.f}, c2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int s = 0; s < DP / 32; ++s) {
          mma16816(c, k0[s].x, k1[s].x, k0[s].y, k1[s].y, qf[s].x, qf[s].y);
          mma16816(c2, k0[s].z, k1[s].z, k0[s].w, k1[s].w, qf[s].z, qf[s].w);
        }
        const int left = blk ? nb - gi * 16 : pos + 1 - first - (gi - b_groups) * 16;   // keys of the group
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int j = g + (x >> 1) * 8, h = h0 + 2 * tq + (x & 1);
          if (h < Gq) S[(gk * Gq + h) * L.pitch_s + i0 + j] = j < left ? (c[x] + c2[x]) * a.scale * kLog2e : -INFINITY;
        }
      }
    }
  __syncthreads();
  // ---- maxima and sums (log2 units), over the cluster; a sink is one more term ----
  for (int h = warp; h < H; h += kWarps) {
    float m = -INFINITY, l = 0.f;
    for (int i = lane; i < n_keys; i += 32) m = fmaxf(m, S[h * L.pitch_s + i]);
#pragma unroll
    for (int w = 16; w; w >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, w));
    for (int i = lane; i < n_keys; i += 32) l += fast_exp2(S[h * L.pitch_s + i] - m);
#pragma unroll
    for (int w = 16; w; w >>= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
    if (lane == 0) ml[h] = make_float2(m, n_keys ? l : 0.f);
  }
  if (ns > 1) cl.sync();
  else __syncthreads();
  for (int h = tid; h < H; h += kThreads) {
    float2 s[kMaxCluster];
    float m = a.sinks ? a.sinks[h] * kLog2e : -INFINITY;
    const float sink = m;
#pragma unroll
    for (int k = 0; k < kMaxCluster; ++k) {
      s[k] = k < ns ? (ns > 1 ? *cl.map_shared_rank(ml + h, k) : ml[h]) : make_float2(-INFINITY, 0.f);
      m = fmaxf(m, s[k].x);
    }
    float den = a.sinks ? fast_exp2(sink - m) : 0.f;
#pragma unroll
    for (int k = 0; k < kMaxCluster; ++k) den += s[k].y > 0.f ? s[k].y * fast_exp2(s[k].x - m) : 0.f;
    ml[H + h] = make_float2(m, 1.0f / den);
  }
  __syncthreads();
  for (int h = warp; h < H; h += kWarps) {
    const float2 f = ml[H + h];
    for (int i = lane; i < n_keys; i += 32) S[h * L.pitch_s + i] = fast_exp2(S[h * L.pitch_s + i] - f.x) * f.y;
  }
  __syncthreads();
  // ---- weights mixed over the heads: thread (key, eight heads) ----
  {
    const int h8 = (H + 7) / 8;
    for (int i = tid; i < n_keys * h8; i += kThreads) {
      const int j = i % n_keys, h0 = i / n_keys * 8;
      float w[8];
#pragma unroll
      for (int x = 0; x < 8; ++x) w[x] = 0.f;
      if (a.mix) {
#pragma unroll 4
        for (int k = 0; k < H; ++k) {
          const float p = S[k * L.pitch_s + j];
#pragma unroll
          for (int x = 0; x < 8; x += 4) {
            const float4 f = *reinterpret_cast<const float4*>(mixer + k * L.pitch_m + h0 + x);
            w[x] = fmaf(f.x, p, w[x]);
            w[x + 1] = fmaf(f.y, p, w[x + 1]);
            w[x + 2] = fmaf(f.z, p, w[x + 2]);
            w[x + 3] = fmaf(f.w, p, w[x + 3]);
          }
        }
      } else {
#pragma unroll
        for (int x = 0; x < 8; ++x) w[x] = S[min(h0 + x, H - 1) * L.pitch_s + j];
      }
#pragma unroll
      for (int x = 0; x < 8; ++x)
        if (h0 + x < H) {
          const __nv_bfloat16 hi = __float2bfloat16_rn(w[x]);
          w_hi[(h0 + x) * L.pitch_w + j] = hi;
          w_lo[(h0 + x) * L.pitch_w + j] = __float2bfloat16_rn(w[x] - __bfloat162float(hi));
        }
    }
  }
  __syncthreads();
  // ---- values: columns of V are the row operand (two keys of a column in one register), heads the columns ----
  constexpr int NM = DP / 16, SLABS = DP / 64;                // (a row of 64: the second half of a tile is columns 4 further on)
  float* O = S;                                               // [sub][H][DP], the scores' place
  for (int task = set; task < tasks; task += n_sets) {
      const int gv = task / tiles, h0 = task % tiles * 8;
      float acc[NM][4];
#pragma unroll
      for (int m = 0; m < NM; ++m)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[m][x] = 0.f;
      const int hr = gv * Gq + min(h0 + g, Gq - 1);           // (columns without a head are not stored)
      const __nv_bfloat16 *wh = w_hi + (size_t)hr * L.pitch_w, *wl = w_lo + (size_t)hr * L.pitch_w;
      uint4 next[4][SLABS];                                   // the next group's keys 2 tq, + 1, + 8, + 9
      auto ask = [&](int gi) {
        const bool blk = gi < b_groups;
        const __nv_bfloat16* base = (blk ? bk.v : kv.v) + (size_t)gv * (blk ? bk.page_tokens : kv.page_tokens) * DP + 8 * g;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const uint4* r = reinterpret_cast<const uint4*>(base + (size_t)rows[(gi - ga) * 16 + 2 * tq + (x & 1) + (x >> 1) * 8] * DP);
#pragma unroll
          for (int s = 0; s < SLABS; ++s) next[x][s] = __ldg(r + 8 * s);
        }
      };
      if (ga + sub < gz) ask(ga + sub);
      for (int gi = ga + sub; gi < gz; gi += wpg) {
        const int i0 = (gi - ga) * 16;
        uint4 v[4][SLABS];
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
          for (int s = 0; s < SLABS; ++s) v[x][s] = next[x][s];
        if (gi + wpg < gz) ask(gi + wpg);
        const uint32_t bh0 = *reinterpret_cast<const uint32_t*>(wh + i0 + 2 * tq), bh1 = *reinterpret_cast<const uint32_t*>(wh + i0 + 2 * tq + 8);
        const uint32_t bl0 = *reinterpret_cast<const uint32_t*>(wl + i0 + 2 * tq), bl1 = *reinterpret_cast<const uint32_t*>(wl + i0 + 2 * tq + 8);
        auto word = [](const uint4& u, int k) { return k == 0 ? u.x : k == 1 ? u.y : k == 2 ? u.z : u.w; };
#pragma unroll
        for (int m = 0; m < NM; ++m) {
          // rows g: column 8 g + m (of slab 0); rows g + 8: the same of slab 1, or column 8 g + m + 4
          constexpr bool two = SLABS == 2;
          const int e0 = m, e1 = two ? m : m + 4, s1 = two ? 1 : 0;
          const uint32_t sel0 = e0 & 1 ? 0x7632 : 0x5410, sel1 = e1 & 1 ? 0x7632 : 0x5410;
          const uint32_t a0 = __byte_perm(word(v[0][0], e0 >> 1), word(v[1][0], e0 >> 1), sel0);
          const uint32_t a1 = __byte_perm(word(v[0][s1], e1 >> 1), word(v[1][s1], e1 >> 1), sel1);
          const uint32_t a2 = __byte_perm(word(v[2][0], e0 >> 1), word(v[3][0], e0 >> 1), sel0);
          const uint32_t a3 = __byte_perm(word(v[2][s1], e1 >> 1), word(v[3][s1], e1 >> 1), sel1);
          mma16816(acc[m], a0, a1, a2, a3, bh0, bh1);
          mma16816(acc[m], a0, a1, a2, a3, bl0, bl1);
        }
      }
#pragma unroll
      for (int m = 0; m < NM; ++m)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int h = h0 + 2 * tq + (x & 1), col = 8 * g + (SLABS == 2 ? m + (x >> 1) * 64 : m + (x >> 1) * 4);
          if (h < Gq) O[((size_t)sub * H + gv * Gq + h) * DP + col] = acc[m][x];
        }
    }
  if (ns > 1) cl.sync();
  else __syncthreads();
  // ---- the shares' outputs, every block a part of them ----
  const int vd = a.vdim, sets = wpg;
  const int quads = (vd + 3) / 4;
  for (int i = share * kThreads + tid; i < H * quads; i += ns * kThreads) {
    const int h = i / quads, c = (i - h * quads) * 4;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < sets; ++s) {
      float4 v[kMaxCluster];
#pragma unroll
      for (int k = 0; k < kMaxCluster; ++k) {
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (k < ns) v[k] = *reinterpret_cast<const float4*>((ns > 1 ? cl.map_shared_rank(O, k) : O) + ((size_t)s * H + h) * DP + c);
      }
#pragma unroll
      for (int k = 0; k < kMaxCluster; ++k) y.x += v[k].x, y.y += v[k].y, y.z += v[k].z, y.w += v[k].w;
    }
    const float o[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      if (c + x >= vd) break;
      float z = o[x];
      if (a.gate) z *= sigmoid_t<__nv_bfloat16>(__bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[(size_t)t * a.gate_stride + h * vd + c + x]));
      static_cast<__nv_bfloat16*>(a.out)[(size_t)t * a.out_stride + h * vd + c + x] = __float2bfloat16_rn(z);
    }
  }
  if (ns > 1) cl.sync();                                      // nobody leaves while its shared memory is read
}

int sm_count() {
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  return n;
}

template <int DP>
int launch_step(const KVView& kv, const KVView& bk, const pace_step_t& st, const pace_attn_pooled_args_t& a, cudaStream_t s) {
  const int H = a.n_q_heads, G = kv.n_kv_heads, T = a.token_end - a.token_begin;
  if (T > 65535) return PACE_ERR_UNSUPPORTED;
  const int64_t window = a.window < a.max_keys ? a.window : a.max_keys;
  const int64_t groups = (window + 15) / 16 + 1 + (a.block > 0 && a.max_keys > a.window ? ((a.max_keys - a.window) / a.block + 15) / 16 + 1 : 0);
  const int o_sets = step_sets(G * ((H / G + 7) / 8));
  // the most blocks per token that are all resident at once and have two groups of keys each; more if a share has no room
  int ns = 1;
  while (ns < kMaxCluster && (int64_t)T * ns * 2 <= sm_count() && groups >= 4 * ns) ns *= 2;
  int smem = 0, cap = 0;
  for (;; ns *= 2) {
    if (ns > kMaxCluster) return PACE_ERR_UNSUPPORTED;
    const int64_t share = (groups + ns - 1) / ns * 16;
    if (share > 65536) continue;
    cap = (int)share;
    const StepSmem L = step_smem(H, cap, DP, o_sets);
    smem = L.total;
    if (smem > 0 && smem <= 226 * 1024) break;
  }
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_pooled_step_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)T, 1);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = (size_t)smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)ns;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  PACE_CUDA_TRY(cudaLaunchKernelEx(&cfg, attn_pooled_step_kernel<DP>, kv, bk, st, a, cap, o_sets));
  PACE_LAUNCH_CHECK("attn_pooled_step_kernel");
  return PACE_OK;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_attn_pooled(const pace_kv_pool_t* p, int32_t layer, const pace_kv_pool_t* bp, int32_t block_layer, const pace_step_t* st,
                     const pace_attn_pooled_args_t* a, void* stream) {
  if (!pooled_args_ok(p, layer, bp, block_layer, st, a) || a->token_begin < 0 || a->token_end > st->n_tokens) return PACE_ERR_INVALID;
  const int row = a->q_elems;
  if (a->token_begin >= a->token_end) return PACE_OK;
  PACE_PROFILE("attn_pooled", stream, "layer=%d tokens=%d heads=%d dims=%d/%d", layer, a->token_end - a->token_begin, a->n_q_heads, a->dim, a->vdim);
  const cudaStream_t s = (cudaStream_t)stream;
  const KVView kv = make_view(p, layer, nullptr), bk = a->block > 0 ? make_view(bp, block_layer, nullptr) : kv;
  if (p->row_format == PACE_ROWS_BF16 && aligned16(a->q)) {
    const int rc = row == 64 ? launch_step<64>(kv, bk, *st, *a, s) : launch_step<128>(kv, bk, *st, *a, s);
    if (rc != PACE_ERR_UNSUPPORTED) return rc;
  }
  return a->dtype == PACE_DTYPE_BF16 ? launch_general<__nv_bfloat16>(kv, bk, *st, *a, s) : launch_general<float>(kv, bk, *st, *a, s);
}

}  // extern "C"
