// Prompt attention over a window of tokens and pooled blocks, weights mixed over the heads, on tcgen05.
//
// Mixing commutes with the sum over the keys: with w_g(j) the finished weights of query head g and v_c(j) the values of KV head c,
//     out_h = sum_j (sum_g mix[h][g] w_g(j)) v_c(j) = sum_g mix[h][g] O[g][c],     O[g][c] = sum_j w_g(j) v_c(j),     c head h's own.
// So a tile of query rows reads the values of several KV heads with one set of scores, and what is mixed is O, behind the
// division by the denominators: 32 / group tokens x group heads of one KV head per warp of rows, the heads of a token in neighbouring
// lanes.  A unit is (entry, tile of tokens, up to three or six KV heads of values); it walks over the KV heads of the keys one after
// the other and adds up their shares of its outputs in fp32 (its own part of a workspace: nobody else touches it); the last one
// multiplies by the gate and stores.
//
// Warps 0-15 softmax (a row of a chunk is four threads' work, a warp per 16 columns of 32 rows), 16 producer (queries, keys, values by
// TMA), 17 issues the products.  Chunks of 64 keys: pages of pooled blocks first, then pages of tokens.  Tensor memory: two slots of 64 columns, scores and then, in their place, the weights in two
// bf16 terms; behind them O.
#include <algorithm>

#include "pooled.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64, kBlockBytes = kChunk * 128, kMaxStages = 6;
constexpr int kGroups = 4, kCols = kChunk / kGroups, kSoftmax = 128 * kGroups, kThreads = kSoftmax + 64;   // softmax: warpgroups, their columns
constexpr uint32_t kColO = 128, kColsO = 512 - kColO;
constexpr float kLazy = 8.0f;  // log2 units a row's maximum may grow before O is rescaled

struct PooledParams {
  KVView kv, bk;
  pace_step_t st;
  const __nv_bfloat16* gate;
  __nv_bfloat16* out;
  float* acc;               // [tokens][H][vdim], of the entries' tokens
  const float* sinks;
  const float* mix;
  int64_t out_stride, gate_stride;
  int H, G, Gq, vdim, window, block;
  int entry0, n_entries, n_tiles, tpw, nv, n_sub, n_stages, smem_bytes;
  float scale_log2;
};

struct Unit {
  int t0, start, count, slot;
  int tok0;                // first token of the tile, counted in the entry
  int c0, nv;              // KV heads of the values
  int g0, g1;              // KV heads of the keys
  int tbase;               // position of the first key of the first token chunk
  int nb_chunks, n;        // chunks of blocks, all chunks
};

__device__ __forceinline__ bool get_unit(const PooledParams& p, int u, Unit* w) {
  const int sub = u % p.n_sub, r = u / p.n_sub, e = p.entry0 + r / p.n_tiles, tile = p.n_tiles - 1 - r % p.n_tiles;   // long units first
  w->t0 = p.st.cu[e];
  w->count = p.st.cu[e + 1] - w->t0;
  w->tok0 = tile * 4 * p.tpw;
  if (w->tok0 >= w->count) return false;
  w->start = p.st.start[e];
  w->slot = p.st.slot[e];
  w->c0 = sub * p.nv;
  w->nv = min(p.nv, p.G - w->c0);
  w->g0 = p.mix ? 0 : w->c0;
  w->g1 = p.mix ? p.G : w->c0 + 1;
  const int pos_a = w->start + w->tok0, pos_z = w->start + min(w->count, w->tok0 + 4 * p.tpw) - 1;
  w->nb_chunks = (blocks_seen(pos_z, p.window, p.block) + kChunk - 1) / kChunk;
  w->tbase = window_first(pos_a, p.window) & ~(kChunk - 1);
  w->n = w->nb_chunks + (pos_z - w->tbase) / kChunk + 1;
  return true;
}

struct Bars {
  uint64_t full[kMaxStages], empty[kMaxStages], s_full[2], p_full[2], pv_done[2], q_full, q_empty, o_free, drain;
};

// behind the queries and the ring in shared memory (no static shared memory: the tiles then begin at a multiple of 1024 anyway)
struct Small {
  Bars b;
  float part[kGroups][kUmmaRows];
  uint32_t tmem_slot;
  int abort_flag;
};

// true where any softmax thread says so; a barrier of all of them
__device__ __forceinline__ bool softmax_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, %2, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"((uint32_t)v), "n"(kSoftmax) : "memory");
  return r != 0;
}

// VB: 64-column blocks of a value
template <int VB>
__device__ __forceinline__ void pooled_softmax(const PooledParams& p, Bars& b, uint32_t tmem, float (*part)[kUmmaRows], int n_units,
                                               volatile int* abort) {
  const int row = threadIdx.x & 127, lane = row & 31, warp = row >> 5, grp = threadIdx.x >> 7;
  const uint32_t t_lane = tmem + ((uint32_t)(row & ~31) << 16), tO = t_lane + kColO;
  const int hh = lane % p.Gq, base_lane = lane - hh;
  const bool in_tile = lane < p.tpw * p.Gq;
  const float scale = p.scale_log2;
  const uint64_t scale2 = pack64(__float_as_uint(scale), __float_as_uint(scale));
  int cnt = 0;  // chunks worked on
  bool gave_up = false;   // (a wait that ran out cuts the waits behind it short; nobody leaves the common barriers)
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    const int tok = un.tok0 + warp * p.tpw + lane / p.Gq;
    const bool live = in_tile && tok < un.count;
    const int pos = un.start + (live ? tok : un.count - 1);
    const int nb = blocks_seen(pos, p.window, p.block), first = window_first(pos, p.window);
    for (int gk = un.g0; gk < un.g1; ++gk) {
      float m = p.sinks ? p.sinks[gk * p.Gq + hh] * kLog2e : -INFINITY, l = p.sinks && grp == 0 ? 1.f : 0.f;   // a sink: one more term of the sum
      for (int c = 0; c < un.n; ++c, ++cnt) {
        const uint32_t tS = t_lane + (cnt & 1) * kChunk;
        if (!gave_up) gave_up = !umma_wait(&b.s_full[cnt & 1], (cnt >> 1) & 1, abort);
        tc_fence_after();
        uint32_t sr[kCols];
        tmem_ld16(tS + grp * kCols, sr);
        tmem_wait_ld();
        const bool blk = c < un.nb_chunks;
        const int p0 = (blk ? c * kChunk : un.tbase + (c - un.nb_chunks) * kChunk) + grp * kCols;
        const int lo = blk ? 0 : max(0, first - p0), hi = blk ? min(kCols, nb - p0) : min(kCols, pos + 1 - p0);   // seen keys: [lo, hi)
        if (!__all_sync(0xffffffffu, !live || (lo <= 0 && hi >= kCols))) {
          const unsigned seen = hi > lo ? (unsigned)(hi - lo) : 0u;
#pragma unroll
          for (int k = 0; k < kCols; ++k)
            if ((unsigned)(k - lo) >= seen) sr[k] = 0xff800000u;  // -inf
        }
        float mx = max3(__uint_as_float(sr[0]), __uint_as_float(sr[1]), __uint_as_float(sr[2]));
        float my = max3(__uint_as_float(sr[3]), __uint_as_float(sr[4]), __uint_as_float(sr[5]));
#pragma unroll
        for (int k = 6; k < kCols - 2; k += 4) {
          mx = max3(mx, __uint_as_float(sr[k]), __uint_as_float(sr[k + 1]));
          my = max3(my, __uint_as_float(sr[k + 2]), __uint_as_float(sr[k + 3]));
        }
        mx = max3(fmaxf(mx, my), __uint_as_float(sr[kCols - 2]), __uint_as_float(sr[kCols - 1])) * scale;  // scale > 0
        // behind this barrier all scores are in registers: weights may take their places
        if (softmax_any(live && mx > m + kLazy)) {
          part[grp][row] = mx;
          asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory");
#pragma unroll
          for (int k = 0; k < kGroups; ++k) mx = fmaxf(mx, part[k][row]);
          const bool grow = mx > m + kLazy;
          const float m_new = grow ? mx : m;
          const float alpha = grow ? ((m == -INFINITY) ? 0.f : fast_exp2(m - m_new)) : 1.f;
          if (c > 0) {  // O holds the sum of the earlier chunks
            if (!gave_up) gave_up = !umma_wait(&b.pv_done[(cnt - 1) & 1], ((cnt - 1) >> 1) & 1, abort);
            tc_fence_after();
            for (int d0 = grp * 16; d0 < un.nv * VB * 64; d0 += kGroups * 16) {
              uint32_t ov[16];
              tmem_ld16(tO + d0, ov);
              tmem_wait_ld();
#pragma unroll
              for (int k = 0; k < 16; ++k) ov[k] = __float_as_uint(__uint_as_float(ov[k]) * alpha);
              tmem_st16(tO + d0, ov);
            }
            tmem_wait_st();
          }
          l *= alpha;
          m = m_new;
          asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory");   // the maxima have been read
        }
        const float ne = (m == -INFINITY) ? 0.f : -m;
        const uint64_t ne2 = pack64(__float_as_uint(ne), __float_as_uint(ne));
        uint64_t l2[2] = {0ull, 0ull};
        uint32_t ph[kCols / 2], pl[kCols / 2];
#pragma unroll
        for (int k = 0; k < kCols / 2; ++k) {
          uint32_t x0, x1;
          unpack64(fma2(pack64(sr[2 * k], sr[2 * k + 1]), scale2, ne2), x0, x1);
          const float p0f = fast_exp2(__uint_as_float(x0)), p1f = fast_exp2(__uint_as_float(x1));
          l2[k & 1] = add2(l2[k & 1], pack64(__float_as_uint(p0f), __float_as_uint(p1f)));
          split_bf2(p0f, p1f, ph[k], pl[k]);
        }
        tmem_st8(tS + grp * (kCols / 2), ph);
        tmem_st8(tS + 32 + grp * (kCols / 2), pl);
        {
          uint32_t a0, a1, b0, b1;
          unpack64(l2[0], a0, a1);
          unpack64(l2[1], b0, b1);
          l += (__uint_as_float(a0) + __uint_as_float(a1)) + (__uint_as_float(b0) + __uint_as_float(b1));
        }
        tmem_wait_st();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&b.p_full[cnt & 1]);
      }
      // ---- this KV head's share of the unit's outputs ----
      part[grp][row] = l;
      asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory");
      l = (part[0][row] + part[1][row]) + (part[2][row] + part[3][row]);
      if (!gave_up) gave_up = !umma_wait(&b.pv_done[(cnt - 1) & 1], ((cnt - 1) >> 1) & 1, abort);
      tc_fence_after();
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      const bool opens = gk == un.g0, closes = gk + 1 == un.g1;
      const size_t t = (size_t)(un.t0 + tok), row0 = (size_t)(un.t0 - p.st.cu[p.entry0] + tok) * p.H;
      const int pieces = (p.vdim + 15) / 16;
      for (int i = grp; i < un.nv * pieces; i += kGroups) {
        const int j = i / pieces, d0 = (i - j * pieces) * 16, h = (un.c0 + j) * p.Gq + hh;
        const float* mix = p.mix ? p.mix + (size_t)h * p.H + gk * p.Gq : nullptr;
        float* acc = p.acc + (row0 + h) * p.vdim;
        uint32_t raw[16];
        tmem_ld16(tO + j * VB * 64 + d0, raw);
        float before[16];
#pragma unroll
        for (int k = 0; k < 16; k += 4) {
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (!opens && live && d0 + k < p.vdim) v = __ldcg(reinterpret_cast<const float4*>(acc + d0 + k));
          before[k] = v.x, before[k + 1] = v.y, before[k + 2] = v.z, before[k + 3] = v.w;
        }
        __syncwarp();
        tmem_wait_ld();
        float o[16], y[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) o[k] = __uint_as_float(raw[k]) * inv;
        if (mix) {
          const float f0 = mix[hh];
#pragma unroll
          for (int k = 0; k < 16; ++k) y[k] = fmaf(f0, o[k], before[k]);
          for (int r = 1; r < p.Gq; ++r) {
            const int g = hh + r < p.Gq ? hh + r : hh + r - p.Gq;
            const float f = mix[g];
            const int src = min(base_lane + g, 31);              // (lanes behind the tile's tokens: any lane)
#pragma unroll
            for (int k = 0; k < 16; ++k) y[k] = fmaf(f, __shfl_sync(0xffffffffu, o[k], src), y[k]);
          }
        } else {
#pragma unroll
          for (int k = 0; k < 16; ++k) y[k] = o[k] + before[k];
        }
        if (live) {
#pragma unroll
          for (int k = 0; k < 16; k += 8) {
            if (d0 + k < p.vdim) {
              if (!closes) {
                __stcg(reinterpret_cast<float4*>(acc + d0 + k), make_float4(y[k], y[k + 1], y[k + 2], y[k + 3]));
                __stcg(reinterpret_cast<float4*>(acc + d0 + k + 4), make_float4(y[k + 4], y[k + 5], y[k + 6], y[k + 7]));
              } else {
                if (p.gate) {
                  float g[8];
                  Vec<__nv_bfloat16, 8>::load(p.gate + t * p.gate_stride + (size_t)h * p.vdim + d0 + k, g);
#pragma unroll
                  for (int x = 0; x < 8; ++x) y[k + x] *= sigmoid_t<__nv_bfloat16>(g[x]);
                }
                Vec<__nv_bfloat16, 8>::store(p.out + t * p.out_stride + (size_t)h * p.vdim + d0 + k, y + k);
              }
            }
          }
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&b.o_free);
    }
  }
}

template <int KB, int VB>
__device__ __forceinline__ void pooled_issue(const PooledParams& p, Bars& b, uint32_t tmem, unsigned char* qs, unsigned char* ring,
                                             int stage_bytes, int n_units, volatile int* abort) {
  constexpr uint32_t IDESC_S = umma_idesc(kChunk, false), IDESC_O = umma_idesc(VB * 64, true);
  constexpr int QB = kUmmaRows * 128;
  const bool leader = elect_one();
  const uint32_t q_lo = (smem_u32(qs) >> 4) | (1u << 16);
  int s = 0, ph = 0;          // stage of the next scores
  int sv = 0;                 // stage of the next values
  int cnt = 0, parts = 0;     // chunks and KV heads of keys so far
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    for (int gk = un.g0; gk < un.g1; ++gk, ++parts) {
      if (!umma_issuer_wait(&b.q_full, parts & 1, abort)) return;
      auto scores = [&](int c, int k) {      // chunk c of this KV head, k-th of all
        if (!umma_issuer_wait(&b.full[s], ph, abort)) return false;
        // the slot's weights (two chunks ago) have been read
        if (k >= 2 && !umma_issuer_wait(&b.pv_done[k & 1], ((k - 2) >> 1) & 1, abort)) return false;
        tc_fence_after();
        if (leader) {
          const uint32_t k_lo = (smem_u32(ring + (size_t)s * stage_bytes) >> 4) | (1u << 16);
#pragma unroll
          for (int kb = 0; kb < KB; ++kb)
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              umma_bf16(tmem + (k & 1) * kChunk, pack64(q_lo + kb * (QB >> 4) + kk * 2, kDescHi),
                        pack64(k_lo + kb * (kBlockBytes >> 4) + kk * 2, kDescHi), IDESC_S, kb | kk ? 1u : 0u);
          umma_commit(&b.s_full[k & 1]);
          if (c + 1 == un.n) umma_commit(&b.q_empty);
        }
        __syncwarp();
        if (++s == p.n_stages) s = 0, ph ^= 1;
        return true;
      };
      if (!scores(0, cnt)) return;
      for (int c = 0; c < un.n; ++c, ++cnt) {
        if (c + 1 < un.n && !scores(c + 1, cnt + 1)) return;
        if (!umma_issuer_wait(&b.p_full[cnt & 1], (cnt >> 1) & 1, abort)) return;
        if (c == 0 && parts > 0 && !umma_issuer_wait(&b.o_free, (parts - 1) & 1, abort)) return;   // O has been taken up
        tc_fence_after();
        if (leader) {
          const uint32_t tP = tmem + (cnt & 1) * kChunk;
          for (int j = 0; j < un.nv; ++j) {
            // MN-major: the next 64 columns lie one block further on
            const uint32_t v_lo = (smem_u32(ring + (size_t)sv * stage_bytes + (KB + j * VB) * kBlockBytes) >> 4) |
                                  ((uint32_t)(kBlockBytes >> 4) << 16);
            const uint32_t tO = tmem + kColO + j * VB * 64;
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_bf16_ts(tO, tP + k * 8, pack64(v_lo + k * (2048 >> 4), kDescHi), IDESC_O, k || c > 0 ? 1u : 0u);
#pragma unroll
            for (int k = 0; k < 4; ++k) umma_bf16_ts(tO, tP + 32 + k * 8, pack64(v_lo + k * (2048 >> 4), kDescHi), IDESC_O, 1u);
          }
          umma_commit(&b.empty[sv]);
          umma_commit(&b.pv_done[cnt & 1]);
        }
        __syncwarp();
        if (++sv == p.n_stages) sv = 0;
      }
    }
  }
}

template <int KB, int VB>
__global__ void __launch_bounds__(kThreads, 1)
    attn_pooled_prompt_kernel(const PooledParams p, const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                              const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmBK,
                              const __grid_constant__ CUtensorMap tmBV) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  unsigned char* qs = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  unsigned char* ring = qs + KB * kUmmaRows * 128;
  Small* sm = reinterpret_cast<Small*>(ring + (size_t)p.n_stages * (KB + p.nv * VB) * kBlockBytes);
  Bars& b = sm->b;
  volatile int* abort = &sm->abort_flag;
  if (reinterpret_cast<unsigned char*>(sm + 1) > smem_raw + p.smem_bytes) {     // (the tiles do not begin where they should)
    if (threadIdx.x == 0) raise_status(p.kv.status, PACE_DEV_BAD_INDEX);
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_units = p.n_entries * p.n_tiles * p.n_sub, stage_bytes = (KB + p.nv * VB) * kBlockBytes;
  if (warp == kSoftmax / 32 + 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_slot)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (tid == 0) {
    sm->abort_flag = 0;
    for (int i = 0; i < p.n_stages; ++i) {
      mbar_init(&b.full[i], 1);
      mbar_init(&b.empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&b.s_full[i], 1);
      mbar_init(&b.p_full[i], kSoftmax / 32);
      mbar_init(&b.pv_done[i], 1);
    }
    mbar_init(&b.q_full, 1);
    mbar_init(&b.q_empty, 1);
    mbar_init(&b.o_free, kSoftmax / 32);
    mbar_init(&b.drain, 1);
    fence_mbar_init();
  }
  // query rows that no copy brings (behind a warp's last whole token) are numbers
  for (int i = tid; i < KB * kUmmaRows * 8; i += kThreads) reinterpret_cast<uint4*>(qs)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&sm->tmem_slot);

  if (warp < kSoftmax / 32) {
    pooled_softmax<VB>(p, b, tmem, sm->part, n_units, abort);
  } else if (warp == kSoftmax / 32) {
    int s = 0, ph = 0, issued = 0, parts = 0;
    bool ok = true;
    for (int u = blockIdx.x; u < n_units && ok; u += gridDim.x) {
      Unit un;
      if (!get_unit(p, u, &un)) continue;
      const int blocks = KB + un.nv * VB;
      for (int gk = un.g0; gk < un.g1 && ok; ++gk, ++parts) {
        if (parts > 0 && !__all_sync(0xffffffffu, mbar_wait(&b.q_empty, (parts - 1) & 1, abort))) {
          ok = false;
          break;
        }
        if (lane == 0) mbar_arrive_expect_tx(&b.q_full, 4 * KB * p.tpw * p.Gq * 128);
        __syncwarp();
        if (lane < 4 * KB) {
          const int w = lane & 3, kb = lane >> 2;
          tma_load_3d(qs + kb * (kUmmaRows * 128) + w * 4096, &tmQ, kb * 64, gk * p.Gq, un.t0 + un.tok0 + w * p.tpw, &b.q_full);
        }
        int page = 0;
        for (int c = 0; c < un.n; ++c) {
          if ((c & 31) == 0) {  // the next 32 chunks' pages, one per lane
            page = 0;
            const int k = c + lane;
            if (k < un.n) {
              const bool blk = k < un.nb_chunks;
              const KVView& v = blk ? p.bk : p.kv;
              page = un.slot >= 0 && un.slot < v.max_seqs ? view_page(v, un.slot, blk ? k : un.tbase / kChunk + k - un.nb_chunks) : -1;
              if (page < 0) {
                raise_status(v.status, PACE_DEV_BAD_INDEX);
                page = 0;
              }
            }
          }
          if (issued >= p.n_stages && !__all_sync(0xffffffffu, mbar_wait(&b.empty[s], ph ^ 1, abort))) {
            ok = false;
            break;
          }
          unsigned char* st = ring + (size_t)s * stage_bytes;
          if (lane == 0) mbar_arrive_expect_tx(&b.full[s], blocks * kBlockBytes);
          __syncwarp();
          const int pg = __shfl_sync(0xffffffffu, page, c & 31);
          const bool blk = c < un.nb_chunks;
          if (lane < KB) {
            tma_load_3d(st + lane * kBlockBytes, blk ? &tmBK : &tmK, lane * 64, 0, pg * p.G + gk, &b.full[s]);
          } else if (lane < blocks) {
            const int j = (lane - KB) / VB, vb = (lane - KB) % VB;
            tma_load_3d(st + lane * kBlockBytes, blk ? &tmBV : &tmV, vb * 64, 0, pg * p.G + un.c0 + j, &b.full[s]);
          }
          ++issued;
          if (++s == p.n_stages) s = 0, ph ^= 1;
        }
      }
    }
    if (!ok) {  // copies in flight land before the block's shared memory is released
      for (int k = issued > p.n_stages ? issued - p.n_stages : 0; k < issued; ++k) mbar_wait(&b.full[k % p.n_stages], (k / p.n_stages) & 1);
      if (parts > 0) mbar_wait(&b.q_full, (parts - 1) & 1);
    }
  } else {
    pooled_issue<KB, VB>(p, b, tmem, qs, ring, stage_bytes, n_units, abort);
    // nothing may still be writing tensor memory when it is handed back
    if (elect_one()) {
      umma_commit(&b.drain);
      for (int k = 0; k < (1 << 20) && !mbar_try_wait(&b.drain, 0); ++k) __nanosleep(64);
    }
    __syncwarp();
  }
  if (lane == 0 && *abort) raise_status(p.kv.status, PACE_DEV_WAIT_TIMEOUT);
  tc_fence_before();
  __syncthreads();
  if (warp == kSoftmax / 32 + 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
  }
}

int sm_count() {
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  return n;
}

template <int KB, int VB>
int launch_prompt(PooledParams& p, const CUtensorMap* tm, cudaStream_t s) {
  const int q_bytes = KB * kUmmaRows * 128, stage = (KB + p.nv * VB) * kBlockBytes, most = 227 * 1024, room = most - (int)sizeof(Small) - q_bytes;
  p.n_stages = std::min(kMaxStages, room / stage);
  if (p.n_stages < 2) return PACE_ERR_UNSUPPORTED;
  const int smem = std::min(most, q_bytes + p.n_stages * stage + (int)sizeof(Small) + 1024);
  p.smem_bytes = smem;
  const int units = p.n_entries * p.n_tiles * p.n_sub, blocks = std::min(units, sm_count());
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_pooled_prompt_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  attn_pooled_prompt_kernel<KB, VB><<<blocks, kThreads, smem, s>>>(p, tm[0], tm[1], tm[2], tm[3], tm[4]);
  PACE_LAUNCH_CHECK("attn_pooled_prompt_kernel");
  return PACE_OK;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" uint64_t pace_attn_pooled_prompt_workspace_bytes(int32_t n_tokens, int32_t n_q_heads, int32_t vdim) {
  if (n_tokens <= 0 || n_q_heads <= 0 || vdim <= 0) return 0;
  return (uint64_t)n_tokens * n_q_heads * vdim * sizeof(float);
}

extern "C" int pace_attn_pooled_prompt(const pace_kv_pool_t* pl, int32_t layer, const pace_kv_pool_t* bp, int32_t block_layer,
                                       const pace_step_t* st, const pace_attn_pooled_args_t* a, void* stream) {
  if (!pooled_args_ok(pl, layer, bp, block_layer, st, a) || a->entry_begin < 0 || a->entry_end < a->entry_begin ||
      a->entry_end > st->n_entries || a->max_tokens < 0)
    return PACE_ERR_INVALID;
  if (a->entry_begin == a->entry_end || a->max_tokens == 0) return PACE_OK;
  PooledParams p;
  p.H = a->n_q_heads;
  p.G = pl->n_kv_heads;
  p.Gq = p.H / p.G;
  if (a->dtype != PACE_DTYPE_BF16 || pl->row_format != PACE_ROWS_BF16 || pl->page_tokens != kChunk || (a->block > 0 && page_rows(*bp) != kChunk) ||
      !(a->scale > 0.f) || p.Gq > 32 || a->vdim % 8 || a->out_stride % 8 || (a->gate && a->gate_stride % 8) || !aligned16(a->q) ||
      !aligned16(a->out) || !aligned16(a->gate))
    return PACE_ERR_UNSUPPORTED;
  const int KB = (a->dim + 63) / 64, VB = (a->vdim + 63) / 64;
  p.kv = make_view(pl, layer, nullptr);
  p.bk = a->block > 0 ? make_view(bp, block_layer, nullptr) : p.kv;
  p.st = *st;
  p.gate = static_cast<const __nv_bfloat16*>(a->gate);
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.acc = static_cast<float*>(a->workspace);
  p.sinks = a->sinks;
  p.mix = a->mix;
  p.out_stride = a->out_stride;
  p.gate_stride = a->gate_stride;
  p.vdim = a->vdim;
  p.window = a->window;
  p.block = a->block;
  p.entry0 = a->entry_begin;
  p.n_entries = a->entry_end - a->entry_begin;
  p.tpw = 32 / p.Gq;
  p.n_tiles = (a->max_tokens + 4 * p.tpw - 1) / (4 * p.tpw);
  const int most = a->mix ? (int)kColsO / (VB * 64) : 1;      // KV heads of values that O has room for
  p.n_sub = (p.G + most - 1) / most;
  p.nv = (p.G + p.n_sub - 1) / p.n_sub;
  p.n_sub = (p.G + p.nv - 1) / p.nv;
  p.scale_log2 = a->scale * kLog2e;
  if ((int64_t)p.n_entries * p.n_tiles * p.n_sub > 0x7fffffff) return PACE_ERR_UNSUPPORTED;
  if (p.mix && p.G > 1 && (!a->workspace || !aligned16(a->workspace) ||
                           a->workspace_bytes < pace_attn_pooled_prompt_workspace_bytes(st->n_tokens, p.H, p.vdim)))
    return PACE_ERR_INVALID;
  CUtensorMap tm[5];
  const uint64_t row = (uint64_t)pl->head_dim;
  const uint64_t dq[3] = {row, (uint64_t)p.H, (uint64_t)st->n_tokens}, sq[2] = {row * 2, row * 2 * p.H};
  const uint32_t bq[3] = {64, (uint32_t)p.Gq, (uint32_t)p.tpw}, box[3] = {64, kChunk, 1};
  int rc = tensor_map_bf16(&tm[0], a->q, 3, dq, sq, bq);
  for (int i = 0; i < 2 && rc == PACE_OK; ++i) {
    const KVView& v = i ? p.bk : p.kv;
    const uint64_t dims[3] = {row, kChunk, (uint64_t)v.n_pages * p.G}, str[2] = {row * 2, row * 2 * kChunk};
    rc = tensor_map_bf16(&tm[1 + 2 * i], v.k, 3, dims, str, box);
    if (rc == PACE_OK) rc = tensor_map_bf16(&tm[2 + 2 * i], v.v, 3, dims, str, box);
  }
  if (rc != PACE_OK) return rc;
  PACE_PROFILE("attn_pooled_prompt", stream, "layer=%d entries=%d tokens<=%d heads=%d dims=%d/%d", layer, p.n_entries, a->max_tokens, p.H,
               a->dim, a->vdim);
  const cudaStream_t s = (cudaStream_t)stream;
#define PACE_POOLED_CASE(kb, vb) \
  if (KB == kb && VB == vb) return launch_prompt<kb, vb>(p, tm, s);
  PACE_POOLED_CASE(1, 1) PACE_POOLED_CASE(2, 1) PACE_POOLED_CASE(1, 2) PACE_POOLED_CASE(2, 2)
#undef PACE_POOLED_CASE
  return PACE_ERR_UNSUPPORTED;
}
