// Prompt attention over a window of tokens and pooled blocks, weights mixed over the heads, on tcgen05.
//
// Mixing commutes with the sum over the keys: with w_g(j) the finished weights of query head g and v_c(j) the values of KV head c,
//     out_h = sum_j (sum_g mix[h][g] w_g(j)) v_c(j) = sum_g mix[h][g] O[g][c],     O[g][c] = sum_j w_g(j) v_c(j),     c head h's own.
// So a tile of query rows reads the values of several KV heads with one set of scores, and what is mixed is O, behind the
// division by the denominators: 32 / group tokens x group heads of one KV head per warp of rows, the heads of a token in neighbouring
// lanes.  A unit is (entry, tile of tokens, up to two or four KV heads of values); it walks over the KV heads of the keys one after
// the other and adds up their shares of its outputs in fp32 (its own part of a workspace: nobody else touches it); the last one
// multiplies by the gate and stores.
//
// Warps 0-15 softmax (a row of a chunk is four threads' work, a warp per 16 columns of 32 rows), 16 producer (queries, keys, values by
// TMA), 17 and 18 issue the products with the keys and with the values.  Chunks of 64 keys: pages of pooled blocks first, then pages of
// tokens.  Tensor memory: four slots of 64 columns, scores and then, in their place, the weights in two bf16 terms (so scores are made
// ahead, in slots whose weights have long been read); behind them O.
#include <algorithm>

#include "pooled.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64, kBlockBytes = kChunk * 128, kMaxStages = 6, kKeyStages = 3;
constexpr int kGroups = 4, kCols = kChunk / kGroups, kSoftmax = 128 * kGroups, kThreads = kSoftmax + 96;   // softmax: warpgroups, their columns
constexpr int kSlots = 4;
constexpr uint32_t kColO = kSlots * kChunk, kColsO = 512 - kColO;
constexpr float kLazy = 8.0f;  // log2 units a row's maximum may grow before O is rescaled

struct PooledParams {
  KVView kv, bk;
  pace_step_t st;
  const __nv_bfloat16* gate;
  __nv_bfloat16* out;
  float4* acc;              // [units][16-column pieces of the unit's outputs][rounds][4][rows]: a thread's sums lie beside those of its warp
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
  uint64_t k_full[kKeyStages], k_empty[kKeyStages], v_full[kMaxStages], v_empty[kMaxStages];
  uint64_t s_full[kSlots], p_full[kSlots], pv_done[kSlots], q_full, q_empty, o_free, drain[2];
};

// behind the queries and the rings in shared memory (no static shared memory: the tiles then begin at a multiple of 1024 anyway)
constexpr int kMixPitch = 20;     // floats of a row's 16 columns: neighbouring rows in different banks
struct Small {
  Bars b;
  float part[kGroups][kUmmaRows];
  alignas(16) float o[kGroups][kUmmaRows][kMixPitch];   // outputs on their way to the token's other heads
  uint32_t tmem_slot;
  int abort_flag;
  alignas(16) float mix[1];                             // [2][KV heads of values][group][group, padded to 4], of the KV head of the keys
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
__device__ __forceinline__ void pooled_softmax(const PooledParams& p, Bars& b, uint32_t tmem, Small& sm, int n_units,
                                               volatile int* abort) {
  float(*part)[kUmmaRows] = sm.part;
  const int row = threadIdx.x & 127, lane = row & 31, warp = row >> 5, grp = threadIdx.x >> 7;
  const uint32_t t_lane = tmem + ((uint32_t)(row & ~31) << 16), tO = t_lane + kColO;
  const int hh = lane % p.Gq;
  const bool in_tile = lane < p.tpw * p.Gq;
  const float scale = p.scale_log2;
  const uint64_t scale2 = pack64(__float_as_uint(scale), __float_as_uint(scale));
  const int mp = (p.Gq + 3) & ~3, pieces = (p.vdim + 15) / 16, parts4 = mp / 4, items = p.tpw * parts4 * 4, rounds = (items + 31) / 32;
  const int item_h4 = (lane >> 2) % parts4 * 4, item_tok = (lane >> 2) / parts4;
  int slot = 0, phase = 0, parts = 0;    // of the next chunk; KV heads of keys so far
  uint64_t* pv = nullptr;                // what the newest chunk's values complete, and the phase
  int pv_phase = 0;
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
      // (the chunks' barriers lie in front of the first use; who is behind still reads the other half)
      float* mixes = sm.mix + (parts++ & 1) * p.nv * p.Gq * mp;       // [KV head of the values][head of the keys][its heads]
      for (int i = threadIdx.x; i < un.nv * p.Gq * mp; i += kSoftmax) {
        const int h = i % mp, g = i / mp % p.Gq, j = i / (mp * p.Gq);
        mixes[i] = h >= p.Gq ? 0.f : p.mix ? p.mix[(size_t)((un.c0 + j) * p.Gq + h) * p.H + gk * p.Gq + g] : h == g ? 1.f : 0.f;
      }
      if (p.gate && gk + 1 == un.g1) {         // the unit's gates are on their way to L2 while its last scores are worked on
        const int lines = (un.nv * p.Gq * p.vdim * 2 + 127) / 128, toks = min(4 * p.tpw, un.count - un.tok0);
        for (int i = threadIdx.x; i < toks * lines; i += kSoftmax)
          asm volatile("prefetch.global.L2 [%0];" ::"l"(p.gate + (size_t)(un.t0 + un.tok0 + i / lines) * p.gate_stride + un.c0 * p.Gq * p.vdim + i % lines * 64));
      }
      for (int c = 0; c < un.n; ++c) {
        const uint32_t tS = t_lane + slot * kChunk;
        if (!gave_up) gave_up = !umma_issuer_wait(&b.s_full[slot], phase, abort);
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
            if (!gave_up) gave_up = !umma_issuer_wait(pv, pv_phase, abort);
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
        if (lane == 0) mbar_arrive(&b.p_full[slot]);
        pv = &b.pv_done[slot];
        pv_phase = phase;
        if (++slot == kSlots) slot = 0, phase ^= 1;
      }
      // ---- this KV head's share of the unit's outputs ----
      part[grp][row] = l;
      asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory");
      l = (part[0][row] + part[1][row]) + (part[2][row] + part[3][row]);
      const float inv = l > 0.f ? 1.0f / l : 0.f;
      const bool opens = gk == un.g0, closes = gk + 1 == un.g1;
      // a lane mixes four columns of one token for up to four of its heads: item = (token, part of its heads, four columns)
      const int per = rounds * 4 * kUmmaRows;          // a piece's sums
      float4* acc = p.acc + (size_t)u * p.nv * pieces * per + row;
      float4 y[4];                                     // the sums so far of the next item
      auto ask = [&](int at, bool live_piece) {
#pragma unroll
        for (int k = 0; k < 4; ++k) y[k] = opens || !live_piece ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcg(acc + at + k * kUmmaRows);
      };
      ask(grp * per, true);
      if (!gave_up) gave_up = !umma_issuer_wait(pv, pv_phase, abort);
      tc_fence_after();
      float* mine = sm.o[grp][row];
      for (int j = 0; j < un.nv; ++j) {
        const float* mix_j = mixes + j * p.Gq * mp;
        for (int d = grp; d < pieces; d += kGroups) {
          uint32_t raw[16];
          tmem_ld16(tO + j * VB * 64 + d * 16, raw);
          tmem_wait_ld();
#pragma unroll
          for (int q = 0; q < 4; ++q)
            *reinterpret_cast<float4*>(mine + q * 4) = make_float4(__uint_as_float(raw[4 * q]) * inv, __uint_as_float(raw[4 * q + 1]) * inv,
                                                                   __uint_as_float(raw[4 * q + 2]) * inv, __uint_as_float(raw[4 * q + 3]) * inv);
          __syncwarp();
          const int at = (j * pieces + d) * per;
          for (int r = 0; r < rounds; ++r) {
            const int it = r * 32 + lane;
            const int h4 = r == 0 ? item_h4 : (it >> 2) % parts4 * 4, tl = r == 0 ? item_tok : (it >> 2) / parts4;
            const bool there = it < items;
            float4 z[4] = {y[0], y[1], y[2], y[3]};
            if (r + 1 < rounds) ask(at + (r + 1) * 4 * kUmmaRows, true);
            else if (d + kGroups < pieces) ask(at + kGroups * per, true);
            else ask(((j + 1) * pieces + grp) * per, j + 1 < un.nv);
            const float* o = sm.o[grp][(row & ~31) + (there ? tl * p.Gq : 0)] + (lane & 3) * 4;
            const float* f = mix_j + (there ? h4 : 0);
            const int tk = un.tok0 + warp * p.tpw + tl, col = d * 16 + (lane & 3) * 4;
            const bool store = closes && there && tk < un.count && col < p.vdim;
            const size_t t = (size_t)(un.t0 + (store ? tk : 0));
            const int out0 = ((un.c0 + j) * p.Gq + h4) * p.vdim + col;
            uint2 gates[4];                            // asked for ahead of the mixing
            if (p.gate) {
#pragma unroll
              for (int k = 0; k < 4; ++k)
                if (store && h4 + k < p.Gq) gates[k] = *reinterpret_cast<const uint2*>(p.gate + t * p.gate_stride + out0 + k * p.vdim);
            }
#pragma unroll 2
            for (int g = 0; g < p.Gq; ++g, o += kMixPitch, f += mp) {
              const float4 v = *reinterpret_cast<const float4*>(o), w = *reinterpret_cast<const float4*>(f);
              z[0].x = fmaf(w.x, v.x, z[0].x), z[0].y = fmaf(w.x, v.y, z[0].y), z[0].z = fmaf(w.x, v.z, z[0].z), z[0].w = fmaf(w.x, v.w, z[0].w);
              z[1].x = fmaf(w.y, v.x, z[1].x), z[1].y = fmaf(w.y, v.y, z[1].y), z[1].z = fmaf(w.y, v.z, z[1].z), z[1].w = fmaf(w.y, v.w, z[1].w);
              z[2].x = fmaf(w.z, v.x, z[2].x), z[2].y = fmaf(w.z, v.y, z[2].y), z[2].z = fmaf(w.z, v.z, z[2].z), z[2].w = fmaf(w.z, v.w, z[2].w);
              z[3].x = fmaf(w.w, v.x, z[3].x), z[3].y = fmaf(w.w, v.y, z[3].y), z[3].z = fmaf(w.w, v.z, z[3].z), z[3].w = fmaf(w.w, v.w, z[3].w);
            }
            if (!closes) {
#pragma unroll
              for (int k = 0; k < 4; ++k) __stcg(acc + at + (r * 4 + k) * kUmmaRows, z[k]);
            } else if (store) {
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                if (h4 + k >= p.Gq) break;
                float v[4] = {z[k].x, z[k].y, z[k].z, z[k].w};
                if (p.gate) {
                  const float2 g0 = bf2_to_f2(gates[k].x), g1 = bf2_to_f2(gates[k].y);
                  v[0] *= sigmoid_t<__nv_bfloat16>(g0.x);
                  v[1] *= sigmoid_t<__nv_bfloat16>(g0.y);
                  v[2] *= sigmoid_t<__nv_bfloat16>(g1.x);
                  v[3] *= sigmoid_t<__nv_bfloat16>(g1.y);
                }
                Vec<__nv_bfloat16, 4>::store(p.out + t * p.out_stride + out0 + k * p.vdim, v);
              }
            }
            __syncwarp();
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&b.o_free);
    }
  }
}

template <int KB>
__device__ __forceinline__ void pooled_issue_scores(const PooledParams& p, Bars& b, uint32_t tmem, unsigned char* qs, unsigned char* k_ring,
                                                    int n_units, volatile int* abort) {
  constexpr uint32_t IDESC = umma_idesc(kChunk, false);
  constexpr int QB = kUmmaRows * 128;
  const bool leader = elect_one();
  const uint32_t q_lo = (smem_u32(qs) >> 4) | (1u << 16);
  int s = 0, ph = 0, slot = 0, used = 0, phase = 1, parts = 0;   // stage; slot, whether all have been used, phase of its newest weights
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    for (int gk = un.g0; gk < un.g1; ++gk, ++parts) {
      if (!umma_issuer_wait(&b.q_full, parts & 1, abort)) return;
      for (int c = 0; c < un.n; ++c) {
        if (!umma_issuer_wait(&b.k_full[s], ph, abort)) return;
        if (used && !umma_issuer_wait(&b.pv_done[slot], phase, abort)) return;   // the slot's weights have been read
        tc_fence_after();
        if (leader) {
          const uint32_t k_lo = (smem_u32(k_ring + s * KB * kBlockBytes) >> 4) | (1u << 16);
#pragma unroll
          for (int kb = 0; kb < KB; ++kb)
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              umma_bf16(tmem + slot * kChunk, pack64(q_lo + kb * (QB >> 4) + kk * 2, kDescHi),
                        pack64(k_lo + kb * (kBlockBytes >> 4) + kk * 2, kDescHi), IDESC, kb | kk ? 1u : 0u);
          umma_commit(&b.k_empty[s]);
          umma_commit(&b.s_full[slot]);
          if (c + 1 == un.n) umma_commit(&b.q_empty);
        }
        __syncwarp();
        if (++s == kKeyStages) s = 0, ph ^= 1;
        if (++slot == kSlots) slot = 0, used = 1, phase ^= 1;
      }
    }
  }
}

template <int VB>
__device__ __forceinline__ void pooled_issue_values(const PooledParams& p, Bars& b, uint32_t tmem, unsigned char* v_ring, int n_units,
                                                    volatile int* abort) {
  constexpr uint32_t IDESC = umma_idesc(VB * 64, true);
  const bool leader = elect_one();
  const int v_bytes = p.nv * VB * kBlockBytes;
  int s = 0, ph = 0, slot = 0, phase = 0, parts = 0;
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    for (int gk = un.g0; gk < un.g1; ++gk, ++parts)
      for (int c = 0; c < un.n; ++c) {
        if (!umma_issuer_wait(&b.v_full[s], ph, abort)) return;
        if (c == 0 && parts > 0 && !umma_issuer_wait(&b.o_free, (parts - 1) & 1, abort)) return;   // O has been taken up
        if (!umma_issuer_wait(&b.p_full[slot], phase, abort)) return;
        tc_fence_after();
        if (leader) {
          // MN-major: the next 64 columns lie one block further on; an accumulator's products follow one another
          const uint32_t v_lo = (smem_u32(v_ring + (size_t)s * v_bytes) >> 4) | ((uint32_t)(kBlockBytes >> 4) << 16);
          const uint32_t tP = tmem + slot * kChunk;
          for (int j = 0; j < un.nv; ++j)
#pragma unroll
            for (int k = 0; k < 8; ++k)
              umma_bf16_ts(tmem + kColO + j * VB * 64, tP + k * 8, pack64(v_lo + j * (VB * kBlockBytes >> 4) + (k & 3) * (2048 >> 4), kDescHi),
                           IDESC, k || c > 0 ? 1u : 0u);
          umma_commit(&b.v_empty[s]);
          umma_commit(&b.pv_done[slot]);
        }
        __syncwarp();
        if (++s == p.n_stages) s = 0, ph ^= 1;
        if (++slot == kSlots) slot = 0, phase ^= 1;
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
  unsigned char* k_ring = qs + KB * kUmmaRows * 128;
  unsigned char* v_ring = k_ring + kKeyStages * KB * kBlockBytes;
  Small* sm = reinterpret_cast<Small*>(v_ring + (size_t)p.n_stages * p.nv * VB * kBlockBytes);
  Bars& b = sm->b;
  volatile int* abort = &sm->abort_flag;
  if (sm->mix + 2 * p.nv * p.Gq * ((p.Gq + 3) & ~3) > reinterpret_cast<float*>(smem_raw + p.smem_bytes)) {     // (the tiles do not begin where they should)
    if (threadIdx.x == 0) raise_status(p.kv.status, PACE_DEV_BAD_INDEX);
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_units = p.n_entries * p.n_tiles * p.n_sub, v_bytes = p.nv * VB * kBlockBytes;
  if (warp == kSoftmax / 32 + 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm->tmem_slot)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (tid == 0) {
    sm->abort_flag = 0;
    for (int i = 0; i < kKeyStages; ++i) {
      mbar_init(&b.k_full[i], 1);
      mbar_init(&b.k_empty[i], 1);
    }
    for (int i = 0; i < p.n_stages; ++i) {
      mbar_init(&b.v_full[i], 1);
      mbar_init(&b.v_empty[i], 1);
    }
    for (int i = 0; i < kSlots; ++i) {
      mbar_init(&b.s_full[i], 1);
      mbar_init(&b.p_full[i], kSoftmax / 32);
      mbar_init(&b.pv_done[i], 1);
    }
    mbar_init(&b.q_full, 1);
    mbar_init(&b.q_empty, 1);
    mbar_init(&b.o_free, kSoftmax / 32);
    for (int i = 0; i < 2; ++i) mbar_init(&b.drain[i], 1);
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
    pooled_softmax<VB>(p, b, tmem, *sm, n_units, abort);
  } else if (warp == kSoftmax / 32) {
    int s = 0, ph = 0, sv = 0, phv = 0, keys = 0, values = 0, parts = 0;   // stages; chunks asked for
    bool ok = true;
    auto free_stage = [&](uint64_t* bar, int phase) { return __all_sync(0xffffffffu, mbar_wait(bar, phase, abort)); };
    for (int u = blockIdx.x; u < n_units && ok; u += gridDim.x) {
      Unit un;
      if (!get_unit(p, u, &un)) continue;
      for (int gk = un.g0; gk < un.g1 && ok; ++gk, ++parts) {
        if (parts > 0 && !free_stage(&b.q_empty, (parts - 1) & 1)) {
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
          const int pg = __shfl_sync(0xffffffffu, page, c & 31);
          const bool blk = c < un.nb_chunks;
          if (keys >= kKeyStages && !free_stage(&b.k_empty[s], ph ^ 1)) {
            ok = false;
            break;
          }
          if (lane == 0) mbar_arrive_expect_tx(&b.k_full[s], KB * kBlockBytes);
          __syncwarp();
          if (lane < KB) tma_load_3d(k_ring + (s * KB + lane) * kBlockBytes, blk ? &tmBK : &tmK, lane * 64, 0, pg * p.G + gk, &b.k_full[s]);
          ++keys;
          if (++s == kKeyStages) s = 0, ph ^= 1;
          if (values >= p.n_stages && !free_stage(&b.v_empty[sv], phv ^ 1)) {
            ok = false;
            break;
          }
          if (lane == 0) mbar_arrive_expect_tx(&b.v_full[sv], un.nv * VB * kBlockBytes);
          __syncwarp();
          if (lane < un.nv * VB)
            tma_load_3d(v_ring + (size_t)sv * v_bytes + lane * kBlockBytes, blk ? &tmBV : &tmV, lane % VB * 64, 0, pg * p.G + un.c0 + lane / VB,
                        &b.v_full[sv]);
          ++values;
          if (++sv == p.n_stages) sv = 0, phv ^= 1;
        }
      }
    }
    if (!ok) {  // copies in flight land before the block's shared memory is released
      for (int k = keys > kKeyStages ? keys - kKeyStages : 0; k < keys; ++k) mbar_wait(&b.k_full[k % kKeyStages], (k / kKeyStages) & 1);
      for (int k = values > p.n_stages ? values - p.n_stages : 0; k < values; ++k) mbar_wait(&b.v_full[k % p.n_stages], (k / p.n_stages) & 1);
      if (parts > 0) mbar_wait(&b.q_full, (parts - 1) & 1);
    }
  } else {
    const int w = warp - kSoftmax / 32 - 1;
    if (w == 0) pooled_issue_scores<KB>(p, b, tmem, qs, k_ring, n_units, abort);
    else pooled_issue_values<VB>(p, b, tmem, v_ring, n_units, abort);
    // nothing may still be writing tensor memory when it is handed back
    if (elect_one()) {
      umma_commit(&b.drain[w]);
      for (int k = 0; k < (1 << 20) && !mbar_try_wait(&b.drain[w], 0); ++k) __nanosleep(64);
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
  const int fixed = KB * kUmmaRows * 128 + kKeyStages * KB * kBlockBytes + (int)sizeof(Small) + 2 * p.nv * p.Gq * ((p.Gq + 3) & ~3) * (int)sizeof(float);
  const int stage = p.nv * VB * kBlockBytes, most = 227 * 1024;
  p.n_stages = std::min(kMaxStages, (most - fixed) / stage);
  if (p.n_stages < 2) return PACE_ERR_UNSUPPORTED;
  const int smem = std::min(most, fixed + p.n_stages * stage + 1024);
  p.smem_bytes = smem;
  const int units = p.n_entries * p.n_tiles * p.n_sub, blocks = std::min(units, sm_count());
  PACE_CUDA_TRY(cudaFuncSetAttribute(attn_pooled_prompt_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  attn_pooled_prompt_kernel<KB, VB><<<blocks, kThreads, smem, s>>>(p, tm[0], tm[1], tm[2], tm[3], tm[4]);
  PACE_LAUNCH_CHECK("attn_pooled_prompt_kernel");
  return PACE_OK;
}

struct Plan {
  int tpw, n_tiles, nv, n_sub;
  uint64_t bytes;             // of the units' sums
};
Plan plan_units(int n_entries, int max_tokens, int H, int G, int vdim, bool mixed) {
  Plan p;
  p.tpw = 32 / (H / G);
  p.n_tiles = (max_tokens + 4 * p.tpw - 1) / (4 * p.tpw);
  const int most = mixed ? (int)kColsO / ((vdim + 63) / 64 * 64) : 1;      // KV heads of values that O has room for
  p.n_sub = (G + most - 1) / most;
  p.nv = (G + p.n_sub - 1) / p.n_sub;
  p.n_sub = (G + p.nv - 1) / p.nv;
  p.bytes = mixed && G > 1 ? (uint64_t)n_entries * p.n_tiles * p.n_sub * p.nv * ((vdim + 15) / 16) *
                                      ((p.tpw * ((H / G + 3) / 4) * 4 + 31) / 32) * 16 * kUmmaRows * sizeof(float) : 0;
  return p;
}
bool plan_ok(int H, int G, int vdim) { return H >= 1 && G >= 1 && H % G == 0 && H / G <= 32 && vdim >= 1 && vdim <= 128; }

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" uint64_t pace_attn_pooled_prompt_workspace_bytes(int32_t n_entries, int32_t max_tokens, int32_t n_q_heads, int32_t n_kv_heads,
                                                            int32_t vdim, int32_t mixed) {
  if (n_entries <= 0 || max_tokens <= 0 || !plan_ok(n_q_heads, n_kv_heads, vdim)) return 0;
  return plan_units(n_entries, max_tokens, n_q_heads, n_kv_heads, vdim, mixed != 0).bytes;
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
      !(a->scale > 0.f) || !plan_ok(p.H, p.G, a->vdim) || a->dim > 128 || a->vdim % 8 || a->out_stride % 8 || (a->gate && a->gate_stride % 8) || !aligned16(a->q) ||
      !aligned16(a->out) || !aligned16(a->gate))
    return PACE_ERR_UNSUPPORTED;
  const int KB = (a->dim + 63) / 64, VB = (a->vdim + 63) / 64;
  p.kv = make_view(pl, layer, nullptr);
  p.bk = a->block > 0 ? make_view(bp, block_layer, nullptr) : p.kv;
  p.st = *st;
  p.gate = static_cast<const __nv_bfloat16*>(a->gate);
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.acc = static_cast<float4*>(a->workspace);
  p.sinks = a->sinks;
  p.mix = a->mix;
  p.out_stride = a->out_stride;
  p.gate_stride = a->gate_stride;
  p.vdim = a->vdim;
  p.window = a->window;
  p.block = a->block;
  p.entry0 = a->entry_begin;
  p.n_entries = a->entry_end - a->entry_begin;
  const Plan plan = plan_units(p.n_entries, a->max_tokens, p.H, p.G, p.vdim, p.mix != nullptr);
  p.tpw = plan.tpw;
  p.n_tiles = plan.n_tiles;
  p.nv = plan.nv;
  p.n_sub = plan.n_sub;
  p.scale_log2 = a->scale * kLog2e;
  if ((int64_t)p.n_entries * p.n_tiles * p.n_sub > 0x7fffffff) return PACE_ERR_UNSUPPORTED;
  if (plan.bytes && (!a->workspace || !aligned16(a->workspace) || a->workspace_bytes < plan.bytes)) return PACE_ERR_INVALID;
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
