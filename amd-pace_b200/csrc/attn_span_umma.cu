// Prompt attention with a span (window or chunk), a distance bias and a sink on tcgen05, keys and values of different
// widths.  The form is the wide one of attn_umma.cuh: 256 query rows (row = token * group + head of the group) of one
// (entry, KV head) are two 128-row tiles, A and B, that share every chunk of 64 keys a block fetches; a softmax warpgroup
// per tile, one query row per thread; weights enter the second product as two bf16 terms.  What differs:
//   * a key is a list of 64-column blocks, those of one tensor and then those of a second one that all heads share
//     (expanded latents: the unrotated part per head, the rotated part once), each a tile of its own in shared memory;
//   * keys come from the pool's pages or from plain tensors of expanded rows, through three-dimensional tensor maps;
//   * each tile has its own range of chunks, from the span of its first row to the last position of its last one; a chunk
//     outside a tile's range costs that tile nothing;
//   * persistent blocks walk whole units, none is cut, nothing meets in a workspace.
// Warps 0-7 softmax (A: 0-3, B: 4-7), 8 producer, 9 QK of both tiles, 10 / 11 PV of A / B.
// Tensor memory: [0, 128) S_A S_B, [128, 192) high halves of P_A P_B, [192, 256) low halves, [256, 512) O_A O_B.
#include <algorithm>

#include "span.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64, kBlockBytes = kChunk * 128, kThreads = 384, kMaxStages = 6;
constexpr uint32_t kColP = 128, kColPLow = 192, kColO = 256;
constexpr float kLazy = 8.0f;  // log2 units a row's maximum may grow before O is rescaled

struct PromptParams {
  KVView kv;
  pace_step_t st;
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  const float* slopes;
  const float* sinks;
  const int32_t* key_cu;   // nullptr: paged
  const int32_t* key_pos;
  int q_elems, out_elems, H, Hkv, G, k_dim, k2_dim, vdim, nb1;
  int entry0, n_entries, n_qt, span, span_size, n_stages;
  float scale_log2;
  ScoreCap cap;
  int64_t out_row;
};

struct Unit {
  int g, t0, start, R, r0, slot;
  int base;        // position of the first key of chunk 0
  int row0;        // expanded rows: row of that key
  int lo[2], hi[2];  // chunks of tile A and B
  int n;
};

__device__ __forceinline__ bool get_unit(const PromptParams& p, int u, Unit* w) {
  const int qt = p.n_qt - 1 - u % p.n_qt, eh = u / p.n_qt;   // long units first
  const int i = eh / p.Hkv, e = p.entry0 + i;
  w->g = eh - i * p.Hkv;
  w->t0 = p.st.cu[e];
  const int count = p.st.cu[e + 1] - w->t0;
  w->R = count * p.G;
  w->r0 = qt * 2 * kUmmaRows;
  if (w->r0 >= w->R) return false;
  w->start = p.st.start[e];
  w->slot = p.st.slot[e];
  int first = span_first(p.span, p.span_size, w->start + w->r0 / p.G);
  w->base = p.key_cu ? first : first & ~(kChunk - 1);
  w->row0 = p.key_cu ? p.key_cu[i] + w->base - p.key_pos[i] : 0;
  w->n = 0;
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    const int ra = w->r0 + t * kUmmaRows, rz = min(w->R, ra + kUmmaRows) - 1;
    w->lo[t] = w->hi[t] = 0;
    if (ra < w->R) {
      w->lo[t] = (span_first(p.span, p.span_size, w->start + ra / p.G) - w->base) / kChunk;
      w->hi[t] = (w->start + rz / p.G - w->base) / kChunk + 1;
      w->n = w->hi[t];
    }
  }
  return true;
}

struct Bars {
  uint64_t full[kMaxStages], empty[kMaxStages], s_full[2], s_free[2], p_full[2], o_full[2], q_ready[2], drain[3];
};

// What happens to a score in front of the softmax: nothing, a distance bias, a cap.
enum { kPlain = 0, kBias = 1, kCap = 2 };

// KB, VB: 64-column blocks of a key and of a value
template <int KB, int VB, int MODE>
__device__ __forceinline__ void prompt_softmax(const PromptParams& p, Bars& b, uint32_t tmem, unsigned char* qs, int n_units,
                                               volatile int* abort) {
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 7, row = tid & 127;
  const uint32_t t_lane = tmem + ((uint32_t)(row & ~31) << 16);
  const uint32_t tS = t_lane + w * kChunk, tP = t_lane + kColP + w * 32, tPl = t_lane + kColPLow + w * 32,
                 tO = t_lane + kColO + w * 128;
  constexpr bool BIAS = MODE == kBias, LOG2 = MODE != kPlain;   // LOG2: the scores are made log2 units first
  unsigned char* qrow = qs + w * KB * (kUmmaRows * 128) + row * 128;
  const float scale = p.scale_log2;
  const uint64_t scale2 = pack64(__float_as_uint(scale), __float_as_uint(scale));
  int cnt = 0;  // chunks this group has worked on
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un) || un.hi[w] == un.lo[w]) continue;
    const int r = un.r0 + w * kUmmaRows + row;
    const bool live = r < un.R;
    const int tok = (live ? r : un.R - 1) / p.G, head = un.g * p.G + (live ? r : un.R - 1) - tok * p.G;
    const int pos = un.start + tok, first = span_first(p.span, p.span_size, pos);
    {
      const uint4* src = reinterpret_cast<const uint4*>(p.q + ((size_t)(un.t0 + tok) * p.H + head) * p.q_elems);
#pragma unroll
      for (int cc = 0; cc < KB * 8; ++cc) {
        const int blk = cc >> 3, off = (cc & 7) * 8;
        const int c1 = blk * 64 + off, c2 = (blk - p.nb1) * 64 + off;
        const bool second = blk >= p.nb1, ok = live && (second ? c2 < p.k2_dim : c1 < p.k_dim);
        const uint4 v = ok ? __ldg(src + (second ? p.k_dim + c2 : c1) / 8) : make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(qrow + blk * (kUmmaRows * 128) + (((cc & 7) ^ (row & 7)) << 4)) = v;
      }
      fence_proxy_async();  // generic-proxy writes before the tensor core's async-proxy reads
      __syncwarp();
      if (lane == 0) mbar_arrive(&b.q_ready[w]);
    }
    const float slope = BIAS ? p.slopes[head] * kLog2e : 0.f;
    float m = -INFINITY, l = 0.f;
    for (int c = un.lo[w]; c < un.hi[w]; ++c, ++cnt) {
      if (!umma_wait(&b.s_full[w], cnt & 1, abort)) return;
      tc_fence_after();
      uint32_t sr[2][32];
      tmem_ld32(tS, sr[0]);
      tmem_ld32(tS + 32, sr[1]);
      tmem_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&b.s_free[w]);   // the scores are in registers
      const int p0 = un.base + c * kChunk;
      if constexpr (BIAS) {
        // scores in log2 units with their bias, slope * (p0 + k - pos)
        const float off = slope * (float)(p0 - pos);
        const uint64_t off2 = pack64(__float_as_uint(off), __float_as_uint(off)),
                       sl2 = pack64(__float_as_uint(slope), __float_as_uint(slope));
#pragma unroll
        for (int k = 0; k < 32; ++k) {
          uint32_t& a0 = sr[k >> 4][(2 * k) & 31];
          uint32_t& a1 = sr[k >> 4][(2 * k + 1) & 31];
          const uint64_t kk = pack64(__float_as_uint((float)(2 * k)), __float_as_uint((float)(2 * k + 1)));
          unpack64(fma2(pack64(a0, a1), scale2, fma2(kk, sl2, off2)), a0, a1);
        }
      }
      if constexpr (MODE == kCap) {
        // two capped scores share a reciprocal: 1 / a = b / (a b); the exponent's bound keeps the product finite
        const float cin = p.cap.in, cout = p.cap.out;
        const uint64_t cin2 = pack64(__float_as_uint(cin), __float_as_uint(cin)),
                       one2 = pack64(0x3f800000u, 0x3f800000u), c2 = pack64(__float_as_uint(cout), __float_as_uint(cout)),
                       zero2 = 0ull;
#pragma unroll
        for (int k = 0; k < 32; ++k) {
          uint32_t& a0 = sr[k >> 4][(2 * k) & 31];
          uint32_t& a1 = sr[k >> 4][(2 * k + 1) & 31];
          uint32_t x0, x1;
          unpack64(fma2(pack64(a0, a1), cin2, zero2), x0, x1);
          const float y0 = fminf(__uint_as_float(x0), 60.f), y1 = fminf(__uint_as_float(x1), 60.f);
          float e0, e1;
          if (k & 1) {
            exp2_poly2_fine(y0, y1, e0, e1);
          } else {
            e0 = fast_exp2(y0);
            e1 = fast_exp2(y1);
          }
          uint32_t d0, d1;
          unpack64(add2(pack64(__float_as_uint(e0), __float_as_uint(e1)), one2), d0, d1);
          const float r = -2.0f * cout * rcp_t<__nv_bfloat16>(__uint_as_float(d0) * __uint_as_float(d1));
          const uint64_t rr = pack64(__float_as_uint(r), __float_as_uint(r));
          unpack64(fma2(rr, pack64(d1, d0), c2), a0, a1);
        }
      }
      const int lo = max(0, first - p0), hi = min(kChunk, pos + 1 - p0);  // visible keys of the chunk: [lo, hi)
      if (!__all_sync(0xffffffffu, !live || (lo <= 0 && hi >= kChunk))) {
        const unsigned seen = hi > lo ? (unsigned)(hi - lo) : 0u;
#pragma unroll
        for (int k = 0; k < 64; ++k)
          if ((unsigned)(k - lo) >= seen) sr[k >> 5][k & 31] = 0xff800000u;  // -inf
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int k = 0; k < 32; ++k)
        mx4[k & 3] = max3(mx4[k & 3], __uint_as_float(sr[k >> 4][(2 * k) & 31]), __uint_as_float(sr[k >> 4][(2 * k + 1) & 31]));
      float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      if (!LOG2) mx *= scale;  // scale > 0
      const bool grow = mx > m + kLazy;
      if (__any_sync(0xffffffffu, grow)) {
        const float m_new = grow ? mx : m;
        const float alpha = grow ? ((m == -INFINITY) ? 0.f : fast_exp2(m - m_new)) : 1.f;
        if (c > un.lo[w]) {  // O holds the sum of the unit's earlier chunks
          if (!umma_wait(&b.o_full[w], (cnt - 1) & 1, abort)) return;
          tc_fence_after();
#pragma unroll
          for (int d0 = 0; d0 < VB * 64; d0 += 16) {
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
      }
      const float ne = (m == -INFINITY) ? 0.f : -m;
      const uint64_t ne2 = pack64(__float_as_uint(ne), __float_as_uint(ne));
      uint64_t l2[2] = {0ull, 0ull};
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        uint32_t ph[16], pl[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) {
          const uint64_t s2 = pack64(sr[hf][2 * k], sr[hf][2 * k + 1]);
          uint32_t x0, x1;
          unpack64(LOG2 ? add2(s2, ne2) : fma2(s2, scale2, ne2), x0, x1);
          float p0f, p1f;
          if (k & 1) {
            exp2_poly2_fine(__uint_as_float(x0), __uint_as_float(x1), p0f, p1f);   // half of them on the FMA pipe
          } else {
            p0f = fast_exp2(__uint_as_float(x0));
            p1f = fast_exp2(__uint_as_float(x1));
          }
          l2[k & 1] = add2(l2[k & 1], pack64(__float_as_uint(p0f), __float_as_uint(p1f)));
          split_bf2(p0f, p1f, ph[k], pl[k]);
        }
        if (hf == 0 && cnt > 0) {  // the products of the group's previous chunk have read P
          if (!umma_wait(&b.o_full[w], (cnt - 1) & 1, abort)) return;
          tc_fence_after();
        }
        tmem_st16(tP + hf * 16, ph);
        tmem_st16(tPl + hf * 16, pl);
      }
      {
        uint32_t a0, a1, b0, b1;
        unpack64(l2[0], a0, a1);
        unpack64(l2[1], b0, b1);
        l += (__uint_as_float(a0) + __uint_as_float(a1)) + (__uint_as_float(b0) + __uint_as_float(b1));
      }
      tmem_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&b.p_full[w]);
    }
    // ---- the unit's rows ----
    if (!umma_wait(&b.o_full[w], (cnt - 1) & 1, abort)) return;
    tc_fence_after();
    float f = 1.f, den = l;
    if (p.sinks) {
      const float sk = p.sinks[head] * kLog2e, top = fmaxf(m, sk);
      f = m == -INFINITY ? 0.f : fast_exp2(m - top);
      den = l * f + fast_exp2(sk - top);
    }
    const float inv = den > 0.f ? f / den : 0.f;
    __nv_bfloat16* dst = p.out + (un.t0 + tok) * p.out_row + (int64_t)head * p.out_elems;
#pragma unroll
    for (int d0 = 0; d0 < VB * 64; d0 += 32) {
      uint32_t om[32];
      tmem_ld32(tO + d0, om);
      tmem_wait_ld();
      if (live) {
#pragma unroll
        for (int q4 = 0; q4 < 4; ++q4) {
          const int d = d0 + q4 * 8;
          float v[8];
#pragma unroll
          for (int k = 0; k < 8; ++k) v[k] = __uint_as_float(om[q4 * 8 + k]) * inv;
          if (d < p.vdim) Vec<__nv_bfloat16, 8>::store(dst + d, v);
        }
      }
    }
    tc_fence_before();
  }
}

template <int KB, int VB>
__device__ __forceinline__ void prompt_issue_qk(const PromptParams& p, Bars& b, uint32_t tmem, unsigned char* qs,
                                                unsigned char* ring, int n_units, volatile int* abort) {
  constexpr uint32_t IDESC = umma_idesc(kChunk, false);
  constexpr int QB = kUmmaRows * 128, STAGE = (KB + VB) * kBlockBytes;
  const bool leader = elect_one();
  const uint32_t q_lo[2] = {(smem_u32(qs) >> 4) | (1u << 16), (smem_u32(qs + KB * QB) >> 4) | (1u << 16)};
  // 16-column steps of the last block of either part that hold anything
  const int last1 = (p.k_dim - (p.nb1 - 1) * 64 + 15) / 16, last2 = KB > p.nb1 ? (p.k2_dim - (KB - p.nb1 - 1) * 64 + 15) / 16 : 4;
  int s = 0, ph = 0, used[2] = {0, 0}, parts[2] = {0, 0};
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    for (int c = 0; c < un.n; ++c) {
      if (!umma_issuer_wait(&b.full[s], ph, abort)) return;
      const uint32_t k_lo = (smem_u32(ring + (size_t)s * STAGE) >> 4) | (1u << 16);
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        if (c < un.lo[w] || c >= un.hi[w]) continue;
        if (c == un.lo[w]) {
          if (!umma_issuer_wait(&b.q_ready[w], parts[w] & 1, abort)) return;
          ++parts[w];
        }
        if (used[w] > 0 && !umma_issuer_wait(&b.s_free[w], (used[w] - 1) & 1, abort)) return;
        // B's scores follow once A's of the same chunk are in registers: the groups' exponentials coincide less
        if (w == 1 && c >= un.lo[0] && c < un.hi[0] && !umma_issuer_wait(&b.s_free[0], (used[0] - 1) & 1, abort)) return;
        tc_fence_after();
        if (leader) {
          uint32_t acc = 0;
#pragma unroll
          for (int kb = 0; kb < KB; ++kb) {
            const int steps = kb == p.nb1 - 1 ? last1 : kb == KB - 1 ? last2 : 4;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              if (kk < steps) {
                umma_bf16(tmem + w * kChunk, pack64(q_lo[w] + kb * (QB >> 4) + kk * 2, kDescHi),
                          pack64(k_lo + kb * (kBlockBytes >> 4) + kk * 2, kDescHi), IDESC, acc);
                acc = 1u;
              }
          }
          umma_commit(&b.s_full[w]);
        }
        __syncwarp();
        ++used[w];
      }
      if (++s == p.n_stages) s = 0, ph ^= 1;
    }
  }
}

template <int KB, int VB>
__device__ __forceinline__ void prompt_issue_pv(const PromptParams& p, Bars& b, uint32_t tmem, unsigned char* ring, int n_units,
                                                int w, volatile int* abort) {
  constexpr uint32_t IDESC = umma_idesc(VB * 64, true);
  constexpr int STAGE = (KB + VB) * kBlockBytes;
  const bool leader = elect_one();
  const uint32_t tO = tmem + kColO + w * 128, tP = tmem + kColP + w * 32, tPl = tmem + kColPLow + w * 32;
  int s = 0, ph = 0, used = 0;
  for (int u = blockIdx.x; u < n_units; u += gridDim.x) {
    Unit un;
    if (!get_unit(p, u, &un)) continue;
    for (int c = 0; c < un.n; ++c) {
      if (c < un.lo[w] || c >= un.hi[w]) {  // nothing for this tile: its share of the stage goes back once the stage is there
        if (!umma_issuer_wait(&b.full[s], ph, abort)) return;
        if (leader) mbar_arrive(&b.empty[s]);
        __syncwarp();
      } else {
        if (!umma_issuer_wait(&b.p_full[w], used & 1, abort)) return;
        tc_fence_after();
        if (leader) {
          // MN-major: the next 64 columns lie one block further on
          const uint32_t v_lo = (smem_u32(ring + (size_t)s * STAGE + KB * kBlockBytes) >> 4) | ((uint32_t)(kBlockBytes >> 4) << 16);
          const uint32_t acc = c > un.lo[w] ? 1u : 0u;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ts(tO, tP + k * 8, pack64(v_lo + k * (2048 >> 4), kDescHi), IDESC, k ? 1u : acc);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_bf16_ts(tO, tPl + k * 8, pack64(v_lo + k * (2048 >> 4), kDescHi), IDESC, 1u);
          umma_commit(&b.empty[s]);
          umma_commit(&b.o_full[w]);
        }
        __syncwarp();
        ++used;
      }
      if (++s == p.n_stages) s = 0, ph ^= 1;
    }
  }
}

template <int KB, int VB, int MODE>
__global__ void __launch_bounds__(kThreads, 1)
    attn_span_prompt_kernel(const PromptParams p, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmK2,
                            const __grid_constant__ CUtensorMap tmV) {
  constexpr int STAGE = (KB + VB) * kBlockBytes;
  extern __shared__ unsigned char smem_raw[];
  __shared__ Bars b;
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  unsigned char* qs = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  unsigned char* ring = qs + 2 * KB * kUmmaRows * 128;
  volatile int* abort = &abort_flag;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int n_units = p.n_entries * p.Hkv * p.n_qt;
  if (warp == 9) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < p.n_stages; ++i) {
      mbar_init(&b.full[i], 1);
      mbar_init(&b.empty[i], 2);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&b.s_full[i], 1);
      mbar_init(&b.s_free[i], 4);
      mbar_init(&b.p_full[i], 4);
      mbar_init(&b.o_full[i], 1);
      mbar_init(&b.q_ready[i], 4);
    }
    for (int i = 0; i < 3; ++i) mbar_init(&b.drain[i], 1);
    fence_mbar_init();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&tmem_slot);

  if (warp < 8) {
    prompt_softmax<KB, VB, MODE>(p, b, tmem, qs, n_units, abort);
  } else if (warp == 8) {
    int s = 0, ph = 0, issued = 0;
    bool ok = true;
    for (int u = blockIdx.x; u < n_units && ok; u += gridDim.x) {
      Unit un;
      if (!get_unit(p, u, &un)) continue;
      int page = 0;
      for (int c = 0; c < un.n; ++c) {
        if (!p.key_cu && (c & 31) == 0) {  // the next 32 chunks' pages, one per lane
          page = 0;
          if (c + lane < un.n) {
            page = un.slot >= 0 && un.slot < p.kv.max_seqs ? view_page(p.kv, un.slot, un.base / kChunk + c + lane) : -1;
            if (page < 0) {
              raise_status(p.kv.status, PACE_DEV_BAD_INDEX);
              page = 0;
            }
          }
        }
        if (issued >= p.n_stages && !__all_sync(0xffffffffu, mbar_wait(&b.empty[s], ph ^ 1, abort))) {
          ok = false;
          break;
        }
        unsigned char* st = ring + (size_t)s * STAGE;
        if (lane == 0) mbar_arrive_expect_tx(&b.full[s], STAGE);
        __syncwarp();
        const int pg = __shfl_sync(0xffffffffu, page, c & 31);
        const int c1 = p.key_cu ? un.row0 + c * kChunk : 0, c2 = p.key_cu ? un.g : pg * p.Hkv + un.g;
        if (lane < KB) {
          if (lane < p.nb1) tma_load_3d(st + lane * kBlockBytes, &tmK, lane * 64, c1, c2, &b.full[s]);
          else tma_load_2d(st + lane * kBlockBytes, &tmK2, (lane - p.nb1) * 64, c1, &b.full[s]);
        } else if (lane < KB + VB) {
          tma_load_3d(st + lane * kBlockBytes, &tmV, (lane - KB) * 64, c1, c2, &b.full[s]);
        }
        ++issued;
        if (++s == p.n_stages) s = 0, ph ^= 1;
      }
    }
    if (!ok) {  // copies in flight land before the block's shared memory is released
      for (int k = issued > p.n_stages ? issued - p.n_stages : 0; k < issued; ++k) mbar_wait(&b.full[k % p.n_stages], (k / p.n_stages) & 1);
    }
  } else {
    if (warp == 9) prompt_issue_qk<KB, VB>(p, b, tmem, qs, ring, n_units, abort);
    else prompt_issue_pv<KB, VB>(p, b, tmem, ring, n_units, warp - 10, abort);
    // nothing may still be writing tensor memory when it is handed back
    if (elect_one()) {
      umma_commit(&b.drain[warp - 9]);
      for (int k = 0; k < (1 << 20) && !mbar_try_wait(&b.drain[warp - 9], 0); ++k) __nanosleep(64);
    }
    __syncwarp();
  }
  if (lane == 0 && *abort) raise_status(p.kv.status, PACE_DEV_WAIT_TIMEOUT);
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
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
int launch_prompt(PromptParams& p, const CUtensorMap& tk, const CUtensorMap& tk2, const CUtensorMap& tv, cudaStream_t s) {
  constexpr int STAGE = (KB + VB) * kBlockBytes, QBYTES = 2 * KB * kUmmaRows * 128;
  p.n_stages = std::min(kMaxStages, (226 * 1024 - 1024 - 512 - QBYTES) / STAGE);
  static_assert((226 * 1024 - 1024 - 512 - QBYTES) / STAGE >= 2, "two stages fit");
  const int smem = QBYTES + p.n_stages * STAGE + 1024;
  const int units = p.n_entries * p.Hkv * p.n_qt, blocks = std::min(units, sm_count());
  auto launch = [&](auto* fn) {
    PACE_CUDA_TRY(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    fn<<<blocks, kThreads, smem, s>>>(p, tk, tk2, tv);
    return PACE_OK;
  };
  const int rc = p.cap.out != 0.f ? launch(attn_span_prompt_kernel<KB, VB, kCap>)
                 : p.slopes       ? launch(attn_span_prompt_kernel<KB, VB, kBias>)
                                  : launch(attn_span_prompt_kernel<KB, VB, kPlain>);
  if (rc != PACE_OK) return rc;
  PACE_LAUNCH_CHECK("attn_span_prompt_kernel");
  return PACE_OK;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" int pace_attn_span_prefill(const pace_kv_pool_t* pl, int32_t layer, const pace_step_t* st,
                                      const pace_attn_span_prefill_args_t* x, void* stream) {
  if (!pl || !pl->pages || !pl->block_table || !step_ok(st) || !x || layer < 0 || layer >= pl->n_layers) return PACE_ERR_INVALID;
  const pace_attn_span_args_t* a = &x->a;
  const bool paged = !x->k;
  const int Hkv = paged ? pl->n_kv_heads : x->n_kv_heads;
  if (!span_args_ok(st, a, Hkv)) return PACE_ERR_INVALID;
  if (!paged && (!x->v || !x->key_cu || !x->key_pos || x->n_rows < 1 || x->k_dim < 1 || x->k2_dim < 0 || (x->k2_dim && !x->k2) ||
                 x->k_dim + x->k2_dim != a->dim || a->q_elems < a->dim))
    return PACE_ERR_INVALID;
  if (st->n_tokens == 0 || a->entry_begin == a->entry_end || a->max_tokens == 0) return PACE_OK;
  if (a->dtype != PACE_DTYPE_BF16 || !(a->scale > 0.f) || a->vdim > 128 || a->vdim % 8 || a->out_elems % 8 || a->out_row % 8 || (a->slopes && a->softcap > 0.f) || a->q_elems % 8 ||
      !aligned16(a->q) || !aligned16(a->out))
    return PACE_ERR_UNSUPPORTED;
  PromptParams p;
  p.kv = make_view(pl, layer, nullptr);
  p.k_dim = paged ? (a->dim + 7) / 8 * 8 : x->k_dim;   // (pool and query rows are zero up to the next multiple of 8)
  p.k2_dim = paged ? 0 : x->k2_dim;
  p.nb1 = (p.k_dim + 63) / 64;
  const int nb2 = (p.k2_dim + 63) / 64, KB = p.nb1 + nb2, VB = (a->vdim + 63) / 64;
  if (KB > 4 || p.k_dim % 8 || p.k2_dim % 8) return PACE_ERR_UNSUPPORTED;
  CUtensorMap tk, tk2, tv;
  const uint32_t box[3] = {64, kChunk, 1};
  int rc;
  if (paged) {
    if (pl->row_format != PACE_ROWS_BF16 || pl->page_tokens != kChunk) return PACE_ERR_UNSUPPORTED;
    const uint64_t row = (uint64_t)pl->head_dim;
    const uint64_t dims[3] = {row, kChunk, (uint64_t)pl->n_pages * Hkv}, str[2] = {row * 2, row * 2 * kChunk};
    rc = tensor_map_bf16(&tk, p.kv.k, 3, dims, str, box);
    if (rc == PACE_OK) rc = tensor_map_bf16(&tv, p.kv.v, 3, dims, str, box);
    tk2 = tk;
  } else {
    if (x->k_row % 8 || x->k_head % 8 || x->v_row % 8 || x->v_head % 8 || !aligned16(x->k) || !aligned16(x->v) ||
        (x->k2_dim && (x->k2_row % 8 || !aligned16(x->k2))))
      return PACE_ERR_UNSUPPORTED;
    const uint64_t n = (uint64_t)x->n_rows;
    const uint64_t dk[3] = {(uint64_t)x->k_dim, n, (uint64_t)Hkv}, sk[2] = {(uint64_t)x->k_row * 2, (uint64_t)x->k_head * 2};
    const uint64_t dv[3] = {(uint64_t)a->vdim, n, (uint64_t)Hkv}, sv[2] = {(uint64_t)x->v_row * 2, (uint64_t)x->v_head * 2};
    rc = tensor_map_bf16(&tk, x->k, 3, dk, sk, box);
    if (rc == PACE_OK) rc = tensor_map_bf16(&tv, x->v, 3, dv, sv, box);
    tk2 = tk;
    if (rc == PACE_OK && x->k2_dim) {
      const uint64_t d2[2] = {(uint64_t)x->k2_dim, n}, s2[1] = {(uint64_t)x->k2_row * 2};
      rc = tensor_map_bf16(&tk2, x->k2, 2, d2, s2, box);
    }
  }
  if (rc != PACE_OK) return rc;
  p.st = *st;
  p.q = static_cast<const __nv_bfloat16*>(a->q);
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.slopes = a->slopes;
  p.sinks = a->sinks;
  p.key_cu = paged ? nullptr : x->key_cu;
  p.key_pos = paged ? nullptr : x->key_pos;
  p.q_elems = a->q_elems;
  p.out_elems = a->out_elems;
  p.H = a->n_q_heads;
  p.Hkv = Hkv;
  p.G = a->n_q_heads / Hkv;
  p.vdim = a->vdim;
  p.entry0 = a->entry_begin;
  p.n_entries = a->entry_end - a->entry_begin;
  const int64_t n_qt = ((int64_t)a->max_tokens * p.G + 2 * kUmmaRows - 1) / (2 * kUmmaRows);
  if (n_qt * p.n_entries * Hkv > 0x7fffffff) return PACE_ERR_UNSUPPORTED;
  p.n_qt = (int)n_qt;
  p.span = a->span;
  p.span_size = a->span_size;
  p.scale_log2 = a->scale * kLog2e;
  p.cap = score_cap(a->scale, a->softcap);
  p.out_row = span_out_row(*a);
  PACE_PROFILE("attn_span_prefill", stream, "layer=%d entries=%d tokens<=%d heads=%d dims=%d/%d", layer, p.n_entries, a->max_tokens,
               p.H, a->dim, a->vdim);
  const cudaStream_t s = (cudaStream_t)stream;
#define PACE_PROMPT_CASE(kb, vb) \
  if (KB == kb && VB == vb) return launch_prompt<kb, vb>(p, tk, tk2, tv, s);
  PACE_PROMPT_CASE(1, 1) PACE_PROMPT_CASE(2, 1) PACE_PROMPT_CASE(3, 1) PACE_PROMPT_CASE(4, 1)
  PACE_PROMPT_CASE(1, 2) PACE_PROMPT_CASE(2, 2) PACE_PROMPT_CASE(3, 2) PACE_PROMPT_CASE(4, 2)
#undef PACE_PROMPT_CASE
  return PACE_ERR_UNSUPPORTED;
}
