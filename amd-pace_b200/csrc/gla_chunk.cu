// Gated linear attention with a decay per key channel over many tokens, in chunks of 64 on the tensor cores.
//
// With G_i the sum of the chunk's log decays up to token i (a vector over the key channels), x^(G) for the elementwise product with
// e^G, and S the state in front of the chunk
//     P_ij = q_i . (k_j)^(G_i - G_j)  (j <= i),     O = Q^(G) S + P V,     S' = S^(G_n) + (K^(G_n - G))^T V
// Nothing but S connects the chunks, so a first launch makes Q^(G), K^(G_n - G) and P side by side, a block per (chunk, head,
// entry); a second one walks the chunks, a block per (entry, head, 16 or 32 value columns) with its part of S in fp32 accumulators.
//
// e^(G_i - G_j) is the product of a row's factor e^(G_i - M) and a column's e^(M - G_j), M the sum up to the middle of the column's
// sixteen tokens: both are finite as long as eight tokens decay by less than e^60.  Sixteen columns with a channel beyond
// that take M behind them (both factors are then at most 1 for the rows further down) and their own 16 x 16 block pair by pair.
//
// q, k, v are bf16 values; everything else is fp32: where an fp32 quantity is the operand of a bf16 product it is split into two
// bf16 terms, of whose products with another split quantity the three that matter are taken (16 bits).
#include "chunk_mma.cuh"
#include "gla.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64, kThreads = 256, kTP = kChunk + 8;
constexpr float kRange = 86.0f;   // log2 units eight tokens may decay by on the fast path: e^60

// What the first launch leaves of a (entry, chunk, head), as it lies in shared memory later: bf16 tiles of 64 rows of QP (high,
// low halves), P 64 rows of kTP, then the fp32 decays over the whole chunk.
template <int DP>
struct Slot {
  static constexpr int QP = DP + 8, kTile = kChunk * QP;
  static constexpr int kQ = 0, kP = 2 * kTile, kK = kP + 2 * kChunk * kTP, kHalves = kK + 2 * kTile;
  static constexpr size_t kDecay = (size_t)kHalves * 2, bytes = kDecay + DP * 4;
};

struct Slab {
  unsigned char* scratch;
  int first, n;    // chunks [first, first + n) of every entry
};

template <int DP>
struct Prep {
  static constexpr int QP = DP + 8, GP = DP + 8;
  static constexpr int kK = 0, kQ = kK + kChunk * QP * 2, kG = kQ + kChunk * QP * 2, kHi = kG + kChunk * GP * 4, kLo = kHi + kChunk * QP * 2,
                       kFlag = kLo + kChunk * QP * 2, bytes = kFlag + 16;
};

template <int DP>
__global__ void __launch_bounds__(kThreads, 2) gla_prepare_kernel(pace_step_t st, pace_gla_args_t a, Slab sl) {
  using SL = Slot<DP>;
  using PR = Prep<DP>;
  constexpr int QP = PR::QP, GP = PR::GP;
  const int e = blockIdx.z, h = blockIdx.y, d = a.dim, H = a.heads;
  const int count = st.cu[e + 1] - st.cu[e], l0 = (sl.first + (int)blockIdx.x) * kChunk;
  if (l0 >= count) return;
  const int n_tok = min(kChunk, count - l0), t0 = st.cu[e] + l0;
  extern __shared__ __align__(16) unsigned char sm[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(sm + PR::kK);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(sm + PR::kQ);
  float* G = reinterpret_cast<float*>(sm + PR::kG);      // sums of log decays, log2 units
  __nv_bfloat16* kc_hi = reinterpret_cast<__nv_bfloat16*>(sm + PR::kHi);   // the keys with their column factors
  __nv_bfloat16* kc_lo = reinterpret_cast<__nv_bfloat16*>(sm + PR::kLo);
  int* slow = reinterpret_cast<int*>(sm + PR::kFlag);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  unsigned char* slot = sl.scratch + (((size_t)e * sl.n + blockIdx.x) * H + h) * SL::bytes;
  __nv_bfloat16* tiles = reinterpret_cast<__nv_bfloat16*>(slot);

  // ---- operands: keys and queries as they are, log decays ----
  const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(a.qkv) + (size_t)t0 * a.qkv_stride;
  for (int i = tid; i < kChunk * (DP / 8) * 2; i += kThreads) {
    const int which = i / (kChunk * (DP / 8)), r = i - which * (kChunk * (DP / 8)), j = r / (DP / 8), c = (r - j * (DP / 8)) * 8;
    const bool live = j < n_tok && c < d;
    copy16((which ? ks : qs) + j * QP + c, qkv + (live ? (size_t)j * a.qkv_stride + (size_t)(which * H + h) * d + c : 0), live);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (tid < 4) slow[tid] = 0;
  {
    // a thread has eight channels of every (kThreads / (DP / 8))-th token
    const int c = tid % (DP / 8) * 8, j0 = tid / (DP / 8);
    const uint64_t neg = both(-a.inv_tau * kLog2e);
    const __nv_bfloat16* zr = static_cast<const __nv_bfloat16*>(a.z) + (size_t)t0 * a.z_stride + (size_t)h * d + c;
    float bias[8];
#pragma unroll
    for (int x = 0; x < 8; ++x) bias[x] = c < d ? a.z_bias[(size_t)h * d + c + x] : 0.f;
#pragma unroll
    for (int j = j0; j < kChunk; j += kThreads / (DP / 8)) {
      uint64_t v[4] = {0ull, 0ull, 0ull, 0ull};
      if (j < n_tok && c < d) {
        float x[8];
        Vec<__nv_bfloat16, 8>::load(zr + (size_t)j * a.z_stride, x);
#pragma unroll
        for (int u = 0; u < 4; ++u) v[u] = fma2(softplus2(-(x[2 * u] + bias[2 * u]), -(x[2 * u + 1] + bias[2 * u + 1])), neg, 0ull);
      }
#pragma unroll
      for (int u = 0; u < 4; u += 2) {
        uint4 w;
        unpack64(v[u], w.x, w.y);
        unpack64(v[u + 1], w.z, w.w);
        *reinterpret_cast<uint4*>(G + j * GP + c + 2 * u) = w;
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  constexpr int PARTS = kThreads / DP, ROWS = kChunk / PARTS;
  const int gc = tid % DP, part = tid / DP;
  {
    float s = 0.f;
#pragma unroll 8
    for (int j = part * ROWS; j < (part + 1) * ROWS; ++j) G[j * GP + gc] = s += G[j * GP + gc];
  }
  __syncthreads();
  float before = 0.f;
  for (int p = 0; p < part; ++p) before += G[((p + 1) * ROWS - 1) * GP + gc];
  __syncthreads();
  if (part > 0) {
#pragma unroll 8
    for (int j = part * ROWS; j < (part + 1) * ROWS; ++j) G[j * GP + gc] += before;
  }
  __syncthreads();
  for (int i = tid; i < 4 * DP; i += kThreads) {
    const int b = i / DP, c = i - b * DP;
    const float m = G[(16 * b + 7) * GP + c], s = b ? G[(16 * b - 1) * GP + c] : 0.f;
    if (s - m > kRange || m - G[(16 * b + 15) * GP + c] > kRange) slow[b] = 1;
  }
  __syncthreads();
  // ---- keys and queries with their decays: those the walk reads, and the columns of the scores ----
  for (int i = tid; i < kChunk * (DP / 4); i += kThreads) {
    const int j = i / (DP / 4), c = (i - j * (DP / 4)) * 4, b = j >> 4, ref = 16 * b + (slow[b] ? 15 : 7);
    const float4 gg = *reinterpret_cast<const float4*>(G + j * GP + c), m = *reinterpret_cast<const float4*>(G + ref * GP + c),
                 ge = *reinterpret_cast<const float4*>(G + (kChunk - 1) * GP + c);
    float kk[4], qq[4];
    Vec<__nv_bfloat16, 4>::load(ks + j * QP + c, kk);
    Vec<__nv_bfloat16, 4>::load(qs + j * QP + c, qq);
    uint2 hi, lo;
    split_bf2(kk[0] * fast_exp2(m.x - gg.x), kk[1] * fast_exp2(m.y - gg.y), hi.x, lo.x);
    split_bf2(kk[2] * fast_exp2(m.z - gg.z), kk[3] * fast_exp2(m.w - gg.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(kc_hi + j * QP + c) = hi;
    *reinterpret_cast<uint2*>(kc_lo + j * QP + c) = lo;
    split_bf2(kk[0] * fast_exp2(ge.x - gg.x), kk[1] * fast_exp2(ge.y - gg.y), hi.x, lo.x);
    split_bf2(kk[2] * fast_exp2(ge.z - gg.z), kk[3] * fast_exp2(ge.w - gg.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(tiles + SL::kK + j * QP + c) = hi;
    *reinterpret_cast<uint2*>(tiles + SL::kK + SL::kTile + j * QP + c) = lo;
    split_bf2(qq[0] * a.q_scale * fast_exp2(gg.x), qq[1] * a.q_scale * fast_exp2(gg.y), hi.x, lo.x);
    split_bf2(qq[2] * a.q_scale * fast_exp2(gg.z), qq[3] * a.q_scale * fast_exp2(gg.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(tiles + SL::kQ + j * QP + c) = hi;
    *reinterpret_cast<uint2*>(tiles + SL::kQ + SL::kTile + j * QP + c) = lo;
  }
  if (tid < DP) reinterpret_cast<float*>(slot + SL::kDecay)[tid] = fast_exp2(G[(kChunk - 1) * GP + tid]);
  __syncthreads();

  // ---- scores: a warp has one or two of the ten 16 x 16 blocks ----
  {
    // (row block, column block) of a warp's first and second task; -1: none
    constexpr int kRow[2][8] = {{0, 1, 1, 2, 2, 2, 3, 3}, {3, 3, -1, -1, -1, -1, -1, -1}};
    constexpr int kCol[2][8] = {{0, 0, 1, 0, 1, 2, 0, 1}, {2, 3, -1, -1, -1, -1, -1, -1}};
    __nv_bfloat16 *p_hi = tiles + SL::kP, *p_lo = p_hi + kChunk * kTP;
#pragma unroll
    for (int task = 0; task < 2; ++task) {
      int rb = -1, cb = -1;
#pragma unroll
      for (int w = 0; w < 8; ++w)
        if (warp == w) rb = kRow[task][w], cb = kCol[task][w];
      if (rb < 0 || (rb == cb && slow[cb])) continue;
      float acc[2][4];
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[s][x] = 0.f;
      const int i0 = 16 * rb + g, ref = 16 * cb + (slow[cb] ? 15 : 7);
      const int at = (16 * cb + (lane & 7) + (lane >> 4) * 8) * QP + ((lane >> 3) & 1) * 8;   // two tiles of 8 columns
#pragma unroll 2
      for (int k0 = 0; k0 < DP; k0 += 16) {
        const int c0 = k0 + 2 * t;
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldsm4(bh, kc_hi + at + k0);
        ldsm4(bl, kc_lo + at + k0);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int row = i0 + (x & 1) * 8, c = c0 + (x >> 1) * 8;
          const float2 gg = *reinterpret_cast<const float2*>(G + row * GP + c), m = *reinterpret_cast<const float2*>(G + ref * GP + c);
          const float2 v = bf2_to_f2(*reinterpret_cast<const uint32_t*>(qs + row * QP + c));
          split_bf2(v.x * fast_exp2(gg.x - m.x), v.y * fast_exp2(gg.y - m.y), ah[x], al[x]);
        }
        mma_split(acc[0], ah, al, bh, bl);
        mma_split(acc[1], ah, al, bh + 2, bl + 2);
      }
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int i = 16 * rb + g + 8 * x, j = 16 * cb + 8 * s + 2 * t;
          uint32_t hi, lo;
          split_bf2(j <= i ? acc[s][2 * x] * a.q_scale : 0.f, j + 1 <= i ? acc[s][2 * x + 1] * a.q_scale : 0.f, hi, lo);
          *reinterpret_cast<uint32_t*>(p_hi + i * kTP + j) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + i * kTP + j) = lo;
        }
    }
    for (int b = 0; b < 4; ++b) {
      if (!slow[b]) continue;
      const int i = 16 * b + tid / 16, j = 16 * b + tid % 16;   // one pair per thread
      float s = 0.f;
      if (j <= i)
        for (int c = 0; c < DP; ++c)
          s = fmaf(__bfloat162float(qs[i * QP + c]), fast_exp2(G[i * GP + c] - G[j * GP + c]) * __bfloat162float(ks[j * QP + c]), s);
      s *= a.q_scale;
      const __nv_bfloat16 hi = __float2bfloat16_rn(s);
      p_hi[i * kTP + j] = hi;
      p_lo[i * kTP + j] = __float2bfloat16_rn(s - __bfloat162float(hi));
    }
  }
}

// The walk over the chunks, transposed: four warps own 16 value columns, each a quarter of the key channels.  The accumulators of
// S^T (16 columns x DQ channels) are, split in two terms, the row operand of S^T Q^T as they are; V^T is that of V^T P^T (of which
// warp q takes tokens 16 q .. 16 q + 15) and V^T K.  What the four warps have of the outputs meets in shared memory in fragment
// form: warp q sums up tokens 16 q .. 16 q + 15.
template <int DP, int GROUPS>
struct Walk {
  static constexpr int VP = 16 * GROUPS + 8;
  static constexpr int kTiles = Slot<DP>::kHalves * 2, kV = kTiles, kExchange = kV + kChunk * VP * 2, bytes = kExchange + GROUPS * 4 * 8 * 32 * 16;
};

template <int DP, int GROUPS>
__global__ void __launch_bounds__(128 * GROUPS, GROUPS == 1 ? 2 : 1) gla_walk_kernel(pace_step_t st, pace_gla_args_t a, Slab sl) {
  using SL = Slot<DP>;
  using WK = Walk<DP, GROUPS>;
  constexpr int QP = SL::QP, DQ = DP / 4, KS = DQ / 16, ND = DQ / 8, THREADS = 128 * GROUPS, VP = WK::VP;
  const int e = blockIdx.z, h = blockIdx.y, d = a.dim, vd = a.vdim, H = a.heads;
  const int count = st.cu[e + 1] - st.cu[e], chunks = min(sl.n, (count + kChunk - 1) / kChunk - sl.first);
  if (chunks <= 0) return;
  extern __shared__ __align__(16) unsigned char sm[];
  const __nv_bfloat16* tiles = reinterpret_cast<const __nv_bfloat16*>(sm);
  const __nv_bfloat16* vs = reinterpret_cast<const __nv_bfloat16*>(sm + WK::kV);
  const int tid = threadIdx.x, lane = tid & 31, group = tid >> 7, q = (tid >> 5) & 3, g = lane >> 2, t = lane & 3;
  float4* xo = reinterpret_cast<float4*>(sm + WK::kExchange) + group * 4 * 8 * 32;   // [warp][token eighth][lane]
  const int vb = blockIdx.x * GROUPS * 16, v0 = vb + group * 16, c0 = q * DQ;
  const unsigned char* slot = sl.scratch + ((size_t)e * sl.n * H + h) * SL::bytes;
  const __nv_bfloat16* v_in = static_cast<const __nv_bfloat16*>(a.qkv) + (size_t)st.cu[e] * a.qkv_stride + 2 * (size_t)H * d + (size_t)h * vd;
  // Q and P of a chunk, and then K and V
  auto fetch = [&](const unsigned char* from, int c, bool second) {
    const int begin = second ? SL::kK * 2 : 0, end = second ? WK::kTiles : SL::kK * 2;
#pragma unroll 8
    for (int i = begin + tid * 16; i < end; i += THREADS * 16) copy16(sm + i, from + i);
    if (second) {
      const int l0 = (sl.first + c) * kChunk;
      for (int i = tid; i < kChunk * 2 * GROUPS; i += THREADS) {
        const int j = i / (2 * GROUPS), cc = (i - j * 2 * GROUPS) * 8;
        const bool live = l0 + j < count && vb + cc < vd;
        copy16(sm + WK::kV + (j * VP + cc) * 2, v_in + (live ? (size_t)(l0 + j) * a.qkv_stride + vb + cc : 0), live);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(slot, 0, false);
  fetch(slot, 0, true);
  float* state = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  const bool fresh = st.start[e] == 0 && sl.first == 0;
  const bool in0 = v0 + g < vd, in1 = v0 + g + 8 < vd;
  float S[ND][4];      // S^T: columns v0 + g, v0 + g + 8; channels c0 + 8 n + 2 t, + 1
#pragma unroll
  for (int n = 0; n < ND; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int r = c0 + 8 * n + 2 * t + (x & 1);
      S[n][x] = !fresh && r < d && (x < 2 ? in0 : in1) ? state[(size_t)r * vd + v0 + g + (x >> 1) * 8] : 0.f;
    }
  // V^T of tokens 16 kt ..: stored by token, so transposed on the way
  const __nv_bfloat16* vt = vs + ((lane & 7) + (lane >> 4) * 8) * VP + group * 16 + ((lane >> 3) & 1) * 8;
  for (int c = 0; c < chunks; ++c, slot += (size_t)H * SL::bytes) {
    const int l0 = (sl.first + c) * kChunk, n_tok = min(kChunk, count - l0);
    const float2* decay = reinterpret_cast<const float2*>(slot + SL::kDecay) + (c0 >> 1) + t;
    float2 dec[ND];
#pragma unroll
    for (int n = 0; n < ND; ++n) dec[n] = decay[4 * n];
    uint32_t sh[KS][4], so[KS][4];
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int x = 0; x < 4; ++x) split_bf2(S[2 * k + (x >> 1)][2 * (x & 1)], S[2 * k + (x >> 1)][2 * (x & 1) + 1], sh[k][x], so[k][x]);
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();                                           // Q and P are there
    // (16 columns) x (64 tokens): S^T times Q^T, this warp's channels
    float D[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) D[n][0] = D[n][1] = D[n][2] = D[n][3] = 0.f;
#pragma unroll
    for (int n4 = 0; n4 < 8; n4 += 4) {
      uint32_t bh[4][4], bl[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const __nv_bfloat16* p = tiles + SL::kQ + (8 * (n4 + n) + (lane & 7)) * QP + c0;
        if constexpr (KS == 2) {
          ldsm4(bh[n], p + (lane >> 3) * 8);
          ldsm4(bl[n], p + SL::kTile + (lane >> 3) * 8);
        } else {      // both halves in one: matrices 0, 1 high, 2, 3 low
          ldsm4(bh[n], p + (lane >> 4) * SL::kTile + ((lane >> 3) & 1) * 8);
          bl[n][0] = bh[n][2], bl[n][1] = bh[n][3];
        }
      }
#pragma unroll
      for (int k = 0; k < KS; ++k) {
#pragma unroll
        for (int n = 0; n < 4; ++n) mma16816(D[n4 + n], sh[k], bh[n][2 * k], bh[n][2 * k + 1]);
#pragma unroll
        for (int n = 0; n < 4; ++n) mma16816(D[n4 + n], sh[k], bl[n][2 * k], bl[n][2 * k + 1]);
#pragma unroll
        for (int n = 0; n < 4; ++n) mma16816(D[n4 + n], so[k], bh[n][2 * k], bh[n][2 * k + 1]);
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                           // K and V are there
    // the outputs' share of tokens 16 q .. + 15
    {
      uint32_t v[4];
      ldsm4t(v, vt + 16 * q * VP);
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        if (n < 2 * q) continue;
        uint32_t b[4];      // matrices 0, 1 high, 2, 3 low
        ldsm4(b, tiles + SL::kP + (lane >> 4) * kChunk * kTP + (8 * n + (lane & 7)) * kTP + 16 * q + ((lane >> 3) & 1) * 8);
        mma16816(D[n], v, b[0], b[1]);
        mma16816(D[n], v, b[2], b[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) xo[(q * 8 + n) * 32 + lane] = make_float4(D[n][0], D[n][1], D[n][2], D[n][3]);
    __syncthreads();                                           // the outputs are there; Q and P have been read
    if (c + 1 < chunks) fetch(slot + (size_t)H * SL::bytes, c + 1, false);
    float Z[ND][4];                                            // the low halves' sum
#pragma unroll
    for (int n = 0; n < ND; ++n) {
      S[n][0] *= dec[n].x; S[n][1] *= dec[n].y;
      S[n][2] *= dec[n].x; S[n][3] *= dec[n].y;
      Z[n][0] = Z[n][1] = Z[n][2] = Z[n][3] = 0.f;
    }
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t v[4];
      ldsm4t(v, vt + 16 * kt * VP);
      const __nv_bfloat16* p = tiles + SL::kK + (16 * kt + (lane & 15)) * QP + c0 + (lane >> 4) * 8;
#pragma unroll
      for (int n = 0; n < ND; n += 2) {
        uint32_t bh[4], bl[4];
        ldsm4t(bh, p + 8 * n);
        ldsm4t(bl, p + SL::kTile + 8 * n);
        mma16816(S[n], v, bh[0], bh[1]);
        mma16816(S[n + 1], v, bh[2], bh[3]);
        mma16816(Z[n], v, bl[0], bl[1]);
        mma16816(Z[n + 1], v, bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < ND; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) S[n][x] += Z[n][x];
    // tokens 16 q .. + 15: neighbouring columns lie in lanes that differ in bit 2, which exchange one of two tokens
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (size_t)(st.cu[e] + l0) * a.out_stride + (size_t)h * vd + v0;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      float4 s = xo[(2 * q + hf) * 32 + lane];
#pragma unroll
      for (int w = 1; w < 4; ++w) {
        const float4 v = xo[(w * 8 + 2 * q + hf) * 32 + lane];
        s.x += v.x, s.y += v.y, s.z += v.z, s.w += v.w;
      }
      const bool odd = g & 1;
      const float g0 = __shfl_xor_sync(0xffffffffu, odd ? s.x : s.y, 4), g1 = __shfl_xor_sync(0xffffffffu, odd ? s.z : s.w, 4);
      const int tok = 16 * q + 8 * hf + 2 * t + (odd ? 1 : 0), col = g & ~1;
      if (tok < n_tok) {
        if (v0 + col < vd) *reinterpret_cast<uint32_t*>(out + (size_t)tok * a.out_stride + col) = odd ? f2_to_bf2(g0, s.y) : f2_to_bf2(s.x, g0);
        if (v0 + col + 8 < vd) *reinterpret_cast<uint32_t*>(out + (size_t)tok * a.out_stride + col + 8) = odd ? f2_to_bf2(g1, s.w) : f2_to_bf2(s.z, g1);
      }
    }
    __syncthreads();                                           // K and V have been read, and the exchange
    if (c + 1 < chunks) fetch(slot + (size_t)H * SL::bytes, c + 1, true);
  }
#pragma unroll
  for (int n = 0; n < ND; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int r = c0 + 8 * n + 2 * t + (x & 1);
      if (r < d && (x < 2 ? in0 : in1)) state[(size_t)r * vd + v0 + g + (x >> 1) * 8] = S[n][x];
    }
}

constexpr uint64_t kBudget = 512ull << 20;   // bytes of scratch a launch pair may use

struct Plan {
  int dp, slab;      // padded key size, chunks of an entry per launch pair
  uint64_t bytes;
};
Plan plan_chunks(int n_entries, int max_count, int heads, int dim) {
  Plan p;
  p.dp = dim <= 64 ? 64 : 128;
  const uint64_t slot = p.dp == 64 ? Slot<64>::bytes : Slot<128>::bytes, row = slot * heads * n_entries;
  const int chunks = (max_count + kChunk - 1) / kChunk;
  const uint64_t fit = kBudget / row;
  p.slab = fit < 1 ? 1 : fit < (uint64_t)chunks ? (int)fit : chunks;
  p.bytes = row * p.slab;
  return p;
}

template <int DP, int GROUPS>
int launch_walk(const pace_step_t& st, const pace_gla_args_t& a, const Slab& sl, cudaStream_t s) {
  PACE_CUDA_TRY(cudaFuncSetAttribute(gla_walk_kernel<DP, GROUPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Walk<DP, GROUPS>::bytes));
  const dim3 grid((unsigned)((a.vdim + 16 * GROUPS - 1) / (16 * GROUPS)), (unsigned)a.heads, (unsigned)st.n_entries);
  gla_walk_kernel<DP, GROUPS><<<grid, 128 * GROUPS, Walk<DP, GROUPS>::bytes, s>>>(st, a, sl);
  PACE_LAUNCH_CHECK("gla_walk_kernel");
  return PACE_OK;
}

template <int DP>
int launch_chunked(const pace_step_t& st, const pace_gla_args_t& a, const Plan& p, cudaStream_t s) {
  PACE_CUDA_TRY(cudaFuncSetAttribute(gla_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Prep<DP>::bytes));
  const int chunks = (st.max_count + kChunk - 1) / kChunk;
  // few sequences and heads: narrow columns, so that more SMs take part
  const bool narrow = (int64_t)st.n_entries * a.heads * ((a.vdim + 31) / 32) <= 148;
  for (int c = 0; c < chunks; c += p.slab) {
    Slab sl;
    sl.scratch = static_cast<unsigned char*>(a.workspace);
    sl.first = c;
    sl.n = p.slab;
    const int n = chunks - c < p.slab ? chunks - c : p.slab;
    gla_prepare_kernel<DP><<<dim3((unsigned)n, (unsigned)a.heads, (unsigned)st.n_entries), kThreads, Prep<DP>::bytes, s>>>(st, a, sl);
    PACE_LAUNCH_CHECK("gla_prepare_kernel");
    const int rc = narrow ? launch_walk<DP, 1>(st, a, sl, s) : launch_walk<DP, 2>(st, a, sl, s);
    if (rc != PACE_OK) return rc;
  }
  return PACE_OK;
}

}  // namespace

// bf16, key sizes that the tiles cover and 16-byte pieces; everything else is the token-by-token kernel's
bool gla_chunked_fits(const pace_gla_args_t& a) {
  return a.dtype == PACE_DTYPE_BF16 && a.dim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.qkv_stride % 8 == 0 && a.z_stride % 8 == 0 &&
         a.out_stride % 2 == 0 && aligned16(a.qkv) && aligned16(a.z) && ((uintptr_t)a.out & 3) == 0;
}

int gla_chunked(const pace_step_t& st, const pace_gla_args_t& a, cudaStream_t s) {
  const Plan p = plan_chunks(st.n_entries, st.max_count, a.heads, a.dim);
  if (!a.workspace || a.workspace_bytes < p.bytes || !aligned16(a.workspace)) return PACE_ERR_INVALID;
  return p.dp == 64 ? launch_chunked<64>(st, a, p, s) : launch_chunked<128>(st, a, p, s);
}

}  // namespace pace

extern "C" uint64_t pace_gla_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t dim, int32_t dtype) {
  if (n_entries <= 0 || max_count <= 0 || heads <= 0 || dim <= 0 || dim > 128 || dtype != PACE_DTYPE_BF16) return 0;
  return pace::plan_chunks(n_entries, max_count, heads, dim).bytes;
}
