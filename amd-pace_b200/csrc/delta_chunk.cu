// Gated delta rule with a decay per key channel over many tokens, in chunks of 64 on the tensor cores.
//
// With G_i the sum of the chunk's log decays up to token i (a vector over the key channels), x^(G) for the elementwise product with
// e^G, and S the state in front of the chunk, the corrections u and the outputs of a chunk are
//     A_ij = k_i . (k_j)^(G_i - G_j)  (j < i),   P_ij = q_i . (k_j)^(G_i - G_j)  (j <= i),   T = (1 + diag(beta) A)^-1 diag(beta)
//     U = T V - (T K^(G)) S,     O = Q^(G) S + P U,     S' = S^(G_n) + (K^(G_n - G))^T U
// Nothing but S connects the chunks, so a first launch makes everything else side by side, a block per (chunk, head, entry):
// W = T K^(G), T V, Q^(G), K^(G_n - G) and P; a second one walks the chunks, a block per (entry, head, 16 or 32 value columns)
// with its part of S in fp32 accumulators.
//
// e^(G_i - G_j) is the product of a row's factor e^(G_i - M) and a column's e^(M - G_j), M the sum up to the middle of the column's
// sixteen tokens: both are finite as long as eight tokens decay by less than e^60.  Sixteen columns with a channel beyond
// that take M behind them (both factors are then at most 1 for the rows further down) and their own 16 x 16 block pair by pair.
//
// q, k, v are bf16 values; everything else is fp32: where an fp32 quantity is the operand of a bf16 product it is split into two
// bf16 terms, of whose four products the three that matter are taken (16 bits); T is made in fp32 on the CUDA cores.
#include "chunk_mma.cuh"
#include "delta.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64, kThreads = 512, kLP = kChunk + 8, kTP = kChunk + 8;
constexpr float kRange = 86.0f;   // log2 units eight tokens may decay by on the fast path: e^60

// What the first launch leaves of a (entry, chunk, head), as it lies in shared memory later: bf16 tiles of 64 rows of QP (high,
// low halves), P 64 rows of kTP, then fp32.
template <int DP>
struct Slot {
  static constexpr int QP = DP + 8, kTile = kChunk * QP;
  static constexpr int kW = 0, kQ = 2 * kTile, kK = 4 * kTile, kP = 6 * kTile, kHalves = kP + 2 * kChunk * kTP;
  static constexpr size_t kDecay = (size_t)kHalves * 2;               // bytes: [DP] decays over the whole chunk
  static constexpr size_t kUv = kDecay + DP * 4;                      // [vdim][64] the columns of T V
  static __host__ __device__ size_t bytes(int vdim) { return kUv + (size_t)kChunk * vdim * 4; }
};

struct Slab {
  unsigned char* scratch;
  int first, n;    // chunks [first, first + n) of every entry
};

template <int DP>
struct Prep {
  static constexpr int QP = DP + 8, GP = DP + 8;
  static constexpr int kVMost = 128, VP = kVMost + 8;            // value columns that pass through shared memory
  static_assert(VP >= QP, "the columns' high half fits where V will be");
  static constexpr int kK = 0, kQ = kK + kChunk * QP * 2, kG = kQ + kChunk * QP * 2, kL = kG + kChunk * GP * 4,
                       kV = kL + kChunk * kLP * 4, kVec = kV + kChunk * VP * 2, bytes = kVec + (3 * kChunk + 4) * 4;
  static_assert(kChunk * kLP * 4 >= 2 * kChunk * kTP * 2, "the halves of T take the place of L");
};

template <int DP>
__global__ void __launch_bounds__(kThreads, 2) delta_prepare_kernel(pace_step_t st, pace_delta_args_t a, Slab sl) {
  using SL = Slot<DP>;
  using PR = Prep<DP>;
  constexpr int QP = PR::QP, GP = PR::GP;
  const int e = blockIdx.z, h = blockIdx.y, d = a.dim, vd = a.vdim, H = a.heads, KV = a.kv_heads, kh = h / (H / KV);
  const int count = st.cu[e + 1] - st.cu[e], l0 = (sl.first + (int)blockIdx.x) * kChunk;
  if (l0 >= count) return;
  const int n_tok = min(kChunk, count - l0), t0 = st.cu[e] + l0;
  extern __shared__ __align__(16) unsigned char sm[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(sm + PR::kK);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(sm + PR::kQ);
  float* G = reinterpret_cast<float*>(sm + PR::kG);      // sums of log decays, log2 units
  float* L = reinterpret_cast<float*>(sm + PR::kL);      // diag(beta) A, then (1 + L)^-1 in its place
  __nv_bfloat16* t_hi = reinterpret_cast<__nv_bfloat16*>(sm + PR::kL);   // at the end, in L's place
  __nv_bfloat16* t_lo = t_hi + kChunk * kTP;
  __nv_bfloat16* vs = reinterpret_cast<__nv_bfloat16*>(sm + PR::kV);
  float* fk = reinterpret_cast<float*>(sm + PR::kVec);
  float* fq = fk + kChunk;
  float* beta = fq + kChunk;
  int* slow = reinterpret_cast<int*>(beta + kChunk);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  unsigned char* slot = sl.scratch + (((size_t)e * sl.n + blockIdx.x) * H + h) * SL::bytes(vd);
  __nv_bfloat16* tiles = reinterpret_cast<__nv_bfloat16*>(slot);

  // ---- operands: keys and queries as they are, log decays, unit factors ----
  const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(a.qkv) + (size_t)t0 * a.qkv_stride;
  for (int i = tid; i < kChunk * (DP / 8) * 2; i += kThreads) {
    const int which = i / (kChunk * (DP / 8)), r = i - which * (kChunk * (DP / 8)), j = r / (DP / 8), c = (r - j * (DP / 8)) * 8;
    const bool live = j < n_tok && c < d;
    copy16((which ? ks : qs) + j * QP + c, qkv + (live ? (size_t)j * a.qkv_stride + (size_t)(which * KV + kh) * d + c : 0), live);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (tid < 4) slow[tid] = 0;
  if (tid < kChunk)
    beta[tid] = tid < n_tok ? sigmoid_t<__nv_bfloat16>(
        __bfloat162float(static_cast<const __nv_bfloat16*>(a.b_raw)[(size_t)(t0 + tid) * a.b_stride + h])) : 0.f;
  {
    // a thread has eight channels of every (kThreads / (DP / 8))-th token
    const int c = tid % (DP / 8) * 8, j0 = tid / (DP / 8);
    const uint64_t neg_a = both(a.neg_a[h] * kLog2e);
    const __nv_bfloat16* ar = static_cast<const __nv_bfloat16*>(a.a_raw) + (size_t)t0 * a.a_stride + (size_t)h * d + c;
    float bias[8];
#pragma unroll
    for (int x = 0; x < 8; ++x) bias[x] = c < d ? a.dt_bias[(size_t)h * d + c + x] : 0.f;
#pragma unroll
    for (int j = j0; j < kChunk; j += kThreads / (DP / 8)) {
      uint64_t v[4] = {0ull, 0ull, 0ull, 0ull};
      if (j < n_tok && c < d) {
        float x[8];
        Vec<__nv_bfloat16, 8>::load(ar + (size_t)j * a.a_stride, x);
#pragma unroll
        for (int u = 0; u < 4; ++u) v[u] = fma2(softplus2(x[2 * u] + bias[2 * u], x[2 * u + 1] + bias[2 * u + 1]), neg_a, 0ull);
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
  {
    const int j = tid >> 3;                                // eight threads a token
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int c = (tid & 7) * 8; c < DP; c += 64) {
      float x[8], y[8];
      Vec<__nv_bfloat16, 8>::load(qs + j * QP + c, x);
      Vec<__nv_bfloat16, 8>::load(ks + j * QP + c, y);
#pragma unroll
      for (int u = 0; u < 8; ++u) sq = fmaf(x[u], x[u], sq), sk = fmaf(y[u], y[u], sk);
    }
#pragma unroll
    for (int o = 4; o; o >>= 1) {
      sq += __shfl_xor_sync(0xffffffffu, sq, o);
      sk += __shfl_xor_sync(0xffffffffu, sk, o);
    }
    if ((tid & 7) == 0) {
      fq[j] = a.q_scale / sqrtf(sq + a.unit_eps);
      fk[j] = 1.0f / sqrtf(sk + a.unit_eps);
    }
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
  // ---- columns: the keys with their factors, in two halves, where V and L will be ----
  __nv_bfloat16 *kc_hi = vs, *kc_lo = t_hi;
  for (int i = tid; i < kChunk * (DP / 4); i += kThreads) {
    const int j = i / (DP / 4), c = (i - j * (DP / 4)) * 4, b = j >> 4, ref = 16 * b + (slow[b] ? 15 : 7);
    const float4 gg = *reinterpret_cast<const float4*>(G + j * GP + c), m = *reinterpret_cast<const float4*>(G + ref * GP + c);
    float kk[4];
    Vec<__nv_bfloat16, 4>::load(ks + j * QP + c, kk);
    uint2 hi, lo;
    split_bf2(kk[0] * fast_exp2(m.x - gg.x), kk[1] * fast_exp2(m.y - gg.y), hi.x, lo.x);
    split_bf2(kk[2] * fast_exp2(m.z - gg.z), kk[3] * fast_exp2(m.w - gg.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(kc_hi + j * QP + c) = hi;
    *reinterpret_cast<uint2*>(kc_lo + j * QP + c) = lo;
  }
  __syncthreads();

  // ---- scores: warp (keys or queries as rows, one or two of the ten 16 x 16 blocks) ----
  {
    const bool is_q = warp >= 8;
    const __nv_bfloat16* rows = is_q ? qs : ks;
    // (row block, column block) of a warp's first and second task; -1: none
    constexpr int kRow[2][8] = {{0, 1, 1, 2, 2, 2, 3, 3}, {3, 3, -1, -1, -1, -1, -1, -1}};
    constexpr int kCol[2][8] = {{0, 0, 1, 0, 1, 2, 0, 1}, {2, 3, -1, -1, -1, -1, -1, -1}};
    float acc[2][2][4];
    const int w8 = warp & 7;
#pragma unroll
    for (int task = 0; task < 2; ++task) {
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[task][s][x] = 0.f;
      int rb = -1, cb = -1;
#pragma unroll
      for (int w = 0; w < 8; ++w)
        if (w8 == w) rb = kRow[task][w], cb = kCol[task][w];
      if (rb < 0 || (rb == cb && slow[cb])) continue;
      const int i0 = 16 * rb + g, ref = 16 * cb + (slow[cb] ? 15 : 7);
      const __nv_bfloat16* cols = kc_hi + (16 * cb + (lane & 7) + (lane >> 4) * 8) * QP + ((lane >> 3) & 1) * 8;   // two tiles of 8 columns
      const int low = (int)(kc_lo - kc_hi);
#pragma unroll 2
      for (int k0 = 0; k0 < DP; k0 += 16) {
        const int c0 = k0 + 2 * t;
        uint32_t ah[4], al[4], bh[4], bl[4];
        ldsm4(bh, cols + k0);
        ldsm4(bl, cols + low + k0);
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int row = i0 + (x & 1) * 8, c = c0 + (x >> 1) * 8;
          const float2 gg = *reinterpret_cast<const float2*>(G + row * GP + c), m = *reinterpret_cast<const float2*>(G + ref * GP + c);
          const float2 v = bf2_to_f2(*reinterpret_cast<const uint32_t*>(rows + row * QP + c));
          split_bf2(v.x * fast_exp2(gg.x - m.x), v.y * fast_exp2(gg.y - m.y), ah[x], al[x]);
        }
        mma_split(acc[task][0], ah, al, bh, bl);
        mma_split(acc[task][1], ah, al, bh + 2, bl + 2);
      }
    }
    __syncthreads();                                           // the columns have been read: L takes the place of a half
    for (int i = tid; i < kChunk * kLP / 4; i += kThreads) reinterpret_cast<float4*>(L)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
    __nv_bfloat16 *p_hi = tiles + SL::kP, *p_lo = p_hi + kChunk * kTP;
#pragma unroll
    for (int task = 0; task < 2; ++task) {
      int rb = -1, cb = -1;
#pragma unroll
      for (int w = 0; w < 8; ++w)
        if (w8 == w) rb = kRow[task][w], cb = kCol[task][w];
      if (rb < 0 || (rb == cb && slow[cb])) continue;
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int i = 16 * rb + g + 8 * x, j = 16 * cb + 8 * s + 2 * t;
          const float f = is_q ? fq[i] : beta[i] * fk[i], y0 = acc[task][s][2 * x] * f * fk[j], y1 = acc[task][s][2 * x + 1] * f * fk[j + 1];
          if (is_q) {
            uint32_t hi, lo;
            split_bf2(j <= i ? y0 : 0.f, j + 1 <= i ? y1 : 0.f, hi, lo);
            *reinterpret_cast<uint32_t*>(p_hi + i * kTP + j) = hi;
            *reinterpret_cast<uint32_t*>(p_lo + i * kTP + j) = lo;
          } else {
            *reinterpret_cast<float2*>(L + i * kLP + j) = make_float2(j < i ? y0 : 0.f, j + 1 < i ? y1 : 0.f);
          }
        }
    }
  }
  const bool v_here = vd <= PR::kVMost;                        // (needed at the end: on their way while T is made)
  if (v_here) {
    const int pieces = (vd + 15) / 16 * 2;                     // 16 bytes each, whole items of 16 columns
    for (int i = tid; i < kChunk * pieces; i += kThreads) {
      const int j = i / pieces, c = (i - j * pieces) * 8;
      const bool live = j < n_tok && c < vd;
      copy16(vs + j * PR::VP + c, qkv + (live ? (size_t)j * a.qkv_stride + 2 * (size_t)KV * d + (size_t)h * vd + c : 0), live);
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int b = 0; b < 4; ++b) {
    if (!slow[b] || tid >= 256) continue;
    __nv_bfloat16 *p_hi = tiles + SL::kP, *p_lo = p_hi + kChunk * kTP;
    const int i = 16 * b + tid / 16, j = 16 * b + tid % 16;   // one pair per thread
    float sk = 0.f, sq = 0.f;
    if (j <= i) {
      for (int c = 0; c < DP; ++c) {
        const float f = fast_exp2(G[i * GP + c] - G[j * GP + c]) * __bfloat162float(ks[j * QP + c]);
        sk = fmaf(__bfloat162float(ks[i * QP + c]), f, sk);
        sq = fmaf(__bfloat162float(qs[i * QP + c]), f, sq);
      }
    }
    L[i * kLP + j] = j < i ? sk * beta[i] * fk[i] * fk[j] : 0.f;
    const float p = sq * fq[i] * fk[j];
    const __nv_bfloat16 hi = __float2bfloat16_rn(p);
    p_hi[i * kTP + j] = hi;
    p_lo[i * kTP + j] = __float2bfloat16_rn(p - __bfloat162float(hi));
  }
  __syncthreads();
  // ---- queries and keys with their decays; the halves of K^(G) take the places of the keys and the queries ----
  for (int i = tid; i < kChunk * (DP / 2); i += kThreads) {
    const int j = i / (DP / 2), c = (i - j * (DP / 2)) * 2;
    const float2 gg = *reinterpret_cast<const float2*>(G + j * GP + c), ge = *reinterpret_cast<const float2*>(G + (kChunk - 1) * GP + c);
    uint32_t* kp = reinterpret_cast<uint32_t*>(ks + j * QP + c);
    uint32_t* qp = reinterpret_cast<uint32_t*>(qs + j * QP + c);
    const float2 kk = bf2_to_f2(*kp), qq = bf2_to_f2(*qp);
    const float e0 = fast_exp2(gg.x), e1 = fast_exp2(gg.y), k0 = kk.x * fk[j], k1 = kk.y * fk[j], f = fq[j];
    uint32_t hi, lo;
    split_bf2(qq.x * f * e0, qq.y * f * e1, hi, lo);
    *reinterpret_cast<uint32_t*>(tiles + SL::kQ + j * QP + c) = hi;
    *reinterpret_cast<uint32_t*>(tiles + SL::kQ + SL::kTile + j * QP + c) = lo;
    split_bf2(k0 * fast_exp2(ge.x - gg.x), k1 * fast_exp2(ge.y - gg.y), hi, lo);
    *reinterpret_cast<uint32_t*>(tiles + SL::kK + j * QP + c) = hi;
    *reinterpret_cast<uint32_t*>(tiles + SL::kK + SL::kTile + j * QP + c) = lo;
    split_bf2(k0 * e0, k1 * e1, hi, lo);
    *kp = hi;
    *qp = lo;
  }
  if (tid < DP) reinterpret_cast<float*>(slot + SL::kDecay)[tid] = fast_exp2(G[(kChunk - 1) * GP + tid]);

  // ---- (1 + L)^-1 in place of L: blocks of 16, then of 32, then of 64 ----
  {
    const int b = (tid >> 4) & 3, col = tid & 15;
    float x[16];
    if (tid < 64) {
#pragma unroll
      for (int i = 0; i < 16; ++i) x[i] = i == col ? 1.f : 0.f;
      const float* Lb = L + 16 * b * kLP + 16 * b;
#pragma unroll
      for (int j = 0; j < 15; ++j)
#pragma unroll
        for (int i = j + 1; i < 16; ++i) x[i] = fmaf(-Lb[i * kLP + j], x[j], x[i]);
    }
    __syncthreads();
    if (tid < 64) {
#pragma unroll
      for (int i = 0; i < 16; ++i) L[(16 * b + i) * kLP + 16 * b + col] = x[i];
    }
    __syncthreads();
    // lower left block of a pair: -T_bb (L_ba T_aa); a thread's outputs lie in one column of one pair
    auto combine = [&](auto size_c) {
      constexpr int N = decltype(size_c)::value, PAIRS = kChunk / (2 * N), PER = PAIRS * N * N / kThreads, RS = kThreads / (PAIRS * N);
      const int pr = tid / (kThreads / PAIRS), at = 2 * N * pr, j = tid % N, i0 = tid % (kThreads / PAIRS) / N;
#pragma unroll
      for (int step = 0; step < 2; ++step) {
        const float* rows = L + (at + N + i0) * kLP + at + (step ? N : 0);            // of L_ba, then of T_bb
        const float* cols = L + (at + (step ? N : 0)) * kLP + at + j;                 // of T_aa, then of the product
        float y[PER];
#pragma unroll
        for (int k = 0; k < PER; ++k) y[k] = 0.f;
#pragma unroll
        for (int x = 0; x < N; x += 4) {
          float c[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) c[u] = cols[(x + u) * kLP];
#pragma unroll
          for (int k = 0; k < PER; ++k) {
            const float4 r = *reinterpret_cast<const float4*>(rows + k * RS * kLP + x);
            y[k] = fmaf(r.x, c[0], fmaf(r.y, c[1], fmaf(r.z, c[2], fmaf(r.w, c[3], y[k]))));
          }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < PER; ++k) L[(at + N + i0 + k * RS) * kLP + at + j] = step ? -y[k] : y[k];
        __syncthreads();
      }
    };
    combine(std::integral_constant<int, 16>());
    combine(std::integral_constant<int, 32>());
  }
  {
    uint32_t hi[kChunk * kChunk / 2 / kThreads], lo[kChunk * kChunk / 2 / kThreads];
#pragma unroll
    for (int k = 0; k < kChunk * kChunk / 2 / kThreads; ++k) {
      const int i = k * kThreads + tid, r = i / (kChunk / 2), c = (i - r * (kChunk / 2)) * 2;
      split_bf2(L[r * kLP + c] * beta[c], L[r * kLP + c + 1] * beta[c + 1], hi[k], lo[k]);
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kChunk * kChunk / 2 / kThreads; ++k) {
      const int i = k * kThreads + tid, r = i / (kChunk / 2), c = (i - r * (kChunk / 2)) * 2;
      *reinterpret_cast<uint32_t*>(t_hi + r * kTP + c) = hi[k];
      *reinterpret_cast<uint32_t*>(t_lo + r * kTP + c) = lo[k];
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  // ---- T K^(G) and T V, 16 columns at a time ----
  const int w_items = DP / 16, items = w_items + (vd + 15) / 16;
  for (int it = warp; it < items; it += kThreads / 32) {
    const bool is_w = it < w_items;
    const int n0 = (is_w ? it : it - w_items) * 16;
    float acc[4][2][4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[m][s][x] = 0.f;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t bh[4], bl[4];
      if (is_w) {
        ldsm4t(bh, ks + (16 * kt + (lane & 15)) * QP + n0 + (lane >> 4) * 8);
        ldsm4t(bl, qs + (16 * kt + (lane & 15)) * QP + n0 + (lane >> 4) * 8);
      } else if (v_here) {
        ldsm4t(bh, vs + (16 * kt + (lane & 15)) * PR::VP + n0 + (lane >> 4) * 8);
      } else {
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int c = n0 + 8 * (x >> 1) + g, j = 16 * kt + 2 * t + 8 * (x & 1);
          const unsigned short* v = reinterpret_cast<const unsigned short*>(qkv) + (size_t)j * a.qkv_stride + 2 * (size_t)KV * d + (size_t)h * vd + c;
          const uint32_t lo16 = j < n_tok && c < vd ? v[0] : 0, hi16 = j + 1 < n_tok && c < vd ? v[a.qkv_stride] : 0;
          bh[x] = lo16 | (hi16 << 16);
        }
      }
#pragma unroll
      for (int m = kt; m < 4; ++m) {
        uint32_t ah[4], al[4];
        ldsm4(ah, t_hi + (16 * m + (lane & 15)) * kTP + 16 * kt + (lane >> 4) * 8);
        ldsm4(al, t_lo + (16 * m + (lane & 15)) * kTP + 16 * kt + (lane >> 4) * 8);
#pragma unroll
        for (int s = 0; s < 2; ++s) {
          mma16816(acc[m][s], ah, bh[2 * s], bh[2 * s + 1]);
          mma16816(acc[m][s], al, bh[2 * s], bh[2 * s + 1]);
          if (is_w) mma16816(acc[m][s], ah, bl[2 * s], bl[2 * s + 1]);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int i = 16 * m + g + 8 * x, c = n0 + 8 * s + 2 * t;
          if (is_w) {
            uint32_t hi, lo;
            split_bf2(acc[m][s][2 * x], acc[m][s][2 * x + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(tiles + SL::kW + i * QP + c) = hi;
            *reinterpret_cast<uint32_t*>(tiles + SL::kW + SL::kTile + i * QP + c) = lo;
          } else if (c < vd) {
            float* uv = reinterpret_cast<float*>(slot + SL::kUv) + (size_t)c * kChunk + i;
            uv[0] = acc[m][s][2 * x];
            uv[kChunk] = acc[m][s][2 * x + 1];
          }
        }
  }
}

// The walk over the chunks, transposed: four warps own 16 value columns, each a quarter of the key channels.  The accumulators of
// S^T (16 columns x DQ channels) are, split in two terms, the row operand of S^T W^T and S^T Q^T as they are, and those of U^T that
// of U^T K and U^T P^T; the chunk's tiles are the other operand.  What the four warps have of W S and of the outputs meets in shared
// memory in fragment form: warp q sums up tokens 16 q .. 16 q + 15 and hands the corrections to the others.
template <int DP, int GROUPS>
struct Walk {
  static constexpr int kTiles = Slot<DP>::kHalves * 2, kExchange = 4 * 4 * 2 * 32 * 16, kU = 4 * 2 * 32 * 16;   // bytes
  static constexpr int bytes = kTiles + GROUPS * (2 * kExchange + kU);
};

template <int DP, int GROUPS>
__global__ void __launch_bounds__(128 * GROUPS, 1) delta_walk_kernel(pace_step_t st, pace_delta_args_t a, Slab sl) {
  using SL = Slot<DP>;
  using WK = Walk<DP, GROUPS>;
  constexpr int QP = SL::QP, DQ = DP / 4, KS = DQ / 16, ND = DQ / 8, THREADS = 128 * GROUPS;
  const int e = blockIdx.z, h = blockIdx.y, d = a.dim, vd = a.vdim, H = a.heads;
  const int count = st.cu[e + 1] - st.cu[e], chunks = min(sl.n, (count + kChunk - 1) / kChunk - sl.first);
  if (chunks <= 0) return;
  extern __shared__ __align__(16) unsigned char sm[];
  const __nv_bfloat16* tiles = reinterpret_cast<const __nv_bfloat16*>(sm);
  const int tid = threadIdx.x, lane = tid & 31, group = tid >> 7, q = (tid >> 5) & 3, g = lane >> 2, t = lane & 3;
  float4* xw = reinterpret_cast<float4*>(sm + WK::kTiles + group * (2 * WK::kExchange + WK::kU));   // [warp][quarter][half][lane]
  float4* xo = xw + WK::kExchange / 16;
  uint4* uf = reinterpret_cast<uint4*>(xo + WK::kExchange / 16);                                    // [quarter][high, low][lane]
  const int v0 = (blockIdx.x * GROUPS + group) * 16, c0 = q * DQ;
  const size_t slot_bytes = SL::bytes(vd);
  const unsigned char* slot = sl.scratch + ((size_t)e * sl.n * H + h) * slot_bytes;
  auto fetch = [&](const unsigned char* from, int begin, int end) {   // bytes of a slot, to their places
#pragma unroll 8
    for (int i = begin + tid * 16; i < end; i += THREADS * 16) copy16(sm + i, from + i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(slot, 0, SL::kK * 2);
  fetch(slot, SL::kK * 2, WK::kTiles);
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
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  for (int c = 0; c < chunks; ++c, slot += (size_t)H * slot_bytes) {
    const int l0 = (sl.first + c) * kChunk, n_tok = min(kChunk, count - l0);
    const float2* decay = reinterpret_cast<const float2*>(slot + SL::kDecay) + (c0 >> 1) + t;
    const float* uvp = reinterpret_cast<const float*>(slot + SL::kUv) + (size_t)(v0 + g) * kChunk + 16 * q + 2 * t;
    float2 dec[ND], uv[2][2];
#pragma unroll
    for (int n = 0; n < ND; ++n) dec[n] = decay[4 * n];
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      uv[hf][0] = in0 ? *reinterpret_cast<const float2*>(uvp + 8 * hf) : make_float2(0.f, 0.f);
      uv[hf][1] = in1 ? *reinterpret_cast<const float2*>(uvp + 8 * kChunk + 8 * hf) : make_float2(0.f, 0.f);
    }
    uint32_t sh[KS][4], so[KS][4];
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int x = 0; x < 4; ++x) split_bf2(S[2 * k + (x >> 1)][2 * (x & 1)], S[2 * k + (x >> 1)][2 * (x & 1) + 1], sh[k][x], so[k][x]);
    // (16 columns) x (64 tokens): S^T times a tile, this warp's channels
    float D[8][4];
    auto answer = [&](int tile) {
#pragma unroll
      for (int n = 0; n < 8; ++n) D[n][0] = D[n][1] = D[n][2] = D[n][3] = 0.f;
#pragma unroll
      for (int n4 = 0; n4 < 8; n4 += 4) {
        uint32_t bh[4][4], bl[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          const __nv_bfloat16* p = tiles + tile + (8 * (n4 + n) + (lane & 7)) * QP + c0;
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
    };
    auto put = [&](float4* x) {
#pragma unroll
      for (int n = 0; n < 8; ++n) x[(q * 8 + n) * 32 + lane] = make_float4(D[n][0], D[n][1], D[n][2], D[n][3]);
    };
    auto sum = [&](const float4* x, int hf) {
      float4 s = x[(2 * q + hf) * 32 + lane];
#pragma unroll
      for (int w = 1; w < 4; ++w) {
        const float4 v = x[(w * 8 + 2 * q + hf) * 32 + lane];
        s.x += v.x, s.y += v.y, s.z += v.z, s.w += v.w;
      }
      return s;
    };
    answer(SL::kW);
    put(xw);
    answer(SL::kQ);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                           // W S is there, and K and P; W and Q have been read
    if (c + 1 < chunks) fetch(slot + (size_t)H * slot_bytes, 0, SL::kK * 2);
    uint32_t mh[4], ml[4];                                     // corrections of tokens 16 q .. + 15
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const float4 s = sum(xw, hf);
      split_bf2(uv[hf][0].x - s.x, uv[hf][0].y - s.y, mh[2 * hf], ml[2 * hf]);
      split_bf2(uv[hf][1].x - s.z, uv[hf][1].y - s.w, mh[2 * hf + 1], ml[2 * hf + 1]);
    }
    uf[(2 * q) * 32 + lane] = make_uint4(mh[0], mh[1], mh[2], mh[3]);
    uf[(2 * q + 1) * 32 + lane] = make_uint4(ml[0], ml[1], ml[2], ml[3]);
    // the outputs' share of these tokens' corrections
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      if (n < 2 * q) continue;
      uint32_t b[4];      // matrices 0, 1 high, 2, 3 low
      ldsm4(b, tiles + SL::kP + (lane >> 4) * kChunk * kTP + (8 * n + (lane & 7)) * kTP + 16 * q + ((lane >> 3) & 1) * 8);
      mma16816(D[n], mh, b[0], b[1]);
      mma16816(D[n], mh, b[2], b[3]);
      mma16816(D[n], ml, b[0], b[1]);
    }
    put(xo);
    __syncthreads();                                           // the corrections are there, and the outputs
    float Z[ND][4];                                            // cross terms
#pragma unroll
    for (int n = 0; n < ND; ++n) {
      S[n][0] *= dec[n].x; S[n][1] *= dec[n].y;
      S[n][2] *= dec[n].x; S[n][3] *= dec[n].y;
      Z[n][0] = Z[n][1] = Z[n][2] = Z[n][3] = 0.f;
    }
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      const uint4 h4 = uf[(2 * kt) * 32 + lane], l4 = uf[(2 * kt + 1) * 32 + lane];
      const uint32_t ah[4] = {h4.x, h4.y, h4.z, h4.w}, al[4] = {l4.x, l4.y, l4.z, l4.w};
      const __nv_bfloat16* p = tiles + SL::kK + (16 * kt + (lane & 15)) * QP + c0 + (lane >> 4) * 8;
#pragma unroll
      for (int n = 0; n < ND; n += 2) {
        uint32_t bh[4], bl[4];
        ldsm4t(bh, p + 8 * n);
        ldsm4t(bl, p + SL::kTile + 8 * n);
        mma16816(S[n], ah, bh[0], bh[1]);
        mma16816(S[n + 1], ah, bh[2], bh[3]);
        mma16816(Z[n], ah, bl[0], bl[1]);
        mma16816(Z[n + 1], ah, bl[2], bl[3]);
        mma16816(Z[n], al, bh[0], bh[1]);
        mma16816(Z[n + 1], al, bh[2], bh[3]);
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
      const float4 s = sum(xo, hf);
      const bool odd = g & 1;
      const float g0 = __shfl_xor_sync(0xffffffffu, odd ? s.x : s.y, 4), g1 = __shfl_xor_sync(0xffffffffu, odd ? s.z : s.w, 4);
      const int tok = 16 * q + 8 * hf + 2 * t + (odd ? 1 : 0), col = g & ~1;
      if (tok < n_tok) {
        if (v0 + col < vd) *reinterpret_cast<uint32_t*>(out + (size_t)tok * a.out_stride + col) = odd ? f2_to_bf2(g0, s.y) : f2_to_bf2(s.x, g0);
        if (v0 + col + 8 < vd) *reinterpret_cast<uint32_t*>(out + (size_t)tok * a.out_stride + col + 8) = odd ? f2_to_bf2(g1, s.w) : f2_to_bf2(s.z, g1);
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                           // the next W and Q are there; K and P have been read
    if (c + 1 < chunks) fetch(slot + (size_t)H * slot_bytes, SL::kK * 2, WK::kTiles);
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
Plan plan_chunks(int n_entries, int max_count, int heads, int dim, int vdim) {
  Plan p;
  p.dp = dim <= 64 ? 64 : 128;
  const uint64_t slot = p.dp == 64 ? Slot<64>::bytes(vdim) : Slot<128>::bytes(vdim), row = slot * heads * n_entries;
  const int chunks = (max_count + kChunk - 1) / kChunk;
  const uint64_t fit = kBudget / row;
  p.slab = fit < 1 ? 1 : fit < (uint64_t)chunks ? (int)fit : chunks;
  p.bytes = row * p.slab;
  return p;
}

template <int DP, int GROUPS>
int launch_walk(const pace_step_t& st, const pace_delta_args_t& a, const Slab& sl, cudaStream_t s) {
  PACE_CUDA_TRY(cudaFuncSetAttribute(delta_walk_kernel<DP, GROUPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Walk<DP, GROUPS>::bytes));
  const dim3 grid((unsigned)((a.vdim + 16 * GROUPS - 1) / (16 * GROUPS)), (unsigned)a.heads, (unsigned)st.n_entries);
  delta_walk_kernel<DP, GROUPS><<<grid, 128 * GROUPS, Walk<DP, GROUPS>::bytes, s>>>(st, a, sl);
  PACE_LAUNCH_CHECK("delta_walk_kernel");
  return PACE_OK;
}

template <int DP>
int launch_chunked(const pace_step_t& st, const pace_delta_args_t& a, const Plan& p, cudaStream_t s) {
  PACE_CUDA_TRY(cudaFuncSetAttribute(delta_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Prep<DP>::bytes));
  const int chunks = (st.max_count + kChunk - 1) / kChunk;
  // few sequences and heads: narrow columns, so that more SMs take part
  const bool narrow = (int64_t)st.n_entries * a.heads * ((a.vdim + 31) / 32) <= 74;
  for (int c = 0; c < chunks; c += p.slab) {
    Slab sl;
    sl.scratch = static_cast<unsigned char*>(a.workspace);
    sl.first = c;
    sl.n = p.slab;
    const int n = chunks - c < p.slab ? chunks - c : p.slab;
    delta_prepare_kernel<DP><<<dim3((unsigned)n, (unsigned)a.heads, (unsigned)st.n_entries), kThreads, Prep<DP>::bytes, s>>>(st, a, sl);
    PACE_LAUNCH_CHECK("delta_prepare_kernel");
    const int rc = narrow ? launch_walk<DP, 1>(st, a, sl, s) : launch_walk<DP, 2>(st, a, sl, s);
    if (rc != PACE_OK) return rc;
  }
  return PACE_OK;
}

}  // namespace

// bf16, key sizes that the tiles cover and 16-byte pieces; everything else is the token-by-token kernel's
bool delta_chunked_fits(const pace_delta_args_t& a) {
  return a.dtype == PACE_DTYPE_BF16 && a.dim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.qkv_stride % 8 == 0 && a.a_stride % 8 == 0 &&
         a.out_stride % 2 == 0 && aligned16(a.qkv) && aligned16(a.a_raw) &&
         ((uintptr_t)a.out & 3) == 0 && ((uintptr_t)a.s_state & 7) == 0;
}

int delta_chunked(const pace_step_t& st, const pace_delta_args_t& a, cudaStream_t s) {
  const Plan p = plan_chunks(st.n_entries, st.max_count, a.heads, a.dim, a.vdim);
  if (!a.workspace || a.workspace_bytes < p.bytes || !aligned16(a.workspace)) return PACE_ERR_INVALID;
  return p.dp == 64 ? launch_chunked<64>(st, a, p, s) : launch_chunked<128>(st, a, p, s);
}

}  // namespace pace

extern "C" uint64_t pace_delta_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t dim, int32_t vdim, int32_t dtype) {
  if (n_entries <= 0 || max_count <= 0 || heads <= 0 || dim <= 0 || vdim <= 0 || dim > 128 || dtype != PACE_DTYPE_BF16) return 0;
  return pace::plan_chunks(n_entries, max_count, heads, dim, vdim).bytes;
}
