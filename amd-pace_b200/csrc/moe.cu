// Mixtures of experts: routing (sigmoid or softmax scores, choice by corrected scores) and the chosen experts'
// feed-forwards, gated or not, as grouped products.
//
// Grouped product on tcgen05 (moe_grouped_kernel): the weights are the 128-row operand, the tokens the columns, so an
// expert with a handful of tokens costs a narrow tile and not a padded one.  A tile is (expert, 2 x 128 weight rows, NT
// tokens): two accumulators that share every token tile - gate and up rows of the same features (gated first product), two
// neighbouring row tiles (everything else).  Persistent blocks of ten warps: TMA producer, MMA issuer, eight epilogue warps;
// two sets of accumulators in tensor memory, so that a tile is stored while the next one is computed.  The first
// product's token rows come through the router's lists: narrow tiles gather them by TMA (tile::gather4), wide ones read
// rows that moe_spread_kernel has copied into expert order (32 gathers per 64 columns would pace a wide tile).  Its results
// are written by expert, and the second product reads them in place.  The tile list is made by every block from the experts' counts: nothing comes
// back to the host.
#include "hybrid.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kMaxExperts = 1024, kMaxTop = 64;

// ---------------------------------------------------------------------------
// routing
// ---------------------------------------------------------------------------
// A warp per token.  A block numbers the tokens of an expert among its own first; one block over all tokens (WHOLE) is
// done with that, several take their place by one atomic per expert.
template <bool WHOLE>
__global__ void moe_route_kernel(pace_moe_route_args_t a, int rounds) {
  extern __shared__ float sh[];
  const int E = a.n_experts, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5, slots = warps * rounds * a.top;
  float* score = sh + warp * 2 * E;
  float* choice = score + E;
  int* cnt = reinterpret_cast<int*>(sh + warps * 2 * E);   // tokens of this block per expert, then the first one's number
  int* sel = cnt + E;                                      // [token of the block][top]: expert and number in the block
  const int t_first = blockIdx.x * warps * rounds;
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int r = 0; r < rounds; ++r) {
    const int local = r * warps + warp, t = t_first + local;
    if (t >= a.n_tokens) break;
    const float* z = a.logits + (size_t)t * E;
    if (a.softmax) {
      float top = -INFINITY, sum = 0.f;
      for (int e = lane; e < E; e += 32) top = fmaxf(top, z[e]);
#pragma unroll
      for (int o = 16; o; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
      for (int e = lane; e < E; e += 32) sum += score[e] = expf(z[e] - top);
#pragma unroll
      for (int o = 16; o; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      for (int e = lane; e < E; e += 32) score[e] /= sum;
    } else {
      for (int e = lane; e < E; e += 32) score[e] = 1.0f / (1.0f + expf(-z[e]));
    }
    for (int e = lane; e < E; e += 32) choice[e] = score[e] + (a.correction ? a.correction[e] : 0.f);
    __syncwarp();
    float chosen = 0.f;
    for (int k = 0; k < a.top; ++k) {
      float best = -INFINITY;
      int at = -1;
      for (int e = lane; e < E; e += 32)
        if (choice[e] > best) best = choice[e], at = e;
#pragma unroll
      for (int o = 16; o; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const int i = __shfl_xor_sync(0xffffffffu, at, o);
        if (i >= 0 && (at < 0 || v > best || (v == best && i < at))) best = v, at = i;
      }
      if (at < 0) at = k;  // (scores that are not numbers: any expert)
      chosen += score[at];
      if (lane == (at & 31)) {
        choice[at] = -INFINITY;
        const size_t s = (size_t)t * a.top + k;
        a.slot_expert[s] = at;
        a.slot_weight[s] = score[at];
        sel[2 * (local * a.top + k)] = at;
        sel[2 * (local * a.top + k) + 1] = atomicAdd(&cnt[at], 1);
      }
    }
    __syncwarp();
    if (a.normalise)
      for (int k = lane; k < a.top; k += 32)
        a.slot_weight[(size_t)t * a.top + k] = score[sel[2 * (local * a.top + k)]] / (chosen + 1e-20f) * a.weight_scale;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int n = cnt[e];
    if (WHOLE) {
      a.expert_count[e] = n;
      cnt[e] = 0;
    } else {
      cnt[e] = n ? atomicAdd(&a.expert_count[e], n) : 0;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < slots; i += blockDim.x) {
    const int t = t_first + i / a.top;
    if (t >= a.n_tokens) break;
    const int e = sel[2 * i], rank = cnt[e] + sel[2 * i + 1];
    a.slot_rank[(size_t)t_first * a.top + i] = rank;
    if (rank < a.n_tokens) a.expert_list[(size_t)e * a.n_tokens + rank] = t;
  }
}
size_t route_smem(int warps, int rounds, int E, int top) { return (size_t)(2 * warps + 1) * E * 4 + (size_t)warps * rounds * top * 8; }

// ---------------------------------------------------------------------------
// experts on the CUDA cores: fp32 models, sizes that are not multiples of 8
// ---------------------------------------------------------------------------
// what row r of the expert-ordered buffers is: its expert, its place among the expert's tokens
__device__ __forceinline__ bool find_row(const int32_t* count, int E, int r, int* expert, int* rank) {
  for (int e = 0; e < E; ++e) {
    const int n = count[e];
    if (r < n) {
      *expert = e;
      *rank = r;
      return true;
    }
    r -= n;
  }
  return false;
}

// a block per row, a warp per output feature at a time
template <typename T, bool FIRST>
__global__ void __launch_bounds__(256) moe_simple_kernel(pace_moe_experts_args_t a) {
  extern __shared__ float xs[];
  __shared__ int who[2];
  const int r = blockIdx.x;
  if (threadIdx.x == 0) {
    int e = -1, k = 0;
    who[0] = find_row(a.expert_count, a.n_experts, r, &e, &k) && k < a.n_tokens ? e : -1;
    who[1] = k;
  }
  __syncthreads();
  const int e = who[0];
  if (e < 0) return;
  const int K = FIRST ? a.width : a.ff, N = FIRST ? a.ff : a.width;
  const bool glu = FIRST && a.gated;
  const T* x;
  if (FIRST) x = static_cast<const T*>(a.x) + (size_t)a.expert_list[(size_t)e * a.n_tokens + who[1]] * K;
  else x = static_cast<const T*>(a.hidden) + (size_t)r * K;
  for (int c = threadIdx.x; c < K; c += blockDim.x) xs[c] = to_f<T>(x[c]);
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int f = threadIdx.x >> 5; f < N; f += blockDim.x >> 5) {
    const T* w0 = FIRST ? static_cast<const T*>(a.gate_up) + ((size_t)e * (glu ? 2 : 1) * N + f) * K
                        : static_cast<const T*>(a.down) + ((size_t)e * N + f) * K;
    const T* w1 = w0 + (size_t)N * K;
    float s0 = 0.f, s1 = 0.f;
    for (int c = lane; c < K; c += 32) {
      s0 = fmaf(to_f<T>(w0[c]), xs[c], s0);
      if (glu) s1 = fmaf(to_f<T>(w1[c]), xs[c], s1);
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) {
      s0 += __shfl_xor_sync(0xffffffffu, s0, o);
      s1 += __shfl_xor_sync(0xffffffffu, s1, o);
    }
    if (lane == 0) {
      const float y = FIRST ? act_t<T>(a.act, s0) * (glu ? s1 : 1.f) : s0;
      (FIRST ? static_cast<T*>(a.hidden) : static_cast<T*>(a.y))[(size_t)r * N + f] = from_f<T>(y);
    }
  }
}

template <typename T>
int experts_simple(const pace_moe_experts_args_t& a, cudaStream_t s) {
  const unsigned rows = (unsigned)(a.n_tokens * a.top);
  const size_t sm0 = (size_t)a.width * 4, sm1 = (size_t)a.ff * 4;
  if (sm0 > 227 * 1024 || sm1 > 227 * 1024) return PACE_ERR_UNSUPPORTED;
  PACE_CUDA_TRY(cudaFuncSetAttribute(moe_simple_kernel<T, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm0));
  PACE_CUDA_TRY(cudaFuncSetAttribute(moe_simple_kernel<T, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm1));
  moe_simple_kernel<T, true><<<rows, 256, sm0, s>>>(a);
  PACE_LAUNCH_CHECK("moe_simple_kernel");
  moe_simple_kernel<T, false><<<rows, 256, sm1, s>>>(a);
  PACE_LAUNCH_CHECK("moe_simple_kernel");
  return PACE_OK;
}

// token rows -> expert order, a block per token: read once, stored once per chosen expert
__global__ void __launch_bounds__(256) moe_spread_kernel(pace_moe_experts_args_t a) {
  __shared__ int row[kMaxTop];
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  for (int k = threadIdx.x >> 5; k < a.top; k += blockDim.x >> 5) {
    const int e = a.slot_expert[(size_t)t * a.top + k];
    int n = 0;
    for (int i = lane; i < e && e < a.n_experts; i += 32) n += a.expert_count[i];
#pragma unroll
    for (int o = 16; o; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
    if (lane == 0) row[k] = e < a.n_experts ? n + a.slot_rank[(size_t)t * a.top + k] : -1;   // -1: an identity expert
  }
  __syncthreads();
  const int pieces = a.width / 8;
  const uint4* src = static_cast<const uint4*>(a.x) + (size_t)t * pieces;
  for (int c = threadIdx.x; c < pieces; c += blockDim.x) {
    const uint4 v = src[c];
    for (int k = 0; k < a.top; ++k)
      if (row[k] >= 0) static_cast<uint4*>(a.scratch)[(size_t)row[k] * pieces + c] = v;
  }
}

// ---------------------------------------------------------------------------
// grouped products on tcgen05
// ---------------------------------------------------------------------------
constexpr int kThreads = 320, kProducerWarp = 8, kIssuerWarp = 9, kKStep = 64;
constexpr int kABytes = 128 * kKStep * 2;

struct GroupedParams {
  const int32_t* count;
  const int32_t* list;
  int32_t* status;
  __nv_bfloat16* out;
  int n_tokens, n_experts, n_rows;   // n_rows: rows of the expert-ordered buffers
  int K, N, a_rows, a_second;        // a_rows: weight rows per expert; a_second: from the first row tile to the second
  int m_tiles, n_stages, act;
};

struct Tile {
  int e, m, row0, first, live;  // row0: first output row, first: place among the expert's tokens, live: tokens
};

template <int NT>
__host__ __device__ constexpr int stage_bytes() { return 2 * kABytes + NT * 128; }

// GLU: act(gate) * up; otherwise act of plain products (second products: none).  GATHER: token rows through the lists, otherwise in expert order.
template <int NT, bool GLU, bool GATHER>
__global__ void __launch_bounds__(kThreads, 1)
    moe_grouped_kernel(const GroupedParams p, const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmB) {
  constexpr int STAGE = stage_bytes<NT>();
  constexpr int COLS = 4 * NT < 32 ? 32 : 4 * NT;  // tensor memory: two sets of two accumulators
  static_assert(COLS == 128 || COLS == 256 || COLS == 512, "a power of two");
  extern __shared__ unsigned char smem_raw[];
  __shared__ uint64_t full[8], empty[8], t_full[2], t_empty[2];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_flag;
  __shared__ int tile_end[kMaxExperts], row_end[kMaxExperts];  // inclusive prefix sums over the experts
  unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  volatile int* abort = &abort_flag;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = p.n_experts, S = p.n_stages;

  if (warp == kIssuerWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(COLS)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (tid == 0) {
    abort_flag = 0;
    for (int i = 0; i < S; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&t_full[i], 1);
      mbar_init(&t_empty[i], 8);
    }
    fence_mbar_init();
  }
  if (warp == 0) {  // prefix sums of tokens and token tiles
    int carry_t = 0, carry_r = 0;
    for (int b = 0; b < E; b += 32) {
      int n = b + lane < E ? p.count[b + lane] : 0, t = (n + NT - 1) / NT;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int un = __shfl_up_sync(0xffffffffu, n, o), ut = __shfl_up_sync(0xffffffffu, t, o);
        if (lane >= o) n += un, t += ut;
      }
      if (b + lane < E) {
        row_end[b + lane] = carry_r + n;
        tile_end[b + lane] = carry_t + t;
      }
      carry_r += __shfl_sync(0xffffffffu, n, 31);
      carry_t += __shfl_sync(0xffffffffu, t, 31);
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&tmem_slot);
  const int n_tiles = tile_end[E - 1] * p.m_tiles;
  // tile number -> expert, row tile, token tile; token tiles of one row tile are neighbours (their weights stay in L2)
  auto tile_of = [&](int i) {
    Tile t;
    int lo = 0, hi = E - 1;
    while (lo < hi) {
      const int mid = (lo + hi) >> 1;
      if (tile_end[mid] * p.m_tiles > i) hi = mid;
      else lo = mid + 1;
    }
    t.e = lo;
    const int before_t = lo ? tile_end[lo - 1] : 0, before_r = lo ? row_end[lo - 1] : 0;
    const int n_t = tile_end[lo] - before_t, r = i - before_t * p.m_tiles;
    t.m = r / n_t;
    t.first = (r - t.m * n_t) * NT;
    t.row0 = before_r + t.first;
    t.live = min(NT, row_end[lo] - t.row0);
    return t;
  };
  const int k_steps = (p.K + kKStep - 1) / kKStep;

  if (warp == kProducerWarp) {
    int s = 0, ph = 0, issued = 0;
    bool ok = true;
    for (int i = blockIdx.x; i < n_tiles && ok; i += gridDim.x) {
      const Tile t = tile_of(i);
      const int a0 = t.e * p.a_rows + t.m * (GLU ? 128 : 256), a1 = a0 + p.a_second;
      int r[4];
      if (GATHER) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int k = 4 * lane + j;
          r[j] = k < t.live && t.first + k < p.n_tokens ? p.list[(size_t)t.e * p.n_tokens + t.first + k] : 0;
        }
      }
      for (int ks = 0; ks < k_steps; ++ks) {
        if (issued >= S && !__all_sync(0xffffffffu, mbar_wait(&empty[s], ph ^ 1, abort))) {
          ok = false;
          break;
        }
        unsigned char* st = ring + (size_t)s * STAGE;
        if (lane == 0) {
          mbar_arrive_expect_tx(&full[s], STAGE);
          tma_load_2d(st, &tmA, ks * kKStep, a0, &full[s]);
          tma_load_2d(st + kABytes, &tmA, ks * kKStep, a1, &full[s]);
          if (!GATHER) tma_load_2d(st + 2 * kABytes, &tmB, ks * kKStep, t.row0, &full[s]);
        }
        __syncwarp();
        if (GATHER && lane < NT / 4) tma_gather4(st + 2 * kABytes + lane * 512, &tmB, ks * kKStep, r[0], r[1], r[2], r[3], &full[s]);
        ++issued;
        if (++s == S) s = 0, ph ^= 1;
      }
    }
    if (!ok) {  // copies in flight land before the block's shared memory is released
      for (int k = issued > S ? issued - S : 0; k < issued; ++k) mbar_wait(&full[k % S], (k / S) & 1);
    }
  } else if (warp == kIssuerWarp) {
    constexpr uint32_t IDESC = umma_idesc(NT, false);
    const bool leader = elect_one();
    int s = 0, ph = 0, n = 0;
    bool ok = true;
    for (int i = blockIdx.x; i < n_tiles && ok; i += gridDim.x, ++n) {
      const int buf = n & 1;
      if (n >= 2 && !umma_issuer_wait(&t_empty[buf], ((n >> 1) - 1) & 1, abort)) break;
      tc_fence_after();
      const uint32_t d0 = tmem + buf * 2 * NT, d1 = d0 + NT;
      for (int ks = 0; ks < k_steps; ++ks) {
        if (!umma_issuer_wait(&full[s], ph, abort)) {
          ok = false;
          break;
        }
        tc_fence_after();
        if (leader) {
          const uint32_t a_lo = (smem_u32(ring + (size_t)s * STAGE) >> 4) | (1u << 16);
          const uint32_t b_lo = a_lo + (2 * kABytes >> 4);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) {
            const uint64_t bd = pack64(b_lo + kk * 2, kDescHi);
            umma_bf16(d0, pack64(a_lo + kk * 2, kDescHi), bd, IDESC, (ks | kk) ? 1u : 0u);
            umma_bf16(d1, pack64(a_lo + (kABytes >> 4) + kk * 2, kDescHi), bd, IDESC, (ks | kk) ? 1u : 0u);
          }
          umma_commit(&empty[s]);
          if (ks == k_steps - 1) umma_commit(&t_full[buf]);
        }
        __syncwarp();
        if (++s == S) s = 0, ph ^= 1;
      }
    }
    // (every product of a whole run is waited for by the epilogue; after an abort those in flight end here)
    if (*abort && leader) {
      umma_commit(&t_full[0]);
      for (int k = 0; k < 4096; ++k) __nanosleep(256);
    }
    __syncwarp();
  } else {
    const int wg = warp >> 2, row = (warp & 3) * 32 + lane;  // tensor-memory lane = weight row of the tile
    const uint32_t t_lane = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    int n = 0;
    for (int i = blockIdx.x; i < n_tiles; i += gridDim.x, ++n) {
      const int buf = n & 1;
      const Tile t = tile_of(i);
      if (!__all_sync(0xffffffffu, mbar_wait(&t_full[buf], (n >> 1) & 1, abort))) break;
      tc_fence_after();
      constexpr int HALF = NT / 2, STEP = HALF < 16 ? HALF : 16;
      static_assert(STEP == 16, "half a tile's columns in pieces of 16");
      const int f0 = t.m * (GLU ? 128 : 256) + row;
#pragma unroll 1
      for (int c0 = wg * HALF; c0 < (wg + 1) * HALF; c0 += STEP) {
        if (c0 >= t.live) break;
        uint32_t x0[16], x1[16];
        tmem_ld16(t_lane + buf * 2 * NT + c0, x0);
        tmem_ld16(t_lane + buf * 2 * NT + NT + c0, x1);
        tmem_wait_ld();
        float v[GLU ? 1 : 2][16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const float u0 = __uint_as_float(x0[j]), u1 = __uint_as_float(x1[j]);
          if constexpr (GLU) {
            v[0][j] = act_t<__nv_bfloat16>(p.act, u0) * u1;
          } else {
            v[0][j] = act_t<__nv_bfloat16>(p.act, u0);
            v[1][j] = act_t<__nv_bfloat16>(p.act, u1);
          }
        }
        // neighbouring lanes hold neighbouring features: they exchange one of two tokens and store pairs
#pragma unroll
        for (int q = 0; q < (GLU ? 1 : 2); ++q) {
          const int f = (f0 & ~1) + q * 128;
#pragma unroll
          for (int j = 0; j < 16; j += 2) {
            const float mine = (lane & 1) ? v[q][j + 1] : v[q][j], give = (lane & 1) ? v[q][j] : v[q][j + 1];
            const float got = __shfl_xor_sync(0xffffffffu, give, 1);
            const int col = c0 + j + (lane & 1);
            if (col < t.live && f < p.N && t.row0 + col < p.n_rows)
              *reinterpret_cast<uint32_t*>(p.out + (size_t)(t.row0 + col) * p.N + f) =
                  (lane & 1) ? f2_to_bf2(got, mine) : f2_to_bf2(mine, got);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&t_empty[buf]);
    }
  }
  if (lane == 0 && *abort) raise_status(p.status, PACE_DEV_WAIT_TIMEOUT);
  tc_fence_before();
  __syncthreads();
  if (warp == kIssuerWarp) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(COLS) : "memory");
  }
}

int sm_count() {
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  return n;
}

template <int NT, bool GLU, bool GATHER>
int grouped(GroupedParams p, const void* weights, const void* rows, int n_b_rows, cudaStream_t s) {
  CUtensorMap tmA, tmB;
  const uint64_t st[1] = {(uint64_t)p.K * 2};
  const uint64_t da[2] = {(uint64_t)p.K, (uint64_t)p.n_experts * p.a_rows}, db[2] = {(uint64_t)p.K, (uint64_t)n_b_rows};
  const uint32_t ba[2] = {kKStep, 128}, bb[2] = {kKStep, GATHER ? 1u : (uint32_t)NT};
  int rc = tensor_map_bf16(&tmA, weights, 2, da, st, ba);
  if (rc == PACE_OK) rc = tensor_map_bf16(&tmB, rows, 2, db, st, bb);
  if (rc != PACE_OK) return rc;
  p.n_stages = (220 * 1024) / stage_bytes<NT>();
  if (p.n_stages > 8) p.n_stages = 8;
  p.m_tiles = (p.N + (GLU ? 127 : 255)) / (GLU ? 128 : 256);
  const int smem = p.n_stages * stage_bytes<NT>() + 1024;
  PACE_CUDA_TRY(cudaFuncSetAttribute(moe_grouped_kernel<NT, GLU, GATHER>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  moe_grouped_kernel<NT, GLU, GATHER><<<sm_count(), kThreads, smem, s>>>(p, tmA, tmB);
  PACE_LAUNCH_CHECK("moe_grouped_kernel");
  return PACE_OK;
}

template <int NT, bool GATHER>
int experts_umma(const pace_moe_experts_args_t& a, cudaStream_t s) {
  GroupedParams p;
  p.count = a.expert_count;
  p.list = a.expert_list;
  p.status = a.status;
  p.n_tokens = a.n_tokens;
  p.n_experts = a.n_experts;
  p.n_rows = a.n_tokens * a.top;
  p.act = a.act;
  p.out = static_cast<__nv_bfloat16*>(a.hidden);
  p.K = a.width;
  p.N = a.ff;
  p.a_rows = a.gated ? 2 * a.ff : a.ff;
  p.a_second = a.gated ? a.ff : 128;
  const void* rows = GATHER ? a.x : a.scratch;
  const int n_b_rows = GATHER ? a.n_tokens : p.n_rows;
  const int rc = a.gated ? grouped<NT, true, GATHER>(p, a.gate_up, rows, n_b_rows, s)
                         : grouped<NT, false, GATHER>(p, a.gate_up, rows, n_b_rows, s);
  if (rc != PACE_OK) return rc;
  p.act = PACE_ACT_NONE;
  p.out = static_cast<__nv_bfloat16*>(a.y);
  p.K = a.ff;
  p.N = a.width;
  p.a_rows = a.width;
  p.a_second = 128;
  return grouped<NT, false, false>(p, a.down, a.hidden, p.n_rows, s);
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" {

int pace_moe_route(const pace_moe_route_args_t* a, void* stream) {
  if (!a || !a->logits || !a->slot_expert || !a->slot_rank || !a->slot_weight || !a->expert_count || !a->expert_list ||
      a->n_tokens < 0 || a->n_experts < 1 || a->n_experts > kMaxExperts || a->top < 1 || a->top > kMaxTop || a->top > a->n_experts)
    return PACE_ERR_INVALID;
  if ((int64_t)a->n_tokens * a->top > 0x7fffffff) return PACE_ERR_UNSUPPORTED;
  const cudaStream_t s = (cudaStream_t)stream;
  if (a->n_tokens > 0 && a->n_tokens <= 64) {
    const int warps = a->n_tokens < 32 ? a->n_tokens : 32, rounds = (a->n_tokens + warps - 1) / warps;
    const size_t smem = route_smem(warps, rounds, a->n_experts, a->top);
    if (smem <= 200 * 1024) {
      PACE_CUDA_TRY(cudaFuncSetAttribute(moe_route_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
      moe_route_kernel<true><<<1, warps * 32, smem, s>>>(*a, rounds);
      PACE_LAUNCH_CHECK("moe_route_kernel");
      return PACE_OK;
    }
  }
  PACE_CUDA_TRY(cudaMemsetAsync(a->expert_count, 0, (size_t)a->n_experts * 4, s));
  if (a->n_tokens == 0) return PACE_OK;
  const size_t smem = route_smem(8, 1, a->n_experts, a->top);
  PACE_CUDA_TRY(cudaFuncSetAttribute(moe_route_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  moe_route_kernel<false><<<(a->n_tokens + 7) / 8, 256, smem, s>>>(*a, 1);
  PACE_LAUNCH_CHECK("moe_route_kernel");
  return PACE_OK;
}

int pace_moe_experts(const pace_moe_experts_args_t* a, void* stream) {
  if (!a || !a->x || !a->gate_up || !a->down || !a->hidden || !a->y || !a->expert_count || !a->expert_list || a->n_tokens < 0 ||
      a->n_experts < 1 || a->n_experts > kMaxExperts || a->top < 1 || a->width < 1 || a->ff < 1)
    return PACE_ERR_INVALID;
  if (a->act != PACE_ACT_SILU && a->act != PACE_ACT_GELU_TANH && a->act != PACE_ACT_GELU_ERF) return PACE_ERR_INVALID;
  if ((int64_t)a->n_tokens * a->top > 0x7fffffff || (int64_t)a->n_experts * 2 * a->ff > 0x7fffffff ||
      (int64_t)a->n_experts * a->width > 0x7fffffff)
    return PACE_ERR_UNSUPPORTED;
  if (a->n_tokens == 0) return PACE_OK;
  PACE_PROFILE("moe_experts", stream, "tokens=%d experts=%d top=%d width=%d ff=%d", a->n_tokens, a->n_experts, a->top, a->width,
               a->ff);
  const cudaStream_t s = (cudaStream_t)stream;
  if (a->dtype == PACE_DTYPE_FP32) return experts_simple<float>(*a, s);
  if (a->dtype != PACE_DTYPE_BF16) return PACE_ERR_INVALID;
  const bool umma = a->width % 8 == 0 && a->ff % 8 == 0 && aligned16(a->x) && aligned16(a->gate_up) && aligned16(a->down) &&
                    aligned16(a->hidden) && aligned16(a->y);
  if (!umma) return experts_simple<__nv_bfloat16>(*a, s);
  if (!a->scratch) return experts_umma<32, true>(*a, s);
  if (!a->slot_expert || !a->slot_rank || a->top > kMaxTop || !aligned16(a->scratch)) return PACE_ERR_INVALID;
  moe_spread_kernel<<<a->n_tokens, 256, 0, s>>>(*a);
  PACE_LAUNCH_CHECK("moe_spread_kernel");
  return experts_umma<128, false>(*a, s);
}

}  // extern "C"
