// Span attention over latents on tcgen05, for the few query rows of decoding and short portions: the keys are the 128-row
// operand.  A tile of query rows (16 or 32: token * heads + head) is the narrow operand of both products,
//     S^T [128 keys x rows]      = K [128 keys x dim] Q^T          (K as it lies in the page)
//     O^T [128 elements x rows]  = V^T [elements x 128 keys] P^T   (the same tile read the other way, element-major)
// so no row is padded to 128, and the two bf16 terms of the weights are neighbouring columns of one product: every operand
// tile is read once.  The legacy tensor path needs about eight times the cycles for this shape.
//
// A thread block has one tile of query rows and a contiguous share of its visible pages; the shares are the blocks of a
// cluster, merged as in attn_span.cu.  Warps 0-7: scores out of tensor memory (a lane holds a key) into shared memory, softmax
// by rows, weights into shared memory as the second product's operand; 8: TMA producer; 9: MMA issuer.  A chunk is two pages
// in 64-column blocks; a block's place is filled again as soon as the products that read it are done.
#include "span.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kPage = 64, kKeys = 128, kSoftmax = 256, kThreads = kSoftmax + 64;
constexpr int kBlock = kKeys * 128, kBoxRows = 16, kBox = kBoxRows * 128, kMaxBlocks = 16, kSS = kKeys + 4;
constexpr uint32_t kColO = 64;  // tensor memory: [0, rows) S^T, then O^T, 2 * rows columns per 128 elements

struct KeysParams {
  KVView kv;
  pace_step_t st;
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  const float* slopes;
  const float* sinks;
  int q_elems, out_elems, H, Gq, dim, dv, dv16;
  int k_blocks, v_tiles, v_used;   // 64-column blocks of a key, 128-element tiles of a value, blocks that values read
  int entry0, span, span_size, tmem_cols;
  float scale_log2;
  int64_t out_row;
};

struct KeysSmem {
  int k, q, p, s, ml, alpha, sink, bars, total;
};
__host__ __device__ inline KeysSmem keys_smem(int rows, int k_blocks, int dv16) {
  KeysSmem m;
  int off = 0;
  auto take = [&](int bytes, int align) {
    off = (off + align - 1) / align * align;
    const int o = off;
    off += bytes;
    return o;
  };
  m.k = take(k_blocks * kBlock, 1024);             // at the end: the block's results [rows][dv16 + 4] fp32
  if (off < rows * (dv16 + 4) * 4) off = rows * (dv16 + 4) * 4;
  m.q = take(k_blocks * rows * 128, 1024);         // [block][row][128 B]
  m.p = take(2 * (2 * rows) * 128, 1024);          // [64 keys][high rows, low rows][128 B]
  m.s = take(rows * kSS * 4, 16);
  m.ml = take(rows * 8, 8);
  m.alpha = take(rows * 4 + 16, 16);
  m.sink = take(rows * 4, 4);
  m.bars = take((2 * kMaxBlocks + 4) * 8, 8);
  m.total = off + 1024;
  return m;
}

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kSoftmax) : "memory"); }

template <int N>  // query rows of a tile
__global__ void __launch_bounds__(kThreads, 1) 
    attn_span_keys_kernel(const KeysParams p, const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                          const __grid_constant__ CUtensorMap tmPage) {
  constexpr int TPR = kSoftmax / N, PIECES = kKeys / 8 / TPR;
  extern __shared__ unsigned char smem_raw[];
  __shared__ uint32_t tmem_slot;
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const KeysSmem sm = keys_smem(N, p.k_blocks, p.dv16);
  const int ns = gridDim.x, share = blockIdx.x;  // the cluster is the grid's x extent
  const int e = p.entry0 + blockIdx.z;
  const int t0 = p.st.cu[e], count = p.st.cu[e + 1] - t0, start = p.st.start[e];
  const int R = count * p.Gq, r0 = blockIdx.y * N;
  if (r0 >= R) return;  // (the same for the whole cluster)
  const int live = min(N, R - r0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, KB = p.k_blocks;
  const int pos_a = start + r0 / p.Gq, pos_z = start + (r0 + live - 1) / p.Gq;
  const int key_a = span_first(p.span, p.span_size, pos_a), base = key_a & ~(kPage - 1);
  const int n_pages = (pos_z - base) / kPage + 1, per = (n_pages + ns - 1) / ns;
  const int page_a = min(share * per, n_pages), page_z = min(page_a + per, n_pages);
  const int n_chunks = (page_z - page_a + 1) / 2;
  const int end = min(pos_z + 1, base + page_z * kPage);  // keys of this share: positions base + page_a * 64 .. end - 1
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + sm.bars);
  uint64_t* empty = full + kMaxBlocks;
  uint64_t *s_full = empty + kMaxBlocks, *p_ready = s_full + 1, *o_full = s_full + 2;
  float* alpha = reinterpret_cast<float*>(smem + sm.alpha);
  volatile int* flags = reinterpret_cast<volatile int*>(alpha + N);   // [2] some row's maximum grew; [2]: the abort flag
  volatile int* abort = flags + 2;

  // the producer's page numbers: asked for now, needed behind the barrier
  int pages_ahead = 0;
  if (warp == 8) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&tmQ)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&tmPage)) : "memory");
    const int slot = p.st.slot[e];
    if (lane < page_z - page_a)
      pages_ahead = slot >= 0 && slot < p.kv.max_seqs ? view_page(p.kv, slot, base / kPage + page_a + lane) : -1;
  }
  if (warp == 9) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(p.tmem_cols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (tid == kSoftmax) {
    flags[0] = flags[1] = flags[2] = 0;
    for (int i = 0; i < KB; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(s_full, 1);
    mbar_init(p_ready, kSoftmax / 32);
    mbar_init(o_full, 1);
    fence_mbar_init();
  }
  // values of keys that no box of the first chunk brings are multiplied by zero weights and must be numbers (later chunks
  // find those of the first one)
  if (n_chunks > 0) {
    const int p0 = base + page_a * kPage;
    const int row_a = max(0, key_a - p0) / kBoxRows * kBoxRows, row_z = min(kKeys, (end - p0 + kBoxRows - 1) / kBoxRows * kBoxRows);
    const int gap = kKeys - (row_z - row_a);   // rows [0, row_a) and [row_z, 128), eight pieces each
    for (int i = tid; i < KB * gap * 8; i += kThreads) {
      const int b = i / (gap * 8), o = i - b * gap * 8, row = (o >> 3) < row_a ? o >> 3 : row_z + (o >> 3) - row_a;
      *reinterpret_cast<uint4*>(smem + sm.k + b * kBlock + row * 128 + (o & 7) * 16) = make_uint4(0, 0, 0, 0);
    }
  }
  if (tid < N) {
    const int rr = min(r0 + tid, R - 1);
    reinterpret_cast<float*>(smem + sm.sink)[tid] = p.sinks ? p.sinks[rr % p.Gq] * kLog2e : -INFINITY;
  }
  fence_proxy_async();  // generic-proxy writes before TMA's and the tensor core's accesses
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&tmem_slot);

  if (warp == 8) {
    // ================================ producer ================================
    bool ok = true;
    auto page_of = [&](int i) {   // i-th page of the share
      int pg = 0;
      if (i < 32) {
        pg = __shfl_sync(0xffffffffu, pages_ahead, i);
      } else {
        const int slot = p.st.slot[e];
        pg = slot >= 0 && slot < p.kv.max_seqs ? view_page(p.kv, slot, base / kPage + page_a + i) : -1;
      }
      if (pg < 0) {
        if (lane == 0) raise_status(p.kv.status, PACE_DEV_BAD_INDEX);
        pg = 0;
      }
      return pg;
    };
    for (int c = 0; c < n_chunks && ok; ++c) {
      const int p0 = base + (page_a + 2 * c) * kPage;
      int page[2] = {0, 0};
#pragma unroll
      for (int h = 0; h < 2; ++h)
        if (p0 + h * kPage < end) page[h] = page_of(2 * c + h);
      const int box_a = max(0, key_a - p0) / kBoxRows, box_z = min(kKeys, end - p0 + kBoxRows - 1) / kBoxRows;
      for (int b = 0; b < KB; ++b) {
        if (c > 0 && !__all_sync(0xffffffffu, mbar_wait(&empty[b], (c - 1) & 1, abort))) {
          ok = false;
          break;
        }
        if (lane == 0) {
          mbar_arrive_expect_tx(&full[b], (uint32_t)(box_z - box_a) * kBox + (c == 0 ? N * 128u : 0u));
          if (c == 0) tma_load_2d(smem + sm.q + b * (N * 128), &tmQ, b * 64, t0 * p.H + r0, &full[b]);
        }
        __syncwarp();
        // whole pages in one box each, others by 16 keys
        const int bx = box_a + lane, half = bx >> 2;
        const bool whole = box_a <= 4 * half && box_z >= 4 * half + 4;
        if (bx < box_z && whole) {
          if ((bx & 3) == 0) tma_load_3d(smem + sm.k + b * kBlock + bx * kBox, &tmPage, b * 64, 0, page[half & 1], &full[b]);
        } else if (bx < box_z)
          tma_load_3d(smem + sm.k + b * kBlock + bx * kBox, &tmK, b * 64, bx * kBoxRows & (kPage - 1), page[half & 1],
                      &full[b]);
      }
      // what the next chunk needs starts for L2 while this one is worked on
      if (c + 1 < n_chunks) {
        const int i = 2 * (c + 1);
        const int pg0 = page_of(i), pg1 = p0 + 3 * kPage < end ? page_of(i + 1) : -1;
        for (int k = lane; k < 2 * KB; k += 32) {
          const int pg = k < KB ? pg0 : pg1;
          if (pg >= 0) tma_prefetch_3d(&tmPage, (k < KB ? k : k - KB) * 64, 0, pg);
        }
      }
      if (!ok)   // copies in flight land before the block's shared memory is released
        for (int b = 0; b < KB; ++b) mbar_wait(&full[b], (c - 1) & 1), mbar_wait(&full[b], c & 1, abort, 1024);
    }
  } else if (warp == 9) {
    // ================================ MMA issuer ================================
    constexpr uint32_t IDESC_S = umma_idesc(N, false), IDESC_O = umma_idesc_at(2 * N);
    const bool leader = elect_one();
    // (a shared-memory address of a block in a cluster has the block's rank above the 18 bits a descriptor takes)
    auto lo = [&](int at, uint32_t lbo) { return ((smem_u32(smem + at) >> 4) & 0x3FFFu) | (lbo << 16); };
    const uint32_t k_lo = lo(sm.k, 1), q_lo = lo(sm.q, 1), p_lo = lo(sm.p, 1);
    // the tile read element-major: 64-element blocks lie kBlock apart
    const uint32_t v_lo = lo(sm.k, kBlock >> 4);
    const int last = (p.dim - (KB - 1) * 64 + 15) / 16;   // 16-column steps of the last block
    for (int c = 0; c < n_chunks; ++c) {
      bool ok = true;
      for (int b = 0; b < KB; ++b) {
        if (!umma_issuer_wait(&full[b], c & 1, abort)) {
          ok = false;
          break;
        }
        tc_fence_after();
        if (leader) {
          const int steps = b == KB - 1 ? last : 4;
          for (int kk = 0; kk < steps; ++kk)
            umma_bf16(tmem, pack64(k_lo + b * (kBlock >> 4) + kk * 2, kDescHi), pack64(q_lo + b * (N * 128 >> 4) + kk * 2, kDescHi), IDESC_S,
                      (b | kk) ? 1u : 0u);
          if (b >= p.v_used) umma_commit(&empty[b]);   // (values do not read it)
          if (b == KB - 1) umma_commit(s_full);
        }
        __syncwarp();
      }
      if (!ok || !umma_issuer_wait(p_ready, c & 1, abort)) break;
      tc_fence_after();
      if (leader) {
        const int keys = min(kKeys, end - (base + (page_a + 2 * c) * kPage)), ksteps = (keys + 15) / 16;
        for (int j = 0; j < p.v_tiles; ++j) {
          for (int ks = 0; ks < ksteps; ++ks)
            umma_bf16(tmem + kColO + j * 2 * N, pack64(v_lo + j * (2 * kBlock >> 4) + ks * (2048 >> 4), kDescHi),
                      pack64(p_lo + (ks >> 2) * (2 * N * 128 >> 4) + (ks & 3) * 2, kDescHi), IDESC_O, (c | ks) ? 1u : 0u);
          umma_commit(&empty[2 * j]);
          if (2 * j + 1 < p.v_used) umma_commit(&empty[2 * j + 1]);
        }
        if (c == n_chunks - 1) umma_commit(o_full);
      }
      __syncwarp();
    }
    if (*abort && leader)  // products in flight end before tensor memory is handed back
      for (int k = 0; k < 4096; ++k) __nanosleep(256);
    __syncwarp();
  } else {
    // ================================ softmax ================================
    const int quad = warp & 3, half = warp >> 2;
    const uint32_t t_lane = tmem + ((uint32_t)(quad * 32) << 16);
    const int h = tid / TPR, sub = tid % TPR;
    const int srr = r0 + h, stok = srr / p.Gq, shead = srr - stok * p.Gq;
    const int spos = h < live ? start + stok : -1, sfirst = h < live ? span_first(p.span, p.span_size, spos) : 0;
    const float slope = (p.slopes && h < live) ? p.slopes[shead] * kLog2e : 0.f;
    float* S = reinterpret_cast<float*>(smem + sm.s);
    float m = -INFINITY, l = 0.f;
    // (a wait that ran out raises the flag, which cuts the waits behind it short; nobody leaves the common barriers)
    for (int c = 0; c < n_chunks; ++c) {
      umma_wait(s_full, c & 1, abort);
      tc_fence_after();
      for (int c0 = half * 16; c0 < N; c0 += 32) {
        uint32_t x[16];
        tmem_ld16(t_lane + c0, x);
        tmem_wait_ld();
#pragma unroll
        for (int j = 0; j < 16; ++j) S[(c0 + j) * kSS + quad * 32 + lane] = __uint_as_float(x[j]);
      }
      softmax_sync();
      const int p0 = base + (page_a + 2 * c) * kPage;
      float x[PIECES][8], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < PIECES; ++i) {
        const int k = 8 * (sub + TPR * i), pos = p0 + k;
        Vec<float, 8>::load(S + h * kSS + k, x[i]);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const bool seen = pos + j <= spos && pos + j >= sfirst && pos + j < end;
          x[i][j] = seen ? fmaf(x[i][j], p.scale_log2, slope * (float)(pos + j - spos)) : -INFINITY;
          mx = fmaxf(mx, x[i][j]);
        }
      }
#pragma unroll
      for (int d = TPR / 2; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      // the reference maximum moves only when it has to: O^T is rescaled in tensor memory
      const bool grow = mx > m + 8.0f;
      const float f = grow ? (m == -INFINITY ? 0.f : fast_exp2(m - mx)) : 1.f;
      if (grow) m = mx;
      if (sub == 0) alpha[h] = f;
      if (__any_sync(0xffffffffu, grow) && lane == 0) flags[c & 1] = 1;
      const float ref = m == -INFINITY ? 0.f : m;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < PIECES; ++i) {
        const int piece = sub + TPR * i;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float w0 = fast_exp2(x[i][2 * j] - ref), w1 = fast_exp2(x[i][2 * j + 1] - ref);
          sum += w0 + w1;
          split_bf2(w0, w1, hi[j], lo[j]);
        }
        unsigned char* blk = smem + sm.p + (piece >> 3) * (2 * N * 128);
        const int sw = ((piece & 7) ^ (h & 7)) << 4;   // (N is a multiple of 8: row h + N has the same swizzle)
        *reinterpret_cast<uint4*>(blk + h * 128 + sw) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(blk + (N + h) * 128 + sw) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      l = l * f + sum;
      fence_proxy_async();
      softmax_sync();
      if (tid == 0) flags[(c + 1) & 1] = 0;
      if (c > 0 && flags[c & 1]) {
        // (the commit behind this chunk's scores covers the products of the chunk in front)
        for (int j = 0; j < p.v_tiles; ++j)
          for (int c0 = half * 16; c0 < 2 * N; c0 += 32) {
            const uint32_t at = t_lane + kColO + j * 2 * N + c0;
            uint32_t o[16];
            tmem_ld16(at, o);
            tmem_wait_ld();
#pragma unroll
            for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * alpha[(c0 + k) % N]);
            tmem_st16(at, o);
          }
        tmem_wait_st();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    // ---- this block's results to shared memory ----
#pragma unroll
    for (int d = TPR / 2; d; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
    if (sub == 0) reinterpret_cast<float2*>(smem + sm.ml)[h] = make_float2(m, l);
    if (n_chunks > 0) {
      umma_wait(o_full, 0, abort);
      tc_fence_after();
      float* O = reinterpret_cast<float*>(smem + sm.k);
      const int OS = p.dv16 + 4;
      for (int j = 0; j < p.v_tiles; ++j) {
        const int d = j * 128 + quad * 32 + lane;
        for (int c0 = half * 16; c0 < N; c0 += 32) {
          uint32_t a[16], b[16];
          tmem_ld16(t_lane + kColO + j * 2 * N + c0, a);
          tmem_ld16(t_lane + kColO + j * 2 * N + N + c0, b);
          tmem_wait_ld();
          if (d < p.dv16) {
#pragma unroll
            for (int k = 0; k < 16; ++k) O[(c0 + k) * OS + d] = __uint_as_float(a[k]) + __uint_as_float(b[k]);
          }
        }
      }
      tc_fence_before();
    }
  }
  if (lane == 0 && *abort) raise_status(p.kv.status, PACE_DEV_WAIT_TIMEOUT);
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
  }
  cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
  if (ns > 1) cl.sync();
  span_merge(reinterpret_cast<float*>(smem + sm.k), p.dv16 + 4, reinterpret_cast<float2*>(smem + sm.ml),
             reinterpret_cast<float*>(smem + sm.sink), reinterpret_cast<float*>(smem + sm.s), ns, share, tid, kThreads, live, r0, t0, 0, p.Gq, p.dv, p.dv16, p.out, p.out_row, p.out_elems);
  if (ns > 1) cl.sync();  // nobody leaves while its shared memory is read
}

int sm_count() {
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  return n;
}

template <int N>
int launch_keys(KeysParams& p, const CUtensorMap& tk, const CUtensorMap& tpage, int max_tokens, int max_keys, int entries, cudaStream_t s) {
  const int smem = keys_smem(N, p.k_blocks, p.dv16).total;
  if (smem > 227 * 1024 - 64) return PACE_ERR_UNSUPPORTED;
  p.tmem_cols = 128;
  while (p.tmem_cols < (int)kColO + p.v_tiles * 2 * N) p.tmem_cols *= 2;
  if (p.tmem_cols > 512) return PACE_ERR_UNSUPPORTED;
  const int tok = (N - 1) / p.Gq + 2;   // tokens a tile can touch
  if (p.span != PACE_SPAN_ALL && (long long)p.span_size + tok < max_keys) max_keys = p.span_size + tok;
  const int pages = max_keys / kPage + 1;
  const long long tiles = ((long long)max_tokens * p.Gq + N - 1) / N, units = tiles * entries;
  if (tiles > 65535 || entries > 65535) return PACE_ERR_UNSUPPORTED;
  // the share count that leaves the fewest pages per block while all blocks are resident at once (one per SM)
  int ns = 1;
  for (int k = 2; k <= 8 && units * k <= sm_count(); ++k)
    if ((pages + k - 1) / k < (pages + ns - 1) / ns) ns = k;
  CUtensorMap tq;
  const uint64_t dims[2] = {(uint64_t)p.q_elems, (uint64_t)p.st.n_tokens * p.H}, str[1] = {(uint64_t)p.q_elems * 2};
  const uint32_t box[2] = {64, N};
  const int rc = tensor_map_bf16(&tq, p.q, 2, dims, str, box);
  if (rc != PACE_OK) return rc;
  auto* fn = attn_span_keys_kernel<N>;
  PACE_CUDA_TRY(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)tiles, (unsigned)entries);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = (size_t)smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)ns;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  PACE_CUDA_TRY(cudaLaunchKernelEx(&cfg, fn, p, tq, tk, tpage));
  PACE_LAUNCH_CHECK("attn_span_keys_kernel");
  return PACE_OK;
}

}  // namespace

// PACE_ERR_UNSUPPORTED: shapes beyond this kernel (nothing launched)
int attn_span_keys(const pace_kv_pool_t* pl, int layer, const pace_step_t& st, const pace_attn_span_args_t& a, cudaStream_t s) {
  if (pl->row_format != PACE_ROWS_SHARED || pl->n_kv_heads != 1 || pl->page_tokens != kPage || pl->head_dim % 8 || a.q_elems % 8 ||
      a.vdim > 512 || a.vdim > a.dim || a.softcap > 0.f || !aligned16(a.q) || !aligned16(pl->pages) || ((uintptr_t)a.out & 7))
    return PACE_ERR_UNSUPPORTED;
  KeysParams p;
  p.kv = make_view(pl, layer, nullptr);
  p.st = st;
  p.q = static_cast<const __nv_bfloat16*>(a.q);
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.slopes = a.slopes;
  p.sinks = a.sinks;
  p.q_elems = a.q_elems;
  p.out_elems = a.out_elems;
  p.H = p.Gq = a.n_q_heads;
  p.dim = a.dim;
  p.dv = a.vdim;
  p.dv16 = (a.vdim + 15) / 16 * 16;
  p.k_blocks = (a.dim + 63) / 64;
  p.v_tiles = (a.vdim + 127) / 128;
  p.v_used = 2 * p.v_tiles < p.k_blocks ? 2 * p.v_tiles : p.k_blocks;
  p.entry0 = a.entry_begin;
  p.span = a.span;
  p.span_size = a.span_size;
  p.scale_log2 = a.scale * kLog2e;
  p.out_row = span_out_row(a);
  if (p.k_blocks > kMaxBlocks) return PACE_ERR_UNSUPPORTED;
  CUtensorMap tk, tpage;
  const uint64_t row = (uint64_t)pl->head_dim;
  const uint64_t dims[3] = {row, kPage, (uint64_t)pl->n_pages}, str[2] = {row * 2, row * 2 * kPage};
  const uint32_t box[3] = {64, kBoxRows, 1};
  const uint32_t whole[3] = {64, kPage, 1};
  int rc = tensor_map_bf16(&tk, p.kv.k, 3, dims, str, box);
  if (rc == PACE_OK) rc = tensor_map_bf16(&tpage, p.kv.k, 3, dims, str, whole);
  if (rc != PACE_OK) return rc;
  const int E = a.entry_end - a.entry_begin;
  return a.max_tokens * p.Gq <= 16 ? launch_keys<16>(p, tk, tpage, a.max_tokens, a.max_keys, E, s)
                                   : launch_keys<32>(p, tk, tpage, a.max_tokens, a.max_keys, E, s);
}

}  // namespace pace
