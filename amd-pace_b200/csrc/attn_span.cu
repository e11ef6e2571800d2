// Softmax attention over the paged pool with a span (window or chunk), a distance bias and a sink: decode, short
// portions of prompts and whatever the tcgen05 prompt kernel (attn_span_umma.cu) does not take.  bf16 rows of any size,
// keys and values in two planes or (latents) in one.
//
// A thread block works on one tile of 16 * MT query rows (row = token * group + head of the group) of one (entry, KV
// head) and a contiguous share of the tile's visible keys; the shares of a tile are the blocks of a thread-block cluster.
// A producer warp streams tiles of 64 keys (one page) through a ring of shared-memory stages: TMA boxes of 64 columns x 16
// rows with the 128-byte swizzle, only those that hold visible keys.  Eight consumer warps, per tile
//   scores   warp w: all query rows x keys 8 w .. 8 w + 7, mma.sync m16n8k16
//   softmax  256 / rows threads per row, fp32, span and bias from positions; weights leave as two bf16 terms
//   values   warp w: all query rows x the 16-column groups w, w + 8, ...
// At the end every block has (maximum, sum, weighted values) of its keys in shared memory; the blocks of the cluster merge
// them over distributed shared memory, each a part of the outputs.  No workspace, no atomics, no order that varies.
#include "span.cuh"
#include "umma.cuh"

namespace pace {
namespace {

constexpr int kKeys = 64, kConsumers = 256, kThreads = kConsumers + 32, kPS = kKeys + 8, kSS = kKeys + 4;
constexpr int kBlock = kKeys * 128, kBoxRows = 16, kBox = kBoxRows * 128;  // 64 columns x 64 keys, x 16 keys (bytes)

struct SpanParams {
  KVView kv;
  pace_step_t st;
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  const float* slopes;
  const float* sinks;
  int q_elems, out_elems, H, Gq, dv;
  int dk16, dv16, k_blocks, v_blocks;   // sizes rounded up to 16; 64-column blocks of a stage (v_blocks 0: one plane)
  int entry0, span, span_size, n_stages;
  float scale_log2;
  ScoreCap cap;
  int64_t out_row;
};

struct SpanSmem {
  int ring, q, s, ph, pl, alpha, ml, sink, bars, obuf, total;
};
__host__ __device__ inline SpanSmem span_smem(int MR, int dk16, int dv16, int blocks, int n_stages) {
  SpanSmem m;
  int off = 0;
  auto take = [&](int bytes) {
    const int o = off;
    off += (bytes + 15) / 16 * 16;
    return o;
  };
  m.ring = take(n_stages * blocks * kBlock);
  m.obuf = 0;  // behind the last tile the ring's place (and the queries') holds the block's results
  m.q = take(MR * (dk16 + 8) * 2);
  if (off < MR * (dv16 + 4) * 4) off = (MR * (dv16 + 4) * 4 + 15) / 16 * 16;
  m.s = take(MR * kSS * 4);
  m.ph = take(MR * kPS * 2);
  m.pl = take(MR * kPS * 2);
  m.alpha = take(MR * 4);
  m.ml = take(MR * 8);
  m.sink = take(MR * 4);
  m.bars = take(2 * 8 * 8 + 8);
  m.total = off + 1024;  // (the ring starts at a multiple of 1024)
  return m;
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void consumer_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kConsumers) : "memory"); }

// MT: 16-row tiles of query rows; NG: 16-column groups of the values a warp owns
template <int MT, int NG>
__global__ void __launch_bounds__(kThreads, MT * NG <= 4 ? 2 : 1)
    attn_span_kernel(const SpanParams p, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV) {
  constexpr int MR = 16 * MT, TPR = kConsumers / MR, KPT = kKeys / TPR;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int blocks = p.k_blocks + p.v_blocks, STAGE = blocks * kBlock;
  const SpanSmem sm = span_smem(MR, p.dk16, p.dv16, blocks, p.n_stages);
  const int ns = gridDim.x, share = blockIdx.x;  // the cluster is the grid's x extent
  const int Hkv = p.kv.n_kv_heads, g = blockIdx.y % Hkv, e = p.entry0 + blockIdx.z;
  const int t0 = p.st.cu[e], count = p.st.cu[e + 1] - t0, start = p.st.start[e];
  const int R = count * p.Gq, r0 = (int)(blockIdx.y / Hkv) * MR;
  if (r0 >= R) return;  // (the same for the whole cluster)
  const int live = min(MR, R - r0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos_a = start + r0 / p.Gq, pos_z = start + (r0 + live - 1) / p.Gq;
  const int key_a = span_first(p.span, p.span_size, pos_a), base = key_a & ~(kKeys - 1);
  const int n_tiles = (pos_z - base) / kKeys + 1;
  const int per = (n_tiles + ns - 1) / ns;
  const int tile_a = min(share * per, n_tiles), tile_z = min(tile_a + per, n_tiles);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + sm.bars);
  uint64_t* empty = full + 8;
  int* abort_flag = reinterpret_cast<int*>(empty + 8);
  volatile int* abort = abort_flag;
  const uint32_t s_ring = smem_u32(smem + sm.ring), s_q = smem_u32(smem + sm.q);
  const int QSB = (p.dk16 + 8) * 2;  // row stride of the queries, bytes: an odd number of 16-byte units

  // the producer's page numbers: asked for now, needed behind the barrier
  int pages_ahead = 0;
  if (warp == kConsumers / 32) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&tmK)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&tmV)) : "memory");
    const int slot = p.st.slot[e];
    if (tile_a + lane < tile_z)
      pages_ahead = slot >= 0 && slot < p.kv.max_seqs ? view_page(p.kv, slot, base / kKeys + tile_a + lane) : -1;
  }
  if (tid == kConsumers) {
    *abort_flag = 0;
    for (int i = 0; i < p.n_stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], kConsumers / 32);
    }
    fence_mbar_init();
  }
  // values of keys that no box brings into a stage's first tile are multiplied by zero weights and must be numbers (later
  // tiles find those of earlier ones)
  for (int s = 0; s < p.n_stages && tile_a + s < tile_z; ++s) {
    const int p0 = base + (tile_a + s) * kKeys;
    const int row_a = max(0, key_a - p0) / kBoxRows * kBoxRows, row_z = min(kKeys, (pos_z - p0) / kBoxRows * kBoxRows + kBoxRows);
    const int gap = kKeys - (row_z - row_a);   // rows [0, row_a) and [row_z, 64), eight pieces each
    for (int i = tid; i < blocks * gap * 8; i += kThreads) {
      const int b = i / (gap * 8), o = i - b * gap * 8, row = (o >> 3) < row_a ? o >> 3 : row_z + (o >> 3) - row_a;
      *reinterpret_cast<uint4*>(smem + sm.ring + (size_t)s * STAGE + b * kBlock + row * 128 + (o & 7) * 16) = make_uint4(0, 0, 0, 0);
    }
  }
  if (tid < MR) {
    const int rr = min(r0 + tid, R - 1);
    reinterpret_cast<float*>(smem + sm.sink)[tid] = p.sinks ? p.sinks[g * p.Gq + rr % p.Gq] * kLog2e : -INFINITY;
  }
  fence_proxy_async();
  __syncthreads();

  if (warp == kConsumers / 32) {
    // ================================ producer ================================
    int page = 0, s = 0, ph = 0, issued = 0;
    for (int t = tile_a; t < tile_z; ++t) {
      if (((t - tile_a) & 31) == 0) {  // the next 32 tiles' pages, one per lane
        page = pages_ahead;
        if (t > tile_a) {
          const int slot = p.st.slot[e];
          page = t + lane >= tile_z ? 0 : slot >= 0 && slot < p.kv.max_seqs ? view_page(p.kv, slot, base / kKeys + t + lane) : -1;
        }
        if (page < 0) {
          raise_status(p.kv.status, PACE_DEV_BAD_INDEX);
          page = 0;
        }
      }
      const int pg = __shfl_sync(0xffffffffu, page, (t - tile_a) & 31);
      if (issued >= p.n_stages && !__all_sync(0xffffffffu, mbar_wait(&empty[s], ph ^ 1, abort))) break;
      const int p0 = base + t * kKeys;
      const int box_a = max(0, key_a - p0) / kBoxRows, box_z = min(kKeys, pos_z + 1 - p0 + kBoxRows - 1) / kBoxRows;
      if (lane == 0) mbar_arrive_expect_tx(&full[s], (uint32_t)((box_z - box_a) * blocks * kBox));
      __syncwarp();
      unsigned char* st = smem + sm.ring + (size_t)s * STAGE;
      const int n = (box_z - box_a) * blocks;
      for (int i = lane; i < n; i += 32) {
        const int bx = box_a + i / blocks, b = i % blocks;
        const bool is_v = b >= p.k_blocks;
        tma_load_3d(st + b * kBlock + bx * kBox, is_v ? &tmV : &tmK, (is_v ? b - p.k_blocks : b) * 64, bx * kBoxRows, pg * Hkv + g,
                    &full[s]);
      }
      ++issued;
      if (++s == p.n_stages) s = 0, ph ^= 1;
    }
    if (*abort) {  // copies in flight land before the block's shared memory is released
      for (int k = issued > p.n_stages ? issued - p.n_stages : 0; k < issued; ++k) mbar_wait(&full[k % p.n_stages], (k / p.n_stages) & 1);
    }
    if (ns > 1) {
      cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
      cl.sync();
      cl.sync();
    }
    return;
  }

  // ---- consumers: the query rows ----
  {
    const int pieces = p.dk16 / 8;
    for (int r = warp; r < MR; r += kConsumers / 32) {
      const int rr = min(r0 + r, R - 1), tok = rr / p.Gq, hh = g * p.Gq + rr - tok * p.Gq;
      const __nv_bfloat16* src = p.q + ((size_t)(t0 + tok) * p.H + hh) * p.q_elems;
      for (int c = lane; c < pieces; c += 32) {
        const bool ok = r < live && (c + 1) * 8 <= p.q_elems;
        cp_async16(s_q + r * QSB + c * 16, src + (ok ? c * 8 : 0), ok);
      }
    }
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    consumer_sync();
  }

  // softmax role of this thread: one row, keys 4 (sub + TPR i) + 0..3
  const int srow = tid / TPR, sub = tid % TPR;
  const int srr = r0 + srow, stok = srr / p.Gq;
  const int spos = srow < live ? start + stok : -1;
  const int sfirst = srow < live ? span_first(p.span, p.span_size, spos) : 0;
  const int shead = g * p.Gq + (srr - stok * p.Gq);
  const float slope = (p.slopes && srow < live) ? p.slopes[shead] * kLog2e : 0.f;
  float m = -INFINITY, l = 0.f;
  float* S = reinterpret_cast<float*>(smem + sm.s);
  float* alpha = reinterpret_cast<float*>(smem + sm.alpha);
  const uint32_t s_ph = smem_u32(smem + sm.ph), s_pl = smem_u32(smem + sm.pl);

  float o[MT][NG][2][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int b = 0; b < NG; ++b)
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int d = 0; d < 4; ++d) o[a][b][c][d] = 0.f;

  const int n_groups = p.dv16 / 16, ksteps = p.dk16 / 16;
  const int v_off = p.v_blocks ? p.k_blocks * kBlock : 0;
  int st_i = 0, st_ph = 0;
  for (int t = tile_a; t < tile_z; ++t) {
    // (a wait that ran out raises the flag, which cuts the waits behind it short; nobody leaves the common barriers)
    mbar_wait(&full[st_i], st_ph, abort);
    const uint32_t stage = s_ring + (uint32_t)st_i * STAGE;
    // ---- scores ----
    {
      float c[MT][2][4];
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int b = 0; b < 2; ++b)
#pragma unroll
          for (int d = 0; d < 4; ++d) c[a][b][d] = 0.f;
      // ldmatrix x4 over two k-steps of this warp's eight keys; A: rows lane % 16, column half lane / 16.
      // Key tiles: 64-column blocks, 16-byte piece c of row r at ((c ^ r % 8) * 16)
      const uint32_t kb = stage + (warp * 8 + (lane & 7)) * 128;
      const uint32_t kc = (uint32_t)((lane >> 3) ^ (lane & 7)) << 4;   // piece 0 .. 3 of this lane's matrix; 4 .. 7: bit 6 flipped
      const uint32_t qa = s_q + (lane & 15) * QSB + (lane >> 4) * 16;
      int kk = 0;
#pragma unroll 2
      for (; kk + 2 <= ksteps; kk += 2) {
        uint32_t b[4];
        ldsm4(kb + (kk >> 2) * kBlock + (kc ^ ((kk & 2) << 5)), b);
#pragma unroll
        for (int a = 0; a < MT; ++a) {
          uint32_t q0[4], q1[4];
          ldsm4(qa + a * 16 * QSB + kk * 32, q0);
          ldsm4(qa + a * 16 * QSB + kk * 32 + 32, q1);
          mma16816(c[a][0], q0, b[0], b[1]);
          mma16816(c[a][1], q1, b[2], b[3]);
        }
      }
      if (kk < ksteps) {
        uint32_t b[4];   // (the second step's pieces lie in the same block: zeros or what follows, not used)
        ldsm4(kb + (kk >> 2) * kBlock + (kc ^ ((kk & 2) << 5)), b);
#pragma unroll
        for (int a = 0; a < MT; ++a) {
          uint32_t q0[4];
          ldsm4(qa + a * 16 * QSB + kk * 32, q0);
          mma16816(c[a][0], q0, b[0], b[1]);
        }
      }
      const int col = warp * 8 + (lane & 3) * 2;
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        const int r = a * 16 + (lane >> 2);
        *reinterpret_cast<float2*>(S + r * kSS + col) = make_float2(c[a][0][0] + c[a][1][0], c[a][0][1] + c[a][1][1]);
        *reinterpret_cast<float2*>(S + (r + 8) * kSS + col) = make_float2(c[a][0][2] + c[a][1][2], c[a][0][3] + c[a][1][3]);
      }
    }
    consumer_sync();
    // ---- softmax ----
    {
      float x[KPT];
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT / 4; ++i) {
        const int k = 4 * (sub + TPR * i), pos = base + t * kKeys + k;
        const float4 s4 = *reinterpret_cast<const float4*>(S + srow * kSS + k);
        const float sv[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const bool seen = pos + j <= spos && pos + j >= sfirst;
          const float sc = p.cap.out != 0.f ? capped(p.cap, sv[j]) : sv[j] * p.scale_log2;
          x[4 * i + j] = seen ? fmaf(slope, (float)(pos + j - spos), sc) : -INFINITY;
          mx = fmaxf(mx, x[4 * i + j]);
        }
      }
#pragma unroll
      for (int d = TPR / 2; d; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float mn = fmaxf(m, mx);
      const float f = m == -INFINITY ? (mn == -INFINITY ? 1.f : 0.f) : fast_exp2(m - mn);
      const float ref = mn == -INFINITY ? 0.f : mn;
      m = mn;
      float sum = 0.f;
      const uint32_t prow = (uint32_t)srow * (kPS * 2);
#pragma unroll
      for (int i = 0; i < KPT / 4; ++i) {
        uint32_t h0, h1, l0, l1;
        float w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          w[j] = fast_exp2(x[4 * i + j] - ref);
          sum += w[j];
        }
        split_bf2(w[0], w[1], h0, l0);
        split_bf2(w[2], w[3], h1, l1);
        const uint32_t at = prow + 8 * (sub + TPR * i);
        asm volatile("st.shared.v2.b32 [%0], {%1, %2};" ::"r"(s_ph + at), "r"(h0), "r"(h1) : "memory");
        asm volatile("st.shared.v2.b32 [%0], {%1, %2};" ::"r"(s_pl + at), "r"(l0), "r"(l1) : "memory");
      }
      l = l * f + sum;
      if (sub == 0) alpha[srow] = f;
    }
    consumer_sync();
    // ---- values ----
    if (warp < n_groups) {
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        const float f0 = alpha[a * 16 + (lane >> 2)], f1 = alpha[a * 16 + (lane >> 2) + 8];
        if (f0 != 1.f || f1 != 1.f) {
#pragma unroll
          for (int b = 0; b < NG; ++b)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
              o[a][b][c][0] *= f0;
              o[a][b][c][1] *= f0;
              o[a][b][c][2] *= f1;
              o[a][b][c][3] *= f1;
            }
        }
      }
      const uint32_t pa = (uint32_t)(lane & 15) * (kPS * 2) + (lane >> 4) * 16;
      // rows lane % 16 of a k-step; the group's two pieces by lane / 16
      const uint32_t vb = stage + v_off + (lane & 15) * 128;
      const uint32_t vh = (uint32_t)(lane >> 4), vx = (uint32_t)(lane & 7);
#pragma unroll
      for (int ks = 0; ks < kKeys / 16; ++ks) {
        uint32_t ah[MT][4], al[MT][4];
#pragma unroll
        for (int a = 0; a < MT; ++a) {
          ldsm4(s_ph + pa + a * 16 * (kPS * 2) + ks * 32, ah[a]);
          ldsm4(s_pl + pa + a * 16 * (kPS * 2) + ks * 32, al[a]);
        }
#pragma unroll
        for (int b = 0; b < NG; ++b) {
          const int gi = warp + 8 * b;
          if (gi < n_groups) {
            uint32_t v[4];
            ldsm4_t(vb + (gi >> 2) * kBlock + ks * 16 * 128 + (((((uint32_t)gi & 3) * 2 + vh) ^ vx) << 4), v);
#pragma unroll
            for (int a = 0; a < MT; ++a) {
              mma16816(o[a][b][0], ah[a], v[0], v[1]);
              mma16816(o[a][b][1], ah[a], v[2], v[3]);
              mma16816(o[a][b][0], al[a], v[0], v[1]);
              mma16816(o[a][b][1], al[a], v[2], v[3]);
            }
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st_i]);
    if (++st_i == p.n_stages) st_i = 0, st_ph ^= 1;
  }
  consumer_sync();
  if (tid == 0 && *abort) raise_status(p.kv.status, PACE_DEV_WAIT_TIMEOUT);

  // ---- this block's results to shared memory, merge over the cluster ----
  float* O = reinterpret_cast<float*>(smem + sm.obuf);
  float2* ml = reinterpret_cast<float2*>(smem + sm.ml);
  const int OS = p.dv16 + 4;
#pragma unroll
  for (int d = TPR / 2; d; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
  if (sub == 0) ml[srow] = make_float2(m, l);
#pragma unroll
  for (int b = 0; b < NG; ++b) {
    const int gi = warp + 8 * b;
    if (gi < n_groups) {
#pragma unroll
      for (int a = 0; a < MT; ++a)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int r = a * 16 + (lane >> 2), col = gi * 16 + c * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(O + r * OS + col) = make_float2(o[a][b][c][0], o[a][b][c][1]);
          *reinterpret_cast<float2*>(O + (r + 8) * OS + col) = make_float2(o[a][b][c][2], o[a][b][c][3]);
        }
    }
  }
  cooperative_groups::cluster_group cl = cooperative_groups::this_cluster();
  if (ns > 1) cl.sync();
  else consumer_sync();
  span_merge(O, OS, ml, reinterpret_cast<float*>(smem + sm.sink), S, ns, share, tid, kConsumers, live, r0, t0, g, p.Gq, p.dv,
             p.dv16, p.out, p.out_row, p.out_elems);
  if (ns > 1) cl.sync();  // nobody leaves while its shared memory is read
}

template <int MT, int NG>
int launch_span(SpanParams& p, const CUtensorMap& tk, const CUtensorMap& tv, int ns, int tiles, int entries, int smem,
                cudaStream_t s) {
  auto* fn = attn_span_kernel<MT, NG>;
  PACE_CUDA_TRY(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)ns, (unsigned)(tiles * p.kv.n_kv_heads), (unsigned)entries);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = (size_t)smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)ns;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  PACE_CUDA_TRY(cudaLaunchKernelEx(&cfg, fn, p, tk, tv));
  PACE_LAUNCH_CHECK("attn_span_kernel");
  return PACE_OK;
}

constexpr int kSmemMax = 227 * 1024, kSmemHalf = 113 * 1024, kMaxCluster = 8;

int sm_count() {
  int dev = 0, n = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev);
  return n;
}

// PACE_ERR_UNSUPPORTED: shapes beyond this kernel (the caller takes the CUDA-core one)
int span_mma(const pace_kv_pool_t* pl, int layer, const pace_step_t& st, const pace_attn_span_args_t& a, cudaStream_t s) {
  SpanParams p;
  const bool shared = pl->row_format == PACE_ROWS_SHARED;
  p.kv = make_view(pl, layer, nullptr);
  p.st = st;
  p.q = static_cast<const __nv_bfloat16*>(a.q);
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.slopes = a.slopes;
  p.sinks = a.sinks;
  p.q_elems = a.q_elems;
  p.out_elems = a.out_elems;
  p.H = a.n_q_heads;
  p.Gq = a.n_q_heads / pl->n_kv_heads;
  p.dv = a.vdim;
  p.dk16 = (a.dim + 15) / 16 * 16;
  p.dv16 = (a.vdim + 15) / 16 * 16;
  p.k_blocks = (a.dim + 63) / 64;
  p.v_blocks = shared ? 0 : (a.vdim + 63) / 64;
  p.entry0 = a.entry_begin;
  p.span = a.span;
  p.span_size = a.span_size;
  p.scale_log2 = a.scale * kLog2e;
  p.cap = score_cap(a.scale, a.softcap);
  p.out_row = span_out_row(a);
  // (q rows are read in pieces of eight: the caller keeps what lies between dim and the next multiple of 8 zero)
  if (pl->page_tokens != kKeys || a.q_elems % 8 || pl->head_dim % 8 || !aligned16(a.q) || !aligned16(pl->pages) ||
      ((uintptr_t)a.out & 7) || p.dv16 > 512 || (shared && p.dv16 > p.k_blocks * 64))
    return PACE_ERR_UNSUPPORTED;
  const int E = a.entry_end - a.entry_begin, rows = a.max_tokens * p.Gq, blocks = p.k_blocks + p.v_blocks, sms = sm_count();
  const int NG = p.dv16 <= 128 ? 1 : p.dv16 <= 256 ? 2 : 4;
  for (int MT = rows <= 16 ? 1 : rows <= 32 ? 2 : 4; MT; MT >>= 1) {
    int smem = 0, resident = 2;
    p.n_stages = 3;
    smem = span_smem(16 * MT, p.dk16, p.dv16, blocks, 3).total;
    if (smem > kSmemHalf || MT * NG > 4) {
      resident = 1;
      for (p.n_stages = 6; p.n_stages >= 2; --p.n_stages) {
        smem = span_smem(16 * MT, p.dk16, p.dv16, blocks, p.n_stages).total;
        if (smem <= kSmemMax) break;
      }
      if (p.n_stages < 2) continue;
    }
    const int tok = (16 * MT - 1) / p.Gq + 2;   // tokens a tile can touch
    int keys = a.max_keys;                      // visible keys of a tile, at most
    if (a.span != PACE_SPAN_ALL && (long long)a.span_size + tok < keys) keys = a.span_size + tok;
    const int tiles_k = keys / kKeys + 1, tiles = (rows + 16 * MT - 1) / (16 * MT);
    const long long units = (long long)tiles * pl->n_kv_heads * E;
    if ((long long)tiles * pl->n_kv_heads > 65535 || E > 65535) return PACE_ERR_UNSUPPORTED;
    // the share count that leaves the fewest tiles per block while all blocks are resident at once
    int ns = 1;
    for (int k = 2; k <= kMaxCluster && units * k <= (long long)resident * sms; ++k)
      if ((tiles_k + k - 1) / k < (tiles_k + ns - 1) / ns) ns = k;
    CUtensorMap tk, tv;
    const uint64_t row = (uint64_t)pl->head_dim;
    const uint64_t dims[3] = {row, kKeys, (uint64_t)pl->n_pages * pl->n_kv_heads}, str[2] = {row * 2, row * 2 * kKeys};
    const uint32_t box[3] = {64, kBoxRows, 1};
    int rc = tensor_map_bf16(&tk, p.kv.k, 3, dims, str, box);
    if (rc == PACE_OK) rc = tensor_map_bf16(&tv, p.kv.v, 3, dims, str, box);
    if (rc != PACE_OK) return rc;
#define PACE_SPAN_CASE(mt, ng) \
  if (MT == mt && NG == ng) return launch_span<mt, ng>(p, tk, tv, ns, tiles, E, smem, s);
    PACE_SPAN_CASE(1, 1) PACE_SPAN_CASE(1, 2) PACE_SPAN_CASE(1, 4)
    PACE_SPAN_CASE(2, 1) PACE_SPAN_CASE(2, 2) PACE_SPAN_CASE(2, 4)
    PACE_SPAN_CASE(4, 1) PACE_SPAN_CASE(4, 2) PACE_SPAN_CASE(4, 4)
#undef PACE_SPAN_CASE
  }
  return PACE_ERR_UNSUPPORTED;
}

}  // namespace
}  // namespace pace

using namespace pace;

extern "C" int pace_attn_span(const pace_kv_pool_t* p, int32_t layer, const pace_step_t* st, const pace_attn_span_args_t* a,
                              void* stream) {
  if (!p || !p->pages || !p->block_table || !step_ok(st) || layer < 0 || layer >= p->n_layers) return PACE_ERR_INVALID;
  if (!span_args_ok(st, a, p->n_kv_heads)) return PACE_ERR_INVALID;
  const int row = a->dtype == PACE_DTYPE_BF16 ? p->head_dim : p->head_dim / 2;
  if (a->dim > row || a->vdim > row || (p->row_format == PACE_ROWS_BF16 && a->dtype != PACE_DTYPE_BF16)) return PACE_ERR_INVALID;
  if (st->n_tokens == 0 || a->entry_begin == a->entry_end || a->max_tokens == 0) return PACE_OK;
  PACE_PROFILE("attn_span", stream, "layer=%d entries=%d tokens<=%d heads=%d dims=%d/%d", layer, a->entry_end - a->entry_begin,
               a->max_tokens, a->n_q_heads, a->dim, a->vdim);
  if (a->dtype == PACE_DTYPE_BF16) {
    int rc = attn_span_keys(p, layer, *st, *a, (cudaStream_t)stream);
    if (rc == PACE_ERR_UNSUPPORTED) rc = span_mma(p, layer, *st, *a, (cudaStream_t)stream);
    if (rc != PACE_ERR_UNSUPPORTED) return rc;
  }
  return attn_general_span(p, layer, *st, *a, (cudaStream_t)stream);
}
