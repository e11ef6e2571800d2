// State-space recurrence (decay per head and token) over many tokens, in chunks of 64 on the tensor cores.
//
// With l_i the sum of the log decays of the chunk's tokens up to i and S the state in front of the chunk:
//     out_i = e^(l_i) S^T c_i + sum_{j <= i} e^(l_i - l_j) dt_j (c_i . b_j) x_j + d_skip x_i
//     S' = e^(l_n) S + sum_j e^(l_n - l_j) dt_j b_j x_j^T
// b, c, x are bf16 values; everything else is fp32: the state stays in fp32 accumulators, and where an fp32 quantity is the
// operand of a bf16 product it is split into two or three bf16 terms whose sum carries 16 or 24 bits (weights and the state
// that is read: two, the b that enter the state with their decay and step: three).
//
// Blocks and segments as in lightning.cu: a block owns (entry, head, up to 128 value columns) and a segment of chunks;
// sequences that would leave the GPU half empty are cut into several segments, whose states a first launch and a prefix over
// them provide.
#include "ssd.cuh"

namespace pace {
namespace {

constexpr int kChunk = 64;

// `segments` blocks of seg_tokens tokens side by side, per launch: the first launch uses `ratio` times as many (it
// needs fewer registers, so more of its blocks are resident).
struct SegmentArgs {
  float* scratch;     // [entries][stored][heads][state][vdim]: what a segment adds, then the state in front of it
  float* log_decay;   // [entries][stored][heads]: a segment's sum of log decays
  int segments, seg_tokens;
  int stored, ratio;  // states in scratch per entry, and how many of them one segment of this launch spans
};

__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p)));
}
// 16 bytes global -> shared, zeros when `live` is false
__device__ __forceinline__ void copy16(void* dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
template <int DP, int VP, bool STATE_ONLY>
struct Tiles {
  static constexpr int QP = DP + 8, VQ = VP + 8;  // row pitches: 16 bytes beyond a power of two, ldmatrix without conflicts
  static constexpr int kK = 0, kV = kChunk * QP, kQ = kV + kChunk * VQ;           // one chunk: k, v, q
  static constexpr int kStage = STATE_ONLY ? kQ : kQ + kChunk * QP;
  static constexpr int kState = STATE_ONLY ? 0 : DP * VQ;                         // the state's high and low halves
  static constexpr int PP = kChunk + 8, kP = STATE_ONLY ? 0 : kChunk * PP;       // the weights' high and low halves
  static constexpr size_t bytes = sizeof(__nv_bfloat16) * (2 * kStage + 2 * kState + 2 * kP) + sizeof(float) * (2 * kChunk + 4);
  static constexpr int kThreads = STATE_ONLY ? 256 : 512;
};

template <int DP, int VP, bool STATE_ONLY>
__global__ void __launch_bounds__(STATE_ONLY ? 256 : 512, STATE_ONLY ? 2 : 1)
    ssd_chunk_kernel(pace_step_t st, pace_ssd_args_t a, SegmentArgs sg) {
  using TL = Tiles<DP, VP, STATE_ONLY>;
  constexpr int QP = TL::QP, VQ = TL::VQ, PP = TL::PP, kThreads = TL::kThreads;
  constexpr int RG = DP / 16, CG = kThreads / 32 / RG, SC = VP / CG;   // state tile of a warp: 16 rows x SC columns
  constexpr int NT = SC / 8;                               // its 8-column tiles
  constexpr int OT = VP / 32;                              // output tiles of a warp: 16 rows x a quarter of the columns
  extern __shared__ __align__(16) __nv_bfloat16 sm[];
  __nv_bfloat16* s_hi = sm + 2 * TL::kStage;
  __nv_bfloat16* s_lo = s_hi + TL::kState;
  __nv_bfloat16* p_hi = s_lo + TL::kState;
  __nv_bfloat16* p_lo = p_hi + TL::kP;
  float* ls = reinterpret_cast<float*>(p_lo + TL::kP);   // [kChunk] sums of log decays
  float* dts = ls + kChunk;                              // [kChunk] steps, zero behind the end

  const int e = blockIdx.z / sg.segments, seg = blockIdx.z % sg.segments, h = blockIdx.y, v0 = blockIdx.x * VP;
  const int d = a.state, vd = a.vdim, H = a.heads, g = h / (H / a.groups);
  const int t0 = st.cu[e], count = st.cu[e + 1] - t0, first = seg * sg.seg_tokens;
  if (first >= count) return;
  const int end = min(count, first + sg.seg_tokens);
  const bool last = end == count;
  if (STATE_ONLY && last) return;                          // nobody starts behind the last segment
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float neg_a = a.neg_a[h], dt_bias = a.dt_bias[h], skip = a.d_skip[h];
  float l_segment = 0.f;                                   // (kept by warp 0)

  const int inner = H * vd, b_at = inner + g * d, c_at = b_at + a.groups * d;
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(a.xbc) + (size_t)t0 * a.xbc_stride;
  float raw[2] = {0.f, 0.f};                               // warp 0: step projections of the next chunk
  auto fetch = [&](int l0, int buf) {
    __nv_bfloat16* stage = sm + buf * TL::kStage;
    constexpr int per = (2 * DP + VP) / 8;                 // 16-byte pieces of one token
    for (int i = tid; i < kChunk * per; i += kThreads) {
      const int j = i / per, p = i - j * per;
      const bool tok = l0 + j < end;
      const __nv_bfloat16* row = base + (size_t)(tok ? l0 + j : first) * a.xbc_stride;
      if (p < 2 * DP / 8) {
        const int which = p / (DP / 8), c = (p - which * (DP / 8)) * 8;
        if (STATE_ONLY && which == 0) continue;
        copy16(stage + (which == 0 ? TL::kQ : TL::kK) + j * QP + c, row + (which == 0 ? c_at : b_at) + (c < d ? c : 0), tok && c < d);
      } else {
        const int c = (p - 2 * DP / 8) * 8;
        copy16(stage + TL::kV + j * VQ + c, row + (size_t)h * vd + (v0 + c < vd ? v0 + c : 0),
               tok && v0 + c < vd);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (warp == 0) {
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int j = l0 + lane + 32 * k;
        raw[k] = j < end ? __bfloat162float(static_cast<const __nv_bfloat16*>(a.dt_raw)[(size_t)(t0 + j) * a.dt_stride + h]) : 0.f;
      }
    }
  };
  fetch(first, 0);

  // the state in front of the segment
  const int sr = (warp % RG) * 16 + (lane >> 2), sc = (warp / RG) * SC + (lane & 3) * 2;
  float S[NT][4];
  const float* from = nullptr;
  if (!STATE_ONLY) {
    if (sg.segments > 1) from = sg.scratch + (((size_t)e * sg.stored + seg * sg.ratio) * H + h) * d * vd;
    else if (st.start[e] != 0) from = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int r = sr + (q >> 1) * 8, c = v0 + sc + n * 8 + (q & 1);
      S[n][q] = (from && r < d && c < vd) ? from[(size_t)r * vd + c] : 0.f;
    }

  int buf = 0;
  for (int l0 = first; l0 < end; l0 += kChunk, buf ^= 1) {
    const int n_tok = min(kChunk, end - l0);
    __nv_bfloat16* q_s = sm + buf * TL::kStage + TL::kQ;
    __nv_bfloat16* k_s = sm + buf * TL::kStage + TL::kK;
    __nv_bfloat16* v_s = sm + buf * TL::kStage + TL::kV;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // the chunk is here, the previous one is done with
    if (warp == 0) {                                       // steps and sums of log decays
      float dt[2], l[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        dt[k] = lane + 32 * k < n_tok ? softplus_fast(raw[k] + dt_bias) : 0.f;
        l[k] = neg_a * dt[k];
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, l[0], o), y = __shfl_up_sync(0xffffffffu, l[1], o);
        if (lane >= o) l[0] += x, l[1] += y;
      }
      l[1] += __shfl_sync(0xffffffffu, l[0], 31);
#pragma unroll
      for (int k = 0; k < 2; ++k) ls[lane + 32 * k] = l[k], dts[lane + 32 * k] = dt[k];
      l_segment += __shfl_sync(0xffffffffu, l[1], 31);
    }
    if (!STATE_ONLY) {
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int q = 0; q < 4; q += 2) {
          uint32_t hi, lo;
          split_bf2(S[n][q], S[n][q + 1], hi, lo);
          const int at = (sr + (q >> 1) * 8) * VQ + sc + n * 8;
          *reinterpret_cast<uint32_t*>(s_hi + at) = hi;
          *reinterpret_cast<uint32_t*>(s_lo + at) = lo;
        }
    }
    __syncthreads();
    if (l0 + kChunk < end) fetch(l0 + kChunk, buf ^ 1);

    if (!STATE_ONLY) {
      // the four warps of 16 rows each score 16 keys, then own a quarter of the value columns
      const int m0 = (warp & 3) * 16, quarter = warp >> 2, c0 = quarter * (VP / 4);
      const int i0 = m0 + (lane >> 2);
      if (quarter <= (warp & 3)) {                         // (later keys are out of sight)
        float P[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n) P[n][0] = P[n][1] = P[n][2] = P[n][3] = 0.f;
#pragma unroll
        for (int k0 = 0; k0 < DP; k0 += 16) {
          uint32_t A[4], B[4];
          ldsm4(A, q_s + (m0 + (lane & 15)) * QP + k0 + (lane >> 4) * 8);
          ldsm4(B, k_s + (quarter * 16 + (lane & 7) + (lane >> 4) * 8) * QP + k0 + ((lane >> 3) & 1) * 8);
          mma16816(P[0], A, B[0], B[1]);
          mma16816(P[1], A, B[2], B[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int r = i0 + x * 8, j = quarter * 16 + n * 8 + (lane & 3) * 2;
            const float w0 = j <= r ? P[n][2 * x] * (exp_t<__nv_bfloat16>(ls[r] - ls[j]) * dts[j]) : 0.f;
            const float w1 = j + 1 <= r ? P[n][2 * x + 1] * (exp_t<__nv_bfloat16>(ls[r] - ls[j + 1]) * dts[j + 1]) : 0.f;
            uint32_t hi, lo;
            split_bf2(w0, w1, hi, lo);
            *reinterpret_cast<uint32_t*>(p_hi + r * PP + j) = hi;
            *reinterpret_cast<uint32_t*>(p_lo + r * PP + j) = lo;
          }
      }
      float O[OT][4];
#pragma unroll
      for (int n = 0; n < OT; ++n) O[n][0] = O[n][1] = O[n][2] = O[n][3] = 0.f;
#pragma unroll
      for (int k0 = 0; k0 < DP; k0 += 16) {
        uint32_t A[4], B[4];
        ldsm4(A, q_s + (m0 + (lane & 15)) * QP + k0 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < OT; n += 2) {
          const int at = (k0 + (lane & 15)) * VQ + c0 + n * 8 + (lane >> 4) * 8;
          ldsm4t(B, s_hi + at);
          mma16816(O[n], A, B[0], B[1]);
          mma16816(O[n + 1], A, B[2], B[3]);
          ldsm4t(B, s_lo + at);
          mma16816(O[n], A, B[0], B[1]);
          mma16816(O[n + 1], A, B[2], B[3]);
        }
      }
      const float f0 = exp_t<__nv_bfloat16>(ls[i0]), f1 = exp_t<__nv_bfloat16>(ls[i0 + 8]);
#pragma unroll
      for (int n = 0; n < OT; ++n) {
        O[n][0] *= f0; O[n][1] *= f0;
        O[n][2] *= f1; O[n][3] *= f1;
      }
      asm volatile("bar.sync %0, 128;" ::"r"(1 + (warp & 3)) : "memory");   // the weights of these rows are there
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk > (warp & 3)) break;
        uint32_t hi[4], lo[4], B[4];
        ldsm4(hi, p_hi + (m0 + (lane & 15)) * PP + kk * 16 + (lane >> 4) * 8);
        ldsm4(lo, p_lo + (m0 + (lane & 15)) * PP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < OT; n += 2) {
          ldsm4t(B, v_s + (kk * 16 + (lane & 15)) * VQ + c0 + n * 8 + (lane >> 4) * 8);
          mma16816(O[n], hi, B[0], B[1]);
          mma16816(O[n + 1], hi, B[2], B[3]);
          mma16816(O[n], lo, B[0], B[1]);
          mma16816(O[n + 1], lo, B[2], B[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (size_t)(t0 + l0) * a.out_stride + (size_t)h * vd;
#pragma unroll
      for (int n = 0; n < OT; ++n) {
        const int cc = c0 + n * 8 + (lane & 3) * 2, c = v0 + cc;   // (vdim is a multiple of 8: pairs are whole)
        if (c < vd) {
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int i = i0 + 8 * x;
            const float2 xv = bf2_to_f2(*reinterpret_cast<const uint32_t*>(v_s + i * VQ + cc));
            if (i < n_tok)
              *reinterpret_cast<uint32_t*>(out + (size_t)i * a.out_stride + c) =
                  f2_to_bf2(fmaf(skip, xv.x, O[n][2 * x]), fmaf(skip, xv.y, O[n][2 * x + 1]));
          }
        }
      }
    }

    // the state behind the chunk
    const float l_end = ls[kChunk - 1], fs = exp_t<__nv_bfloat16>(l_end);
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      S[n][0] *= fs; S[n][1] *= fs; S[n][2] *= fs; S[n][3] *= fs;
    }
    const int m0 = (warp % RG) * 16, c0 = (warp / RG) * SC;
#pragma unroll
    for (int k0 = 0; k0 < kChunk; k0 += 16) {
      uint32_t K[4], hi[4], mid[4], lo[4], B[4];
      ldsm4t(K, k_s + (k0 + (lane & 7) + (lane >> 4) * 8) * QP + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int j = k0 + (x >> 1) * 8 + (lane & 3) * 2;  // (keys beyond the chunk's end are zero)
        const float2 k = bf2_to_f2(K[x]);
        const float x0 = k.x * (exp_t<__nv_bfloat16>(l_end - ls[j]) * dts[j]),
                    x1 = k.y * (exp_t<__nv_bfloat16>(l_end - ls[j + 1]) * dts[j + 1]);
        hi[x] = f2_to_bf2(x0, x1);
        const float2 g = bf2_to_f2(hi[x]);
        split_bf2(x0 - g.x, x1 - g.y, mid[x], lo[x]);
      }
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        ldsm4t(B, v_s + (k0 + (lane & 15)) * VQ + c0 + n * 8 + (lane >> 4) * 8);
        mma16816(S[n], hi, B[0], B[1]);
        mma16816(S[n + 1], hi, B[2], B[3]);
        mma16816(S[n], mid, B[0], B[1]);
        mma16816(S[n + 1], mid, B[2], B[3]);
        mma16816(S[n], lo, B[0], B[1]);
        mma16816(S[n + 1], lo, B[2], B[3]);
      }
    }
  }

  float* to = nullptr;
  if (STATE_ONLY) {
    to = sg.scratch + (((size_t)e * sg.stored + seg) * H + h) * d * vd;
    if (tid == 0) sg.log_decay[((size_t)e * sg.stored + seg) * H + h] = l_segment;   // (every column block the same)
  } else if (last) to = a.s_state + ((size_t)st.slot[e] * H + h) * d * vd;
  if (!to) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int r = sr + (q >> 1) * 8, c = v0 + sc + n * 8 + (q & 1);
      if (r < d && c < vd) to[(size_t)r * vd + c] = S[n][q];
    }
}

// What the segments add -> the states in front of them, in place.
__global__ void ssd_prefix_kernel(pace_step_t st, pace_ssd_args_t a, SegmentArgs sg) {
  const int e = blockIdx.z, h = blockIdx.y, n = a.state * a.vdim;
  const int count = st.cu[e + 1] - st.cu[e];
  const int used = (count + sg.seg_tokens - 1) / sg.seg_tokens;
  const float* state = a.s_state + ((size_t)st.slot[e] * a.heads + h) * n;
  constexpr int kBatch = 8;                                // loads of a batch are in flight together
  const size_t step = (size_t)a.heads * n;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
    float s = st.start[e] != 0 ? state[i] : 0.f;
    float* p = sg.scratch + ((size_t)e * sg.stored * a.heads + h) * n + i;
    const float* ld = sg.log_decay + (size_t)e * sg.stored * a.heads + h;
    for (int r = 0; r < used; r += kBatch, p += kBatch * step) {
      float add[kBatch], f[kBatch];
#pragma unroll
      for (int j = 0; j < kBatch; ++j)
        if (r + j + 1 < used) add[j] = p[j * step], f[j] = ld[(size_t)(r + j) * a.heads];
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        if (r + j >= used) break;
        p[j * step] = s;
        if (r + j + 1 < used) s = fmaf(exp_t<__nv_bfloat16>(f[j]), s, add[j]);
      }
    }
  }
}

SegmentArgs plan_segments(int entries, int max_count, int heads, int vdim) {
  SegmentArgs s;
  s.scratch = s.log_decay = nullptr;
  const int blocks = entries * heads * ((vdim + 127) / 128);
  int want = 148 / (blocks > 0 ? blocks : 1);
  const int most = max_count / (4 * kChunk);               // a segment is worth its own blocks from four chunks on
  if (want > most) want = most;
  if (want < 1) want = 1;
  s.ratio = max_count / want >= 8 * kChunk ? 2 : 1;
  const int unit = s.ratio * kChunk;
  s.seg_tokens = ((max_count + want - 1) / want + unit - 1) / unit * unit;
  s.segments = (max_count + s.seg_tokens - 1) / s.seg_tokens;
  if (s.segments < 1) s.segments = 1;
  s.stored = s.segments * s.ratio;
  return s;
}
// the first launch's view: one segment per stored state
SegmentArgs state_segments(SegmentArgs s) {
  s.segments = s.stored;
  s.seg_tokens /= s.ratio;
  s.ratio = 1;
  return s;
}

template <int DP, int VP>
int launch_chunked(const pace_step_t& st, const pace_ssd_args_t& a, const SegmentArgs& sg, cudaStream_t s) {
  constexpr size_t smem = Tiles<DP, VP, false>::bytes, smem_state = Tiles<DP, VP, true>::bytes;
  const dim3 grid((unsigned)((a.vdim + VP - 1) / VP), (unsigned)a.heads, (unsigned)(st.n_entries * sg.segments));
  if (sg.segments > 1) {
    PACE_CUDA_TRY(cudaFuncSetAttribute(ssd_chunk_kernel<DP, VP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       (int)smem_state));
    const SegmentArgs ss = state_segments(sg);
    const dim3 grid_state(grid.x, grid.y, (unsigned)(st.n_entries * ss.segments));
    ssd_chunk_kernel<DP, VP, true><<<grid_state, 256, smem_state, s>>>(st, a, ss);
    PACE_LAUNCH_CHECK("ssd_chunk_kernel (states)");
    const int blocks = (a.state * a.vdim + 255) / 256;
    ssd_prefix_kernel<<<dim3((unsigned)(blocks < 64 ? blocks : 64), (unsigned)a.heads, (unsigned)st.n_entries), 256, 0, s>>>(
        st, a, ss);
    PACE_LAUNCH_CHECK("ssd_prefix_kernel");
  }
  PACE_CUDA_TRY(cudaFuncSetAttribute(ssd_chunk_kernel<DP, VP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                     (int)smem));
  ssd_chunk_kernel<DP, VP, false><<<grid, 512, smem, s>>>(st, a, sg);
  PACE_LAUNCH_CHECK("ssd_chunk_kernel");
  return PACE_OK;
}

}  // namespace

uint64_t ssd_scratch(const SegmentArgs& sg, int entries, int heads, int state, int vdim) {
  return sizeof(float) * (uint64_t)entries * sg.stored * heads * ((uint64_t)state * vdim + 1);
}

// bf16, sizes that the tiles cover and 16-byte pieces; everything else is the token-by-token kernel's
bool ssd_chunked_fits(const pace_ssd_args_t& a) {
  return a.dtype == PACE_DTYPE_BF16 && a.state <= 128 && a.state % 8 == 0 && a.vdim % 8 == 0 && a.xbc_stride % 8 == 0 &&
         a.out_stride % 2 == 0 && aligned16(a.xbc) && ((uintptr_t)a.out & 3) == 0;
}

int ssd_chunked(const pace_step_t& st, const pace_ssd_args_t& a, cudaStream_t s) {
  SegmentArgs sg = plan_segments(st.n_entries, st.max_count, a.heads, a.vdim);
  const uint64_t need = ssd_scratch(sg, st.n_entries, a.heads, a.state, a.vdim);
  if (sg.segments > 1 && (!a.workspace || a.workspace_bytes < need)) return PACE_ERR_INVALID;
  if ((int64_t)st.n_entries * sg.stored > 65535) return PACE_ERR_UNSUPPORTED;
  sg.scratch = a.workspace;
  sg.log_decay = a.workspace ? a.workspace + (size_t)st.n_entries * sg.stored * a.heads * a.state * a.vdim : nullptr;
  if (a.state <= 64) return a.vdim <= 64 ? launch_chunked<64, 64>(st, a, sg, s) : launch_chunked<64, 128>(st, a, sg, s);
  return a.vdim <= 64 ? launch_chunked<128, 64>(st, a, sg, s) : launch_chunked<128, 128>(st, a, sg, s);
}

}  // namespace pace

extern "C" uint64_t pace_ssd_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t state, int32_t vdim) {
  if (n_entries <= 0 || max_count <= 0 || heads <= 0 || state <= 0 || vdim <= 0) return 0;
  const pace::SegmentArgs sg = pace::plan_segments(n_entries, max_count, heads, vdim);
  return sg.segments > 1 ? pace::ssd_scratch(sg, n_entries, heads, state, vdim) : 0;
}
