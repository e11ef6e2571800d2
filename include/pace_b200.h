/*
 * pace_b200.h - C ABI of the B200 (sm_100a) KV-cache hot path.
 *
 * Every entry point takes plain pointers and sizes, returns an int status
 * (PACE_OK == 0) and never throws.  Device pointers are marked "device";
 * `stream` is a cudaStream_t passed as void*.  All work is stream-ordered: no
 * call synchronises unless it says so.
 *
 * The library replaces, for CUDA callers, what the reference does on the CPU in
 *   pace/llm/cache.py            (append, growth, rollback, beam gather)
 *   csrc/ops/attention.cpp       (the pace::attention custom op)
 *   csrc/ops/kernels/attention_kernels.cpp (the four-primitive SDPA sequence)
 * Each declaration cites the reference interface it stands in for.
 */
#ifndef PACE_B200_H_
#define PACE_B200_H_

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* ---- return codes (host side) ------------------------------------------ */
#define PACE_OK 0
#define PACE_ERR_INVALID 1     /* an argument failed validation; nothing was launched */
#define PACE_ERR_CUDA 2        /* the CUDA runtime reported an error (see pace_last_cuda_error) */
#define PACE_ERR_UNSUPPORTED 3 /* valid request outside what the kernels are built for */

/* ---- sticky device status bits (pool->status[0]) ----------------------- */
#define PACE_DEV_POOL_EXHAUSTED 1 /* reserve: free list ran dry                    */
#define PACE_DEV_OVER_REMOVE 2    /* truncate: remove_len > cached length          */
#define PACE_DEV_BAD_INDEX 4      /* a sequence slot / page id was out of range    */
#define PACE_DEV_TABLE_FULL 8     /* a sequence needs more pages than its table row*/
#define PACE_DEV_WAIT_TIMEOUT 16  /* a bounded in-kernel wait gave up               */

/*
 * Paged KV pool descriptor.  Geometry + device pointers; plain data, copied by
 * value into kernels.  Storage may come from pace_kv_pool_create() or from the
 * caller (pace_kv_pool_bytes + pace_kv_pool_bind, e.g. a torch allocation).
 *
 *   pages        bf16 [n_layers][2 (K,V)][n_pages][n_kv_heads][page_tokens][head_dim]
 *   block_table  int32 [max_seqs][max_pages_per_seq]  logical page -> physical page
 *   seq_len      int32 [n_layers][max_seqs]  cached tokens, per layer
 *                (the reference keeps one seq_len per layer object, cache.py:184)
 *   seq_pages    int32 [max_seqs]   pages a slot owns; capacity = seq_pages*page_tokens
 *   page_ref     int32 [n_pages]    reference counts (beam gather shares pages)
 *   free_stack   int32 [n_pages]    free physical pages; counters[0] = number free
 *   counters     int32 [8 + n_layers] [0] free pages, [2] pages shared after a gather, [8 + layer] append ticket
 *   status       int32 [4]          [0] sticky PACE_DEV_* bits
 *   table_tmp    int32 [max_seqs][max_pages_per_seq + 1]   scratch of pace_kv_gather
 *
 * row_tokens: consecutive tokens that share a row (0 or 1: a row per token).  A pool of pooled blocks has one row for every
 * row_tokens tokens; lengths and page_tokens (a multiple of row_tokens) stay counts of tokens, so that such a pool is
 * reserved, released and gathered with the calls and numbers of the token pool beside it, and a page has
 * page_tokens / row_tokens rows.
 *
 * page_tokens is the physical page size (the Python host uses 64: one page is one K/V chunk of
 * the attention kernels).  The reference's capacity (whole `tokens_per_split` segments,
 * cache.py:177-181, 292-313) is host bookkeeping on top of the pages and does not depend on it;
 * a page of exactly tokens_per_split tokens makes the two coincide.
 *
 * Between calls the pool's memory belongs to the library: only its kernels write it.
 */
typedef struct pace_kv_pool {
  int32_t n_layers, n_kv_heads, head_dim, page_tokens;
  int32_t n_pages, max_seqs, max_pages_per_seq, owns_memory;
  void* pages;          /* device */
  int32_t* block_table; /* device */
  int32_t* seq_len;     /* device */
  int32_t* seq_pages;   /* device */
  int32_t* page_ref;    /* device */
  int32_t* free_stack;  /* device */
  int32_t* counters;    /* device */
  int32_t* status;      /* device */
  int32_t* table_tmp;   /* device */
  int32_t row_format;   /* PACE_ROWS_*: 0 = bf16 rows of 64 or 128 */
  int32_t row_tokens;   /* 0, 1: a row per token */
} pace_kv_pool_t;

const char* pace_last_cuda_error(void);
const char* pace_version(void);

/* ---- pool lifetime ------------------------------------------------------
 * Reference: BMCKVCache.__init__ / _create_new_segment allocate torch buffers
 * (pace/llm/cache.py:175-193, 242-266); here one pool per model instance is
 * carved into pages once and segments become block-table entries. */
int pace_kv_pool_bytes(const pace_kv_pool_t* geom, uint64_t* pages_bytes, uint64_t* meta_bytes);
int pace_kv_pool_bind(pace_kv_pool_t* pool, void* pages_mem, void* meta_mem); /* host-only pointer carving */
int pace_kv_pool_create(pace_kv_pool_t* pool);  /* cudaMalloc for pages+meta of the filled-in geometry, then reset */
int pace_kv_pool_destroy(pace_kv_pool_t* pool); /* frees what pace_kv_pool_create allocated */
int pace_kv_pool_reset(const pace_kv_pool_t* pool, void* stream); /* all slots empty, all pages free */
/* Sticky status and the kernels' bounded waits.  Every in-kernel wait (on a ring stage, on a result
 * slot) gives up after about a quarter of a second, raises PACE_DEV_WAIT_TIMEOUT and lets its thread
 * block return; the first wait of a block to give up also releases the block's other waits, so a block
 * leaves after one such interval, not one per role.  While the bit stands, every later attention launch
 * on the pool returns at once without touching its output: the host reads the word
 * (pace_kv_pool_query), deals with the cause and clears it (pace_kv_pool_clear_status) to restore
 * service.  (No counterpart in the reference, which has no device.)
 *
 * pace_selftest_wait_timeout makes one wait run out on purpose, harmlessly: a one-block kernel waits on
 * a barrier nobody arrives on for about limit_us microseconds (1 .. 1e6), gives up and raises the bit
 * on this pool.  For health checks and for testing the host's handling of the bit. */
int pace_selftest_wait_timeout(const pace_kv_pool_t* pool, int32_t limit_us, void* stream);
/* Synchronising read of {status bits, free pages, 0, 0}. */
int pace_kv_pool_query(const pace_kv_pool_t* pool, int32_t out[4], void* stream);
int pace_kv_pool_clear_status(const pace_kv_pool_t* pool, void* stream);

/* Give back every page of the listed slots and zero their lengths (all layers).
 * Reference: cache objects are dropped with the manager (generator.py:396-410). */
int pace_kv_seq_release(const pace_kv_pool_t* pool, const int32_t* seq_ids /*device*/, int32_t batch, void* stream);

/* ---- append -------------------------------------------------------------
 * Reference: BMCKVCache.update_cache / DynamicKVCache.update_cache
 * (pace/llm/cache.py:268-326, 370-400).
 *
 * pace_kv_reserve makes sure every listed slot owns ceil((seq_len[layer]+n)/page_tokens)
 * pages (popping the free list; copy-on-write of a shared last page after a beam
 * gather).  pace_kv_append copies n new K/V rows per sequence into the slots
 * [seq_len, seq_len+n) and then advances seq_len[layer].  k_new / v_new are bf16
 * [batch][n_kv_heads][n_new][head_dim] addressed through element strides (the last
 * dimension is contiguous), so the transposed view a model produces needs no copy.
 * n_new_per_seq (device, optional) gives ragged counts <= n_new. */
int pace_kv_reserve(const pace_kv_pool_t* pool, int32_t layer, const int32_t* seq_ids, int32_t batch,
                    int32_t n_new, const int32_t* n_new_per_seq, void* stream);
int pace_kv_append(const pace_kv_pool_t* pool, int32_t layer, const int32_t* seq_ids, int32_t batch,
                   int32_t n_new, const int32_t* n_new_per_seq, const void* k_new, const void* v_new,
                   int64_t stride_b, int64_t stride_h, int64_t stride_t, void* stream);
/* Ordering of the two append entry points against an attention launch in front of them on the
 * stream: the library remembers, per stream, the pool and layer its newest attention launch reads.
 * An append to ANOTHER layer (the decoder-layer pattern attn(l), append(l+1), attn(l+1)) starts
 * while that launch is still running (programmatic dependent launch) - it touches nothing the
 * launch reads.  An append to the SAME pool and layer, or a pace_kv_append_rope whose q_out is the
 * q of that launch, is ordered behind its completion like any other kernel. */

/* One launch for a whole decode step: the rows of layers [layer_begin, layer_end) at once.
 * Reference: the same BMCKVCache.update_cache (cache.py:268-326), called once per layer per
 * generated token (llama.py:159); here the per-layer calls of a step collapse into one kernel that
 * runs after the step's last attention launch, which is possible because the attention entry
 * points can take the step's new row straight from the caller's buffer (PACE_ATTN_PENDING_ROW).
 * k_new / v_new are bf16 [layer][batch][n_kv_heads][n_new][head_dim] through element strides
 * (stride_l first; head_dim contiguous, rows 16-byte aligned); layer `layer_begin` is at offset 0.
 * Every listed layer's seq_len advances by the same counts.  pace_kv_reserve for the step must have
 * run (any one layer: pages are shared by all layers).  k_new = v_new = NULL advances the lengths
 * only: for a step whose rows every layer's attention launch has stored already
 * (PACE_ATTN_PENDING_ROW).  The kernel is ordered behind everything in
 * front of it on the stream and in front of everything behind it (no programmatic overlap). */
int pace_kv_append_layers(const pace_kv_pool_t* pool, int32_t layer_begin, int32_t layer_end,
                          const int32_t* seq_ids, int32_t batch, int32_t n_new, const int32_t* n_new_per_seq,
                          const void* k_new, const void* v_new, int64_t stride_l, int64_t stride_b,
                          int64_t stride_h, int64_t stride_t, void* stream);

/* ---- RoPE + append in one pass -----------------------------------------------
 * Reference: the step in front of the append in every decoder layer,
 * pace/llm/models/llama.py:130-165: q/k/v are viewed as heads, RotaryEmbedding's
 * callable rotates q and k (pace/ops/rotary_embedding.py:375-441: table rows picked
 * by position id, cast to the activations' dtype, NeoX halves or GPT-J pairs, every
 * product and sum rounded to that dtype), then update_cache stores k and v.
 *
 * pace_kv_append_rope reads the projection outputs once, writes the rotated queries
 * to q_out (which may be q itself) and the rotated keys and the values straight into
 * the slots [seq_len, seq_len + n) of the paged cache, then advances seq_len[layer]
 * as pace_kv_append does (pace_kv_reserve must have run).  All tensors are bf16
 * addressed as [batch][token][head][head_dim] through element strides (head_dim
 * contiguous, 16-byte aligned rows): the untransposed output of a fused or split
 * QKV projection needs no copy.  cos/sin are the operator's fp32 tables
 * [table_rows][rotary_dim / 2]; table_row[b * row_stride_b + t] names the row of
 * token t of sequence b (the position id, already shifted for longrope).
 * rotary_dim <= head_dim, a multiple of 16; elements beyond it pass through.
 * A row index outside the table raises PACE_DEV_BAD_INDEX and leaves that token
 * unrotated. */
typedef struct {
  const void* q;        int64_t q_stride_b, q_stride_t, q_stride_h;
  const void* k;        int64_t k_stride_b, k_stride_t, k_stride_h;
  const void* v;        int64_t v_stride_b, v_stride_t, v_stride_h;
  void* q_out;          int64_t o_stride_b, o_stride_t, o_stride_h;
  const int32_t* table_row; /* device */
  int64_t row_stride_b;
  const float* cos_table;   /* device, fp32 [table_rows][rotary_dim / 2] */
  const float* sin_table;
  int32_t table_rows;
  int32_t rotary_dim;
  int32_t gptj_pairs;       /* 0: NeoX halves (d, d + rotary_dim / 2); 1: GPT-J pairs (2d, 2d + 1) */
  int32_t n_q_heads;
  /* Deferred append (decode steps): when k_stage is not NULL the rotated keys and the values go to
   * these staging rows, bf16 [batch][n_kv_heads][token][head_dim] through element strides, instead of
   * the pool, and seq_len is left alone - the rows then ride along with the layer's decode launch
   * (PACE_ATTN_PENDING_ROW) and are committed by pace_kv_append_layers. */
  void* k_stage;
  void* v_stage;
  int64_t stage_stride_b, stage_stride_h, stage_stride_t;
} pace_rope_args_t;
int pace_kv_append_rope(const pace_kv_pool_t* pool, int32_t layer, const int32_t* seq_ids, int32_t batch,
                        int32_t n_new, const int32_t* n_new_per_seq, const pace_rope_args_t* rope, void* stream);

/* ---- rollback -------------------------------------------------------------
 * Reference: BMCKVCache.remove_cache (cache.py:224-240): seq_len -= n, pages kept,
 * data untouched.  Over-removal leaves the length alone and raises
 * PACE_DEV_OVER_REMOVE.  layers [layer_begin, layer_end).  remove_per_seq (device,
 * optional) overrides the scalar per sequence (PARD with per-sequence acceptance). */
int pace_kv_truncate(const pace_kv_pool_t* pool, int32_t layer_begin, int32_t layer_end,
                     const int32_t* seq_ids, int32_t batch, int32_t remove_len,
                     const int32_t* remove_per_seq, void* stream);

/* ---- PARD acceptance ---------------------------------------------------------
 * Reference: Generator._postprocess_speculated_tokens (pace/llm/generator.py:669-713), one sequence
 * at a time on the host there.  Per sequence b of the batch: accept the leading matches among the
 * first d - 1 draft tokens (draft i is accepted while target_next[b][i] == drafts[b][i] and
 * i < n_target[b]; with `forced` given, while forced[b][i] != 0 instead), always keep one more token
 * (the target's own), and say how far the two caches roll back:
 *     keep[b]          = 1 + accepted                                  in [1, d]
 *     target_remove[b] = d - keep + 1  if keep < d,  else 0            (generator.py:696-702)
 *     draft_remove[b]  = d - 1                                         (generator.py:706)
 *     kept[b][0 .. keep)  the tokens that join the history: the accepted ones (the target's tokens;
 *                         the drafts when acceptance is forced) and then target_next[b][min(keep - 1, n_target[b] - 1)]
 * The arrays feed pace_kv_truncate (remove_per_seq) and the next step's ragged counts directly:
 * nothing of a speculative step has to come back to the host.  drafts int64 [batch][d], target_next
 * int64 [batch][d + 1] (n_target[b] of them valid), forced uint8 [batch][d - 1] or NULL, kept int64
 * [batch][d]; all device. */
int pace_pard_accept(const int64_t* drafts, const int64_t* target_next, const int32_t* n_target,
                     const uint8_t* forced, int32_t batch, int32_t d, int32_t* keep, int32_t* target_remove,
                     int32_t* draft_remove, int64_t* kept, void* stream);

/* ---- beam gather ----------------------------------------------------------
 * Reference: KVCacheBase.update_cache_with_beam_indices (cache.py:161-167):
 * row i of the batch becomes a copy of old row beam_idx[i].  Index-only here: the
 * block-table rows and lengths are permuted and page reference counts adjusted. */
int pace_kv_gather(const pace_kv_pool_t* pool, const int32_t* seq_ids, const int64_t* beam_idx /*device*/,
                   int32_t batch, void* stream);

/* ---- cache read-back --------------------------------------------------------
 * Materialises what the reference's update_cache returns (cache.py:326): dense
 * bf16 [batch][n_kv_heads][cap_tokens][head_dim] K and V, rows beyond a slot's
 * pages zero-filled. */
int pace_kv_read_dense(const pace_kv_pool_t* pool, int32_t layer, const int32_t* seq_ids, int32_t batch,
                       void* k_out, void* v_out, int32_t cap_tokens, void* stream);

/* ---- attention --------------------------------------------------------------
 * Reference: pace::attention (csrc/ops/attention.cpp:18-97, schema :104-108) and
 * kernels::attention_kernel Method 1 (csrc/ops/kernels/attention_kernels.cpp:218-257):
 * softmax(Q K^T / sqrt(D) + mask) V with fp32 accumulation, output in Q's dtype.
 *
 * Paged form: K/V come from the pool (layer, slots); the additive mask of the
 * reference (causal tail + left padding + BMC padding columns, llama.py:294-310)
 * is expressed by integers: kv_len = seq_len[layer][slot] (the q_len newest
 * tokens included), query i sees keys [kv_start, kv_len - q_len + i].
 * q / out are bf16 [batch][n_q_heads][q_len][head_dim] through element strides.
 * GQA: n_q_heads = G * n_kv_heads, query head h reads KV head h / G, which is
 * what the reference obtains by repeat_kv before caching (llama.py:152-158). */
typedef struct pace_attn_args {
  const pace_kv_pool_t* pool;
  int32_t layer;
  int32_t batch;
  int32_t n_q_heads;
  int32_t q_len;            /* 1 = decode; d+1 = verify; chunk = prefill */
  const int32_t* seq_ids;   /* device [batch]; NULL = slots 0..batch-1 */
  const int32_t* kv_start;  /* device [batch] or NULL (no left padding) */
  const int32_t* q_lens;    /* device [batch] or NULL: ragged query counts <= q_len */
  const void* q;
  int64_t q_stride_b, q_stride_h, q_stride_s;
  void* out;
  int64_t o_stride_b, o_stride_h, o_stride_s;
  float scale;              /* 0 -> 1/sqrt(head_dim) */
  void* workspace;          /* device scratch, pace_attn_workspace_bytes(); zero it once after allocation */
  uint64_t workspace_bytes;
  uint32_t flags;           /* PACE_ATTN_* bits, 0 = none */
  /* PACE_ATTN_PENDING_ROW only: the step's new K and V row of every (sequence, kv head), bf16
   * [batch][n_kv_heads][head_dim] through element strides (head_dim contiguous, rows 16-byte aligned). */
  const void* k_pending;
  const void* v_pending;
  int64_t pending_stride_b, pending_stride_h;
  /* At most this many thread blocks (a caller that shares the GPU with work on another stream);
   * 0 = the kernels' own choice, one per SM or two for the four-warp decode form.  Any value gives
   * the same result: the kernels cut the work into as many contiguous ranges as there are blocks. */
  int32_t max_ctas;
} pace_attn_args_t;

/* Never cut one (sequence, KV head) stream of keys across thread blocks.  The kernels normally decide
 * this on the device from the cached lengths: cutting balances ragged batches, but the pieces meet in
 * the workspace, and because the host cannot know the outcome a K/V append launched behind the
 * attention launch has to hold its completion until that launch has completed (the next attention
 * launch orders itself after the append only).  A launch with this bit set touches no workspace, the
 * append behind it completes on its own, and the next layer's attention launch learns of this one's
 * completion directly: about 0.5 us less per layer.  Set it when batch * n_kv_heads is not small
 * against the number of SMs and the lengths are about even (the host mirror of the reference's one
 * seq_len per layer, cache.py:184, is enough to tell).  It only changes the schedule, never the result. */
#define PACE_ATTN_WHOLE_UNITS 1u

/* Decode (q_len == 1) over the cache PLUS one row per sequence that is not in the cache yet: the
 * launch first stores k_pending / v_pending in the row's slot of the pool - row number seq_len of
 * the sequence, whose page pace_kv_reserve must have provided - and then attends over keys
 * [kv_start, seq_len].  seq_len itself is NOT advanced.  The result is what pace_kv_append of that
 * row followed by a plain decode launch gives.  This takes the per-layer append out of the chain of
 * a decode step (llama.py:159-165 does update_cache, then attention, in every layer): the rows stay
 * in the caller's staging buffer, every layer's attention launch follows the previous layer's
 * directly, and one pace_kv_append_layers after the last layer advances all layers' lengths (it
 * stores the rows again, which changes nothing).  A row that is never committed is simply a stale
 * row beyond seq_len, as after a rollback.  Served by the tensor-core kernels for every group size
 * below 33 query heads per KV head; PACE_ERR_UNSUPPORTED otherwise. */
#define PACE_ATTN_PENDING_ROW 2u

/* Decode launches normally begin by waiting for the kernel in front of them on the stream
 * (a programmatic dependent launch: only the set-up overlaps).  When the library knows that its own
 * newest launch on the stream was an attention launch - so nothing of the pool this launch reads
 * (lengths, block table, pages) can have been written by the kernel directly in front - a
 * whole-unit decode launch starts streaming K/V pages at once and waits only before it touches q,
 * the pending rows and out.  The K/V stream then runs beside the tail of the kernel in front (the
 * previous layer's attention, or the projection that produces q).  This bit forbids that: set it
 * if seq_ids, kv_start or the pool were written by a kernel of your own directly in front. */
#define PACE_ATTN_NO_EARLY_KV 4u

/* Decode: keep the form with eight consumer warps and one thread block per SM (the kernels fall
 * back to it by themselves when the workspace or shared memory has no room for two blocks per SM). */
#define PACE_ATTN_ONE_CTA_PER_SM 8u

/* The softmax weights enter the product with V as two bf16 terms (high and low, 16 bits of mantissa together)
 * instead of one rounded to bf16, and every exponential is good to fp32's last bits: for models that want weights
 * kept in 32-bit.  Costs one more tensor-core product per key; the cache is read once all the same.  Not for
 * tiles of 33 query rows and more whose output rows are not 16-byte aligned, nor for an additive mask.  (The CUDA-core
 * decode kernel keeps its weights in fp32 anyway.) */
#define PACE_ATTN_SPLIT_WEIGHTS 16u

uint64_t pace_attn_workspace_bytes(int32_t batch, int32_t n_q_heads, int32_t n_kv_heads, int32_t head_dim,
                                   int32_t q_len);
/* q_len == 1.  The grouped query heads of a KV head are packed into one mma.sync tile (any group
 * size); groups of 1 or 2 (plain multi-head attention) run on the CUDA-core kernel instead, whose
 * packed fp32 FMAs cost less than a tile that is seven eighths padding. */
int pace_attn_decode(const pace_attn_args_t* a, void* stream);
/* The CUDA-core decode kernel whatever the group size (1, 2, 4 or 8 query heads per KV head;
 * PACE_ERR_UNSUPPORTED otherwise): 8 lanes per K/V row, packed fp32 FMAs, warp-shuffle online
 * softmax - the form the reference's head-by-head CPU loop maps to most directly.  pace_attn_decode
 * picks it only for groups of 1 or 2; pace_attn_verify with q_len = 1 is the tensor-core form. */
int pace_attn_decode_cuda_cores(const pace_attn_args_t* a, void* stream);
/* q_len >= 1 query tokens per sequence, causal among themselves (PARD verify: d + 1 tokens; a
 * prefill chunk: hundreds).  Tiles of 33 and more query rows (tokens x grouped heads) run on the
 * tcgen05 tensor cores, smaller ones on mma.sync.  pace_attn_prefill is the same entry point under
 * the name the chunked-prefill caller expects. */
int pace_attn_verify(const pace_attn_args_t* a, void* stream);
int pace_attn_prefill(const pace_attn_args_t* a, void* stream);

/* Decode attention without any allocation.  (No counterpart in the reference: its CPU op
 * allocates its score tensor on every call, attention_kernels.cpp:222-226.)
 *
 * For hosts that cannot allocate device memory where a decode step runs - an engine that owns the
 * whole device and lends this library nothing, a serving loop whose memory was fixed at start-up,
 * a thread that must not enter the allocator - and so cannot supply pace_attn_decode's workspace.
 * Same arguments and result as pace_attn_decode; `workspace` / `workspace_bytes` are ignored and
 * the scratch is a fixed device array inside the library (about 3.4 MB per GPU, held until the
 * process exits).  Limits, refused with PACE_ERR_UNSUPPORTED beyond them: at most 16 query heads per
 * KV head, head_dim <= 128, batch * n_kv_heads <= 65536, at most 192 SMs.  The first call on a device
 * resolves the array's address there (make it before any stream capture) and keeps it for the life
 * of the process: after a cudaDeviceReset the kept address is stale and the entry point must not be
 * used again in that process.  Calls share the array: issue them on one stream, or otherwise keep
 * them from overlapping on the GPU. */
int pace_attn_decode_static(const pace_attn_args_t* a, void* stream);

/* Dense form with the reference op's exact operands: q [B,N,S,H], k/v [B,Nkv,L,H]
 * contiguous bf16, additive mask [B,1,mask_rows,L] (mask_rows 1 or S; bf16 or fp32;
 * may be NULL), out [B,N,S,H].  Reference: pace::attention, attention.cpp:18-97. */
int pace_attention_dense(const void* q, const void* k, const void* v, const void* mask, int32_t mask_is_fp32,
                         int32_t mask_rows, void* out, int32_t B, int32_t N, int32_t Nkv, int32_t S, int32_t L,
                         int32_t H, void* workspace, uint64_t workspace_bytes, void* stream);

/* ---- op timing -------------------------------------------------------------------
 * Reference: PROFILE_PACE_FUNCTION / TimingLogger (csrc/core/logging.h:144-212, used at
 * csrc/ops/attention.cpp:24), switched on by the environment variable PACE_LOG_LEVEL=profile.
 * With that value set when the library is loaded, the attention, append, rollback, gather and linear
 * entry points record a CUDA event on their stream before and after their launches and a line
 *     [PACE profile] pace::<op>,<shapes>,<milliseconds>
 * goes to stderr once both events have completed: at a later profiled call, at pace_profile_flush
 * (which waits for the outstanding ones and returns how many it wrote or dropped) or at process exit.
 * The time is device time between the two events.  Calls made while their stream is being captured
 * into a CUDA graph are not timed.  No other value of the variable changes anything. */
int pace_profile_enabled(void);
int pace_profile_flush(void);

/* ---- weight-streaming linear layer for decode steps ------------------------------
 * Reference: the Linear operator's GEMM back ends on a decoder layer's projections and MLP
 * (pace/ops/backends/tpp.py:19-63, pace/ops/backends/imbps.py:19-92, csrc/ops/libxsmm_linear.cpp:225-241).
 * y[M][N] = x[M][K] w[N][K]^T, bf16 in and out, fp32 accumulation, no bias; M <= 32 tokens, N and K
 * multiples of 128 (PACE_ERR_UNSUPPORTED otherwise: larger token counts are compute-bound and belong to
 * a library GEMM).  Row pitches are in elements (x_stride, w_stride multiples of 8, bases 16-byte
 * aligned).  `workspace` is pace_linear_workspace_bytes(largest N) bytes of 32-byte aligned device memory, zeroed once
 * after allocation and not shared by launches that can overlap on the GPU (one per stream); the kernel
 * leaves it zeroed.  `status` (device, may be NULL) takes PACE_DEV_WAIT_TIMEOUT if a bounded wait runs
 * out.  Launched as a programmatic dependent: the weights are fetched while the kernel in front still
 * runs, only x waits for it. */
uint64_t pace_linear_workspace_bytes(int32_t n_max);
int pace_linear_skinny(const void* x, int64_t x_stride, const void* w, int64_t w_stride, void* y, int64_t y_stride,
                       int32_t M, int32_t N, int32_t K, void* workspace, uint64_t workspace_bytes, int32_t* status,
                       void* stream);

/* ==== layers of hybrid decoders (attention beside recurrent layers) =====================================
 * Building blocks for models whose layers are not all softmax attention over the pool: fused norms, the
 * append of normalised keys, an attention kernel for any row format, short convolutions, gated linear
 * recurrences and decayed linear attention.  They work on a step's tokens packed back to back ([n_tokens]
 * rows, all sequences), described by pace_step_t.  `dtype` is the type of activations, projection outputs
 * and cache rows: PACE_DTYPE_BF16 or PACE_DTYPE_FP32; the residual stream, norms, gates, attention scores
 * and recurrent states are fp32 with either.  (No counterpart in the reference, which serves attention-only
 * decoders.) */
#define PACE_DTYPE_BF16 0
#define PACE_DTYPE_FP32 1

/* Values of pace_kv_pool_t::row_format.
 * PACE_ROWS_BF16: K and V rows are head_dim bf16 values, head_dim 64 or 128; every entry point takes them.
 * PACE_ROWS_OPAQUE: rows are head_dim 16-bit units of any content (head_dim a multiple of 8, at most 2048):
 * fp32 rows, other head sizes.  The allocator's entry points (reserve, release, truncate, gather,
 * append_layers without rows, query), pace_kv_append_norm, pace_attn_general and pace_attn_span take them; the rest
 * answers PACE_ERR_UNSUPPORTED.
 * PACE_ROWS_SHARED: as PACE_ROWS_OPAQUE, but a layer has one row per token and head, which is its key and, with its
 * first elements, its value (latents): pages are [layer][page][kv_head][page_tokens][head_dim], half the memory.
 * pace_kv_append_norm does not take them (pace_latent_append writes them). */
#define PACE_ROWS_BF16 0
#define PACE_ROWS_OPAQUE 1
#define PACE_ROWS_SHARED 2

/* The tokens of one step.  Entry e (a sequence that takes part) owns rows [cu[e], cu[e + 1]); its first
 * token has position start[e]; `slot` is its slot in the pool and in the recurrent states.  A state is
 * never cleared: an entry with start[e] == 0 begins from zeros whatever its slot holds.  All device. */
typedef struct pace_step {
  int32_t n_tokens, n_entries, max_count; /* max_count: most tokens any entry has */
  int32_t reserved;
  const int32_t* token;     /* [n_tokens] token ids (embedding lookup) */
  const int32_t* tok_entry; /* [n_tokens] */
  const int32_t* tok_pos;   /* [n_tokens] position in the sequence */
  const int32_t* q_row;     /* [n_tokens] row of the attention staging buffers the token uses */
  const int32_t* cu;        /* [n_entries + 1] */
  const int32_t* start;     /* [n_entries] */
  const int32_t* slot;      /* [n_entries] */
} pace_step_t;

/* One pass over the residual stream x (fp32 [n_tokens][width]) between two sublayers:
 *     x' = (restart ? 0 : x) + rms(y) * w_post + (embed ? embed[token] * embed_scale : 0)
 *     h  = rms(x') * w_next,       rms(z) = z / sqrt(mean(z^2) + eps)
 * y (the sublayer's output) may be NULL, embed may be NULL (with restart and embed it is the embedding
 * lookup in front of the first layer; with y and embed the re-injection of the embeddings between two
 * passes of a loop), w_next / h may be NULL; h without w_next takes x' as it is (sublayers that read the stream
 * itself).  w_post == NULL adds y as it is.  Norm weights are fp32 [width] and used as weight_offset + w (1 for
 * "one plus weight" norms).  embed is dtype [vocab][width].
 * With `top` > 0, y holds the rows of a mixture's experts (pace_moe_experts) and the sublayer's output of token t is
 *     sum over k < top of slot_weight[t][k] * y[expert_row(slot_expert[t][k], slot_rank[t][k])],
 * where a slot_expert of n_experts or more names an identity expert: its row is identity[t].
 * Further terms: `add` (rows of add_stride elements) and y_bias (fp32 [width]) are added to the sublayer's output; with
 * y_mul != 1 and no w_post the sum is multiplied by it; embed_norm normalises the embedding row (rms(row) * weight, in place of
 * embed_scale).  h2 takes a second normalisation of the same x', with the weight w_next2. */
typedef struct {
  float* x;
  const void* y;
  const float* w_post;
  const void* embed;
  const float* w_next;
  void* h;
  int64_t y_stride;
  int32_t width, vocab, restart, dtype;
  float eps, weight_offset, embed_scale;
  int32_t top, n_experts;
  const int32_t* slot_expert;   /* [n_tokens][top], with top > 0 */
  const int32_t* slot_rank;     /* [n_tokens][top] */
  const float* slot_weight;     /* [n_tokens][top] */
  const int32_t* expert_count;  /* [n_experts] */
  const void* identity;         /* dtype [n_tokens][width] */
  const void* add;
  int64_t add_stride;
  const float* y_bias;
  const float* embed_norm;
  const float* w_next2;
  void* h2;
  float y_mul;
} pace_residual_norm_args_t;
int pace_residual_norm(const pace_step_t* step, const pace_residual_norm_args_t* a, void* stream);

/* Projection output -> attention operands, in one pass per token: RMS norm of the whole query and the whole
 * key projection (q_norm / k_norm fp32 weights over all heads; NULL = no norm), queries times
 *     q_mul * (1 + temp_coef * ln(floor((pos + 1) / temp_every) + 1))        (temp_coef 0: no temperature)
 * to q_out rows [q_row][n_q_heads][row elements], keys and values into the pages of pool layer `layer` at
 * positions tok_pos.  The pages must be reserved; lengths are left alone (pace_kv_append_layers without rows
 * advances them).  qkv is dtype [n_tokens][qkv_stride]: q (n_q_heads x dim), k (kv_heads x dim), v (kv_heads
 * x vdim).  A pool row holds max(dim, vdim) or more elements; what a row has beyond dim / vdim is zeroed.
 * per_head: the norms are taken over each head's dim elements instead, without weights (q_norm and k_norm NULL), and
 * row t of q_out belongs to token t (no staging rows). */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const float* q_norm;
  const float* k_norm;
  void* q_out;
  int32_t n_q_heads, dim, vdim, dtype;
  float eps, q_mul, temp_coef;
  double temp_every;
  int32_t per_head;
} pace_append_norm_args_t;
int pace_kv_append_norm(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step,
                        const pace_append_norm_args_t* a, void* stream);

/* Projection output -> attention operands behind short causal convolutions, in one pass: every channel of q, k and v is
 * convolved over time (taps, ring as pace_causal_conv, without bias), then q and k are normalised per head,
 *     rms over dim * q_norm[c] (k_norm[c]; fp32 [dim], shared by the heads)
 * and their pairs (2i, 2i + 1), i < rot_pairs, turned by the angles of the tables (as pace_latent_append); v is multiplied by
 * v_mul.  Row t of q_out [n_tokens][n_q_heads][row elements] belongs to token t; keys and values go to their pages (reserved).
 * qkv as pace_kv_append_norm.  store_ring: also stores the tokens' projections in the ring (one token per entry only:
 * with more, pace_conv_store behind the launch does).  dim, vdim <= 640. */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const float* taps;        /* fp32 [n_taps][all channels] */
  float* ring;
  const float* q_norm;
  const float* k_norm;
  const float* cos_table;
  const float* sin_table;
  void* q_out;
  int32_t n_q_heads, dim, vdim, n_taps, ring_rows, ring_stride, rot_pairs, table_rows, store_ring, dtype;
  float eps, v_mul;
} pace_append_conv_args_t;
int pace_kv_append_conv(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step, const pace_append_conv_args_t* a,
                        void* stream);

/* Causal softmax attention over the pool for any row format: q and out are dtype [q_row][n_q_heads][row
 * elements]; scores, weights and sums in fp32.  dim, vdim <= 512.  CUDA cores; the tensor-core kernels
 * (pace_attn_decode / pace_attn_prefill) take the PACE_ROWS_BF16 pools. */
int pace_attn_general(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step, const void* q, void* out,
                      int32_t n_q_heads, int32_t dim, int32_t vdim, float scale, int32_t dtype, void* stream);

/* Causal softmax attention with a span, a distance bias and a sink, for entries [entry_begin, entry_end) of a step.
 * The query at position i sees key j <= i
 *     PACE_SPAN_ALL     always,
 *     PACE_SPAN_WINDOW  if i - j < span_size,
 *     PACE_SPAN_CHUNK   if i / span_size == j / span_size (integer division, counted from position 0),
 * its score is scale * (q . k), with softcap > 0 replaced by softcap * tanh(score / softcap), minus slopes[h] * (i - j) (slopes
 * NULL: no bias), and exp(sinks[h]) is added to the denominator (sinks NULL: ordinary softmax).  Query head h reads KV head h / (n_q_heads / n_kv_heads).
 * Row t of q (dtype [n_tokens][n_q_heads][q_elems], dim elements used, zero up to the next multiple of 8) and of out
 * ([n_tokens][n_q_heads][out_elems], vdim elements written; tokens out_row elements apart where that is not 0) belongs to
 * token t.  The pool holds the step's own rows already;
 * lengths come from the step.  PACE_ROWS_SHARED pools: the value is the first vdim elements of the key row.
 * Scores, weights and sums are fp32 (with bf16 rows the weights enter the second product as two bf16 terms).
 * max_tokens / max_keys: upper bounds, over the entries, of their tokens and of their last position + 1.
 * bf16: tensor cores (mma.sync), the keys of a query tile split over a thread-block cluster; fp32 and what does not fit
 * that kernel: the CUDA-core kernel of pace_attn_general.  dim, vdim <= 640, 512. */
#define PACE_SPAN_ALL 0
#define PACE_SPAN_WINDOW 1
#define PACE_SPAN_CHUNK 2
typedef struct {
  const void* q;
  void* out;
  const float* slopes;   /* fp32 [n_q_heads] or NULL */
  const float* sinks;    /* fp32 [n_q_heads] or NULL */
  int32_t n_q_heads, dim, vdim, dtype, q_elems, out_elems;
  int32_t entry_begin, entry_end, max_tokens, max_keys;
  int32_t span, span_size;
  float scale;
  float softcap;         /* 0: none */
  int64_t out_row;       /* elements between the tokens of out; 0: n_q_heads * out_elems */
} pace_attn_span_args_t;
int pace_attn_span(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step, const pace_attn_span_args_t* a,
                   void* stream);

/* The same attention for prompts on the tcgen05 tensor cores (bf16): 256 query rows of one (entry, KV head) per thread
 * block, K and V tiles by TMA.  Keys come from the pool (k NULL; PACE_ROWS_BF16), or from plain tensors of expanded
 * rows: the keys of entry e are rows key_cu[e - entry_begin] .. key_cu[e - entry_begin + 1] - 1, of which the first has
 * position key_pos[e - entry_begin]; a key is k[row][head][0 .. k_dim) followed by k2[row][0 .. k2_dim) shared by all heads
 * (k2_dim may be 0), a value v[row][head][0 .. vdim).  Queries then are [0, k_dim) | [k_dim, k_dim + k2_dim).
 * Answers PACE_ERR_UNSUPPORTED (nothing launched) for shapes it does not take: sizes and strides that are not
 * multiples of 8, more than 256 key or 128 value elements (rounded up to 64 per part). */
typedef struct {
  pace_attn_span_args_t a;
  const void* k;
  const void* k2;
  const void* v;
  int64_t k_row, k_head, k2_row, v_row, v_head;   /* strides in elements */
  int32_t k_dim, k2_dim, n_kv_heads, n_rows;
  const int32_t* key_cu;    /* device, [entry_end - entry_begin + 1] */
  const int32_t* key_pos;   /* device, [entry_end - entry_begin] */
} pace_attn_span_prefill_args_t;
int pace_attn_span_prefill(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step,
                           const pace_attn_span_prefill_args_t* a, void* stream);

/* ---- latent attention: what surrounds the products ------------------------------------------------------------------
 * pace_latent_append: one token's down projections, down [n_tokens][down_stride] = query latent (q_rank) | key/value
 * latent (kv_rank) | rotated key part (rot_dim):
 *     cq[t] = rms(query latent) * q_norm                                      (dtype [n_tokens][q_rank]; q_rank 0: none)
 *     page row of token t = rms(kv latent) * kv_norm | rotate(key part) | 0
 * rotate turns the pairs (2i, 2i + 1), i < rot_pairs, by the angles whose cosine and sine are cos[pos][i], sin[pos][i]
 * (fp32 tables of table_rows rows).
 * pace_rotate_heads: the same rotation for n_heads parts of rot_dim elements per token, src[t][h] -> dst[t][h] (strides in
 * elements; may be the same place), zeros in dst up to pad_dim elements.
 * pace_latent_gather: page rows of (slot[i], pos[i]), i < n, into out [n][row elements].
 * The pool is PACE_ROWS_SHARED with one KV head. */
typedef struct {
  const void* down;
  int64_t down_stride;
  const float* q_norm;
  const float* kv_norm;
  const float* cos_table;
  const float* sin_table;
  void* cq;
  int32_t q_rank, kv_rank, rot_dim, rot_pairs, table_rows, dtype;
  float eps;
} pace_latent_append_args_t;
int pace_latent_append(const pace_kv_pool_t* pool, int32_t layer, const pace_step_t* step,
                       const pace_latent_append_args_t* a, void* stream);
typedef struct {
  const void* src;
  void* dst;
  int64_t src_row, src_head, dst_row, dst_head;
  const float* cos_table;
  const float* sin_table;
  int32_t token_begin, token_end, n_heads, rot_dim, rot_pairs, pad_dim, table_rows, dtype;
} pace_rotate_args_t;
int pace_rotate_heads(const pace_step_t* step, const pace_rotate_args_t* a, void* stream);
int pace_latent_gather(const pace_kv_pool_t* pool, int32_t layer, const int32_t* slot, const int32_t* pos, int32_t n,
                       void* out, void* stream);

/* ---- gated feed-forwards and mixtures of experts --------------------------------------------------------------------
 * pace_glu: out[t][i] = act(x[t][i]) * x[t][n + i], x rows of 2 n elements; without `gated` act(x[t][i]), rows of n. */
#define PACE_ACT_SILU 0
#define PACE_ACT_GELU_TANH 1
#define PACE_ACT_GELU_ERF 2
#define PACE_ACT_NONE 3   /* experts' second product */
int pace_glu(const void* x, int64_t x_stride, void* out, int64_t out_stride, int32_t n_tokens, int32_t n, int32_t act,
             int32_t gated, int32_t dtype, void* stream);
/* x = cap * tanh(x / cap) in place, n fp32 elements. */
int pace_soft_cap(float* x, int64_t n, float cap, void* stream);

/* Router: scores = sigmoid(logits) or softmax(logits) (logits fp32 [n_tokens][n_experts]); the `top` experts with the
 * largest scores + correction (fp32 [n_experts] or NULL; ties go to the lower index) are chosen, their weights are the scores
 * without it; `normalise` divides them by their sum + 1e-20 and multiplies them by weight_scale.  Identity experts are the last
 * of n_experts here; pace_moe_experts gets the number of those in front.  slot_expert / slot_weight [n_tokens][top]; expert_count [n_experts] and slot_rank [n_tokens][top] number the tokens
 * of an expert, expert_list [n_experts][n_tokens] lists them.  top <= 64, n_experts <= 1024. */
typedef struct {
  const float* logits;
  const float* correction;
  int32_t* slot_expert;
  int32_t* slot_rank;
  float* slot_weight;
  int32_t* expert_count;
  int32_t* expert_list;
  int32_t n_tokens, n_experts, top;
  int32_t softmax, normalise;
  float weight_scale;
} pace_moe_route_args_t;
int pace_moe_route(const pace_moe_route_args_t* a, void* stream);

/* The chosen experts' feed-forwards: for every (token, expert) pair of the router
 *     hidden = act(gate x) * (up x),  y = down hidden           (without `gated`: hidden = act(up x))
 * x dtype [n_tokens][width], gate_up dtype [n_experts][2 ff][width] (gate rows first; ff rows without `gated`), down dtype [n_experts][width][ff].
 * hidden [n_tokens * top][ff] and y [n_tokens * top][width] are written by expert: expert e's token of rank r is row
 *     expert_row(e, r) = expert_count[0] + .. + expert_count[e - 1] + r.
 * bf16 with width and ff multiples of 8: grouped products on the tcgen05 tensor cores, weights as the 128-row operand.
 * `scratch` (dtype [n_tokens * top][width], or NULL) chooses between tiles of 128 tokens, whose rows are first copied into
 * expert order there, and (NULL) tiles of 32 tokens gathered by TMA, for few tokens per expert.  Otherwise CUDA cores.  `status` (device int32, may be NULL) takes
 * PACE_DEV_WAIT_TIMEOUT if a bounded wait runs out. */
typedef struct {
  const void* x;
  const void* gate_up;
  const void* down;
  void* hidden;
  void* y;
  void* scratch;
  const int32_t* expert_count;
  const int32_t* expert_list;
  const int32_t* slot_expert;   /* with scratch: the router's */
  const int32_t* slot_rank;
  int32_t* status;
  int32_t n_tokens, n_experts, top, width, ff, act, dtype, gated;
} pace_moe_experts_args_t;
int pace_moe_experts(const pace_moe_experts_args_t* a, void* stream);

/* out[t][h * vdim + i] = attn[q_row[t]][h][i] * sigmoid(gate[t][h * vdim + i]);
 * attn rows are [n_heads][row_elems], gate has gate_stride elements per token. */
int pace_gate_heads(const pace_step_t* step, const void* attn, const void* gate, int64_t gate_stride, void* out,
                    int32_t n_heads, int32_t vdim, int32_t row_elems, int32_t dtype, void* stream);
/* out[t] = rms(o[t]) * w * sigmoid(gate[t]) over n elements (w fp32). */
int pace_norm_gate(const void* o, const float* w, const void* gate, int64_t gate_stride, void* out, int32_t n_tokens,
                   int32_t n, float eps, int32_t dtype, void* stream);
#define PACE_GATE_SIGMOID 0
#define PACE_GATE_SILU_FIRST 1
#define PACE_GATE_SILU 2
/* Norms over equal parts of a row, with a gate in front (silu) or behind (sigmoid or silu):
 *     gate_mode PACE_GATE_SILU_FIRST:  out = rms(o * silu(gate)) * w
 *     PACE_GATE_SIGMOID, PACE_GATE_SILU:  out = rms(o) * w * sigmoid(gate), silu(gate)
 * rms over every `part` elements (n a multiple of part), weight w[c % w_period] (fp32). */
typedef struct {
  const void* o;
  const void* gate;
  const float* w;
  void* out;
  int64_t o_stride, gate_stride, out_stride;
  int32_t n_tokens, n, part, w_period, gate_mode, dtype;
  float eps;
} pace_part_norm_gate_args_t;
int pace_part_norm_gate(const pace_part_norm_gate_args_t* a, void* stream);
/* x = relu(x)^2 in place, n elements. */
int pace_relu_squared(void* x, int64_t n, int32_t dtype, void* stream);

/* Causal depthwise convolution: out[t][c] = act(bias[c] + sum_j taps[j][c] in[c](pos - (n_taps - 1) + j)), zeros
 * in front of the sequence; act is silu or nothing, bias may be NULL.  conv_state fp32 [slots][ring_rows][ring_stride] holds
 * each slot's newest inputs in row position % ring_rows (ring_rows >= n_taps - 1, and n_taps where the launch that reads a ring
 * or one beside it writes the current token's row).  This entry point reads it; the recurrence behind it or
 * pace_conv_store stores the new inputs.  `conv_state` points at the first of `channels` channels of a row. */
typedef struct {
  const void* in;
  int64_t in_stride;
  const float* taps;        /* fp32 [n_taps][channels] */
  const float* bias;
  const float* conv_state;
  void* out;
  int64_t out_stride;
  int32_t n_taps, channels, ring_rows, ring_stride, silu, dtype;
} pace_causal_conv_args_t;
int pace_causal_conv(const pace_step_t* step, const pace_causal_conv_args_t* a, void* stream);
/* The newest inputs (the last ring_rows tokens at most) of every entry into its ring. */
int pace_conv_store(const pace_step_t* step, const void* in, int64_t in_stride, float* ring, int32_t ring_rows,
                    int32_t ring_stride, int32_t channels, int32_t dtype, void* stream);

/* Real-gated linear recurrence (RG-LRU) with its branch product:
 *     r = sigmoid(gates_r + ra_bias), i = sigmoid(gates_i + ri_bias), log a = decay_base * r
 *     S_t = a S_(t-1) + sqrt(1 - a^2) i u,    out = S * gelu_tanh(y)
 * decay_base fp32 [width] (= -8 softplus(lam)); state fp32 [slots][width].  yx is dtype [n_tokens][yx_stride]
 * with y in columns [0, width) and the convolution's input in [width, 2 width): its newest rows go to
 * conv_state.
 * pace_rglru_scan: gates fp32 [blocks][n_tokens][2][width / blocks] (r, i) and u dtype [n_tokens][width] come
 * from launches in front (any counts per entry).
 * pace_rglru_step: one token per entry (n_tokens == n_entries); convolution and block-diagonal gates
 * (gate_w dtype [blocks][2][out][in]) are part of the launch. */
typedef struct {
  const void* yx;
  int64_t yx_stride;
  const void* u;          /* scan only */
  const float* gates;     /* scan only */
  const void* gate_w;     /* step only */
  const float* taps;      /* step only: fp32 [n_taps][width] */
  const float* conv_bias; /* step only */
  const float* ra_bias;
  const float* ri_bias;
  const float* decay_base;
  float* state;
  float* conv_state;
  void* out;              /* dtype [n_tokens][width] */
  int32_t width, blocks, n_taps, dtype;
} pace_rglru_args_t;
int pace_rglru_scan(const pace_step_t* step, const pace_rglru_args_t* a, void* stream);
int pace_rglru_step(const pace_step_t* step, const pace_rglru_args_t* a, void* stream);

/* Linear attention with a fixed decay per head: with q, k, v = silu of the projections (rounded to dtype),
 *     S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t.
 * qkv dtype [n_tokens][qkv_stride]: q (heads x dim), k (heads x dim), v (heads x vdim).  state fp32
 * [slots][heads][dim][vdim].  out dtype [n_tokens][heads x vdim].  dim <= 512 (vdim any).
 * pace_lightning_step: one token per entry; pace_lightning_prefill: any counts (bf16 with dim <= 128 and sizes that
 * are multiples of 8: chunks of 64 tokens on the tensor cores; otherwise token by token). */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const float* decay;     /* fp32 [heads] */
  float* state;
  void* out;
  float* workspace;       /* prefill: pace_lightning_workspace_bytes() of scratch, any content */
  uint64_t workspace_bytes;
  int32_t heads, dim, vdim, dtype;
} pace_lightning_args_t;
/* Scratch of a prefill (0: none).  Long sequences are cut into segments that run side by side. */
uint64_t pace_lightning_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t dim, int32_t vdim);
int pace_lightning_prefill(const pace_step_t* step, const pace_lightning_args_t* a, void* stream);
int pace_lightning_step(const pace_step_t* step, const pace_lightning_args_t* a, void* stream);

/* State-space recurrence with a decay per head and token (Mamba-2):
 *     dt = softplus(dt_raw + dt_bias),  S_t = exp(neg_a dt) S_(t-1) + dt b_t x_t^T,  y_t = S_t^T c_t + d_skip x_t
 * per head (S state x vdim; head h reads b and c of group h / (heads / groups)); neg_a = -exp(A_log), all fp32 [heads].
 * xbc dtype [n_tokens][xbc_stride] = x (heads x vdim) | b (groups x state) | c (groups x state); dt_raw dtype
 * [n_tokens][dt_stride].  s_state fp32 [slots][heads][state][vdim].  out dtype [n_tokens][out_stride].
 * pace_ssd_prefill: xbc behind the convolution and silu (any counts per entry).  bf16 with state <= 128 and sizes that
 * are multiples of 8: chunks on the tensor cores; otherwise token by token.
 * pace_ssd_step: one token per entry; xbc in front of the convolution (taps, conv_bias, ring as pace_causal_conv; the launch
 * stores the new rows; ring_rows >= n_taps).  state <= 512. */
typedef struct {
  const void* xbc;
  int64_t xbc_stride;
  const void* dt_raw;
  int64_t dt_stride;
  const float* dt_bias;
  const float* neg_a;
  const float* d_skip;
  float* s_state;
  void* out;
  int64_t out_stride;
  const float* taps;        /* step only */
  const float* conv_bias;   /* step only, may be NULL */
  float* ring;              /* step only */
  float* workspace;         /* prefill: pace_ssd_workspace_bytes() of scratch, any content */
  uint64_t workspace_bytes;
  int32_t heads, groups, state, vdim, n_taps, ring_rows, ring_stride, dtype;
} pace_ssd_args_t;
uint64_t pace_ssd_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t state, int32_t vdim);
int pace_ssd_prefill(const pace_step_t* step, const pace_ssd_args_t* a, void* stream);
int pace_ssd_step(const pace_step_t* step, const pace_ssd_args_t* a, void* stream);

/* Gated delta rule with a decay per head and key channel:
 *     g_t = exp(neg_a softplus(a_raw + dt_bias)),  beta_t = sigmoid(b_raw)
 *     S <- g_t S (rows);  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
 * per head (S dim x vdim); q and k are made unit vectors per head, x / sqrt(sum(x^2) + unit_eps), q times q_scale; head h uses
 * q / k head h / (heads / kv_heads).  qkv dtype [n_tokens][qkv_stride] = q (kv_heads x dim) | k (kv_heads x dim) |
 * v (heads x vdim); a_raw dtype rows of heads x dim, b_raw dtype rows of heads; neg_a = -exp(A_log) fp32 [heads], dt_bias fp32
 * [heads x dim].  s_state fp32 [slots][heads][dim][vdim].  out dtype [n_tokens][out_stride].
 * pace_delta_prefill: qkv behind the convolution and silu.  pace_delta_step: one token per entry, qkv in front of
 * them (taps, ring as pace_ssd_step, no bias).  dim <= 512. */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const void* a_raw;
  int64_t a_stride;
  const void* b_raw;
  int64_t b_stride;
  const float* dt_bias;
  const float* neg_a;
  float* s_state;
  void* out;
  int64_t out_stride;
  const float* taps;        /* step only */
  float* ring;              /* step only */
  void* workspace;          /* prefill: pace_delta_workspace_bytes() of scratch, any content */
  uint64_t workspace_bytes;
  int32_t heads, kv_heads, dim, vdim, n_taps, ring_rows, ring_stride, dtype;
  float unit_eps, q_scale;
} pace_delta_args_t;
uint64_t pace_delta_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t dim, int32_t vdim, int32_t dtype);
int pace_delta_prefill(const pace_step_t* step, const pace_delta_args_t* a, void* stream);
int pace_delta_step(const pace_step_t* step, const pace_delta_args_t* a, void* stream);

/* Gated linear attention with a decay per head and key channel:
 *     alpha_t = sigmoid(z + z_bias)^inv_tau;  S <- diag(alpha_t) S + k_t v_t^T;  o_t = q_scale S^T q_t
 * per head (S dim x vdim).  qkv dtype [n_tokens][qkv_stride] = q (heads x dim) | k (heads x dim) | v (heads x vdim); z dtype rows of
 * heads x dim, z_bias fp32 [heads x dim].  s_state fp32 [slots][heads][dim][vdim].  out dtype [n_tokens][out_stride].
 * pace_gla_step: one token per entry; the outputs are normalised per head and gated as well,
 *     out = rms(o) * norm * silu(gate)           (norm fp32 [vdim], shared by the heads; gate dtype rows of heads x vdim)
 * dim <= 512. */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const void* z;
  int64_t z_stride;
  const float* z_bias;
  float* s_state;
  void* out;
  int64_t out_stride;
  const float* norm;        /* step only */
  const void* gate;         /* step only */
  int64_t gate_stride;
  void* workspace;          /* prefill: pace_gla_workspace_bytes() of scratch, any content */
  uint64_t workspace_bytes;
  int32_t heads, dim, vdim, dtype;
  float inv_tau, q_scale, eps;
} pace_gla_args_t;
uint64_t pace_gla_workspace_bytes(int32_t n_entries, int32_t max_count, int32_t heads, int32_t dim, int32_t dtype);
int pace_gla_prefill(const pace_step_t* step, const pace_gla_args_t* a, void* stream);
int pace_gla_step(const pace_step_t* step, const pace_gla_args_t* a, void* stream);

/* ---- attention over a window and pooled blocks -----------------------------------------------------------------------
 * A layer has two pools of the same row geometry: tokens, and blocks of `block` tokens (row_tokens = block), whose rows are the means
 * of the cached keys and of the cached values of a whole block.
 * pace_kv_append_rotate: qkv dtype [n_tokens][qkv_stride] = q (n_q_heads x dim) | k (kv_heads x dim) | v (kv_heads x vdim); the
 * first 2 rot_pairs elements of every query and key head are turned by the angles of the tables (fp32 [table_rows][rot_pairs]),
 * element i with element i + rot_pairs (`halves`) or 2i with 2i + 1; queries go to q_out [n_tokens][n_q_heads][row elements], keys and
 * values to their pages (reserved), rows are zero beyond dim / vdim.  With block > 0 the blocks that the step's tokens complete
 * get their rows, by a launch behind, or with block_now (one token per entry) by the same one. */
typedef struct {
  const void* qkv;
  int64_t qkv_stride;
  const float* cos_table;
  const float* sin_table;
  void* q_out;
  int32_t n_q_heads, dim, vdim, rot_pairs, halves, table_rows, block, block_now, dtype;
} pace_append_rotate_args_t;
int pace_kv_append_rotate(const pace_kv_pool_t* pool, int32_t layer, const pace_kv_pool_t* blocks, int32_t block_layer,
                          const pace_step_t* step, const pace_append_rotate_args_t* a, void* stream);

/* The query at position i sees the tokens j with 0 <= i - j < window and, with block > 0, the blocks b whose last token
 * b block + block - 1 is at most i - window.  One softmax over both, score = scale * (q . k), with exp(sinks[h]) in the denominator
 * (sinks NULL: ordinary softmax).  mix (fp32 [n_q_heads][n_q_heads], NULL: none) then mixes the heads' weights, weight_h <- sum_g
 * mix[h][g] weight_g, in front of the values of head h's own KV head (h / (n_q_heads / kv_heads)), and gate (dtype rows of n_q_heads x
 * vdim, NULL: none) multiplies the outputs by its sigmoid.  q dtype [n_tokens][n_q_heads][row elements]; out dtype rows of n_q_heads
 * x vdim.  Tokens [token_begin, token_end) of the step; max_keys: upper bound of their positions + 1.
 * pace_attn_pooled: token by token; pace_attn_pooled_prompt: entries [entry_begin, entry_end) of up to max_tokens tokens on tcgen05,
 * with scratch of pace_attn_pooled_prompt_workspace_bytes(); answers PACE_ERR_UNSUPPORTED (nothing launched) for what it does not
 * take: fp32, rows other than PACE_ROWS_BF16 in pages of 64 rows, scales that are not positive, more than 32 query heads per KV
 * head. */
typedef struct {
  const void* q;
  void* out;
  const void* gate;
  const float* sinks;
  const float* mix;
  int64_t out_stride, gate_stride;
  int32_t n_q_heads, dim, vdim, dtype, q_elems, window, block, token_begin, token_end, entry_begin, entry_end, max_tokens, max_keys;
  float scale;
  void* workspace;
  uint64_t workspace_bytes;
} pace_attn_pooled_args_t;
int pace_attn_pooled(const pace_kv_pool_t* pool, int32_t layer, const pace_kv_pool_t* blocks, int32_t block_layer,
                     const pace_step_t* step, const pace_attn_pooled_args_t* a, void* stream);
uint64_t pace_attn_pooled_prompt_workspace_bytes(int32_t n_entries, int32_t max_tokens, int32_t n_q_heads, int32_t n_kv_heads,
                                                 int32_t vdim, int32_t mixed);
int pace_attn_pooled_prompt(const pace_kv_pool_t* pool, int32_t layer, const pace_kv_pool_t* blocks, int32_t block_layer,
                            const pace_step_t* step, const pace_attn_pooled_args_t* a, void* stream);

/* ---- layers that read shifted inputs ---------------------------------------------------------------------------------
 * pace_shift_norm: between two layers,
 *     x_out = x_in + rms(y + y_bias) * w_post + add                       (y, y_bias, add may be NULL; add, y_bias fp32 [width])
 *     n = rms(x_out) * w_next,   h = n + (n' - n) * shift                 (element by element)
 * with n' the n of the sequence's previous token: of the step, or state[slot] (fp32 rows of state_stride), or zeros in front of the
 * first one.  The last n of every entry goes to state_out[slot].  x_out and state_out may be x_in and state in a step of one token per
 * entry; otherwise they must be other buffers (pace_state_commit brings the states over).
 * pace_embed_pairs: x = embed[token] * scale + pairs[(previous token * mul_prev + token * mul_cur) mod buckets]; pairs (dtype
 * [buckets + 1][width], NULL: none) has one more row for a sequence's first token.  last_token int32 [slots]; store_last (one token
 * per entry) also stores the token there.
 * pace_state_commit: to[slot][0 .. n) = from[slot][0 .. n) for the step's slots (rows of `stride`), last_token (or NULL) [slot] =
 * the entry's last token. */
typedef struct {
  const float* x_in;
  float* x_out;
  const void* y;
  int64_t y_stride;
  const float* y_bias;
  const float* w_post;
  const float* add;
  const float* w_next;
  const float* shift;
  const float* state;
  float* state_out;
  int64_t state_stride;
  void* h;
  int32_t width, dtype;
  float eps;
} pace_shift_norm_args_t;
int pace_shift_norm(const pace_step_t* step, const pace_shift_norm_args_t* a, void* stream);
typedef struct {
  float* x;
  const void* embed;
  const void* pairs;
  int32_t* last_token;
  int64_t mul_prev, mul_cur;
  int32_t width, vocab, buckets, store_last, dtype;
  float scale;
} pace_embed_pairs_args_t;
int pace_embed_pairs(const pace_step_t* step, const pace_embed_pairs_args_t* a, void* stream);
int pace_state_commit(const pace_step_t* step, const float* from, float* to, int64_t n, int64_t stride, int32_t* last_token,
                      void* stream);
/* x[t][h][0 .. vdim) *= sigmoid(gate[t][h]) in place; x dense [n_tokens][heads][vdim]. */
int pace_gate_per_head(void* x, const void* gate, int64_t gate_stride, int32_t n_tokens, int32_t heads, int32_t vdim, int32_t dtype,
                       void* stream);

/* Step arrays of a decode step whose tokens and positions the device holds (one token per entry):
 * token[i] = next_token[i], tok_pos[i] = start[i] = position[i]. */
int pace_step_decode(int32_t* token, int32_t* tok_pos, int32_t* start, const int64_t* next_token,
                     const int64_t* position, int32_t n_entries, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* PACE_B200_H_ */
