"""``torch.ops.pace_b200.*``: the KV-pool and paged-attention entry points as dispatcher ops.

The reference reaches its compiled kernels through ops registered with the dispatcher
(``TORCH_LIBRARY_FRAGMENT(pace, m) { m.def("attention(...)") }``, csrc/ops/attention.cpp:104-108);
this module does the same for what replaces its Python cache bookkeeping and its attention op on a
GPU.  Every op is a thin shell over one C-ABI function of libpace_b200.so: tensors go in as device
pointers and element strides, the call is stream-ordered on the current CUDA stream, nothing is
returned (results land in ``out`` / in the pool).  The Python classes of ``pace_b200.llm.cache`` and
``pace_b200.ops.backends.b200`` call these ops, so a caller that works at the dispatcher level
(tracing, ``torch.compile``, C++ through ``c10::Dispatcher``) sees the same calls they make.

A pool is named by ``pool``, the address of its ``pace_kv_pool_t`` descriptor
(``KVPool.handle``); ``pages`` / ``meta`` are the pool's two storage tensors, passed so that the
schema can say what an op writes.
"""
import ctypes as C
import math
from typing import Optional

import torch

from pace_b200 import _C

_lib = torch.library.Library("pace_b200", "DEF")

_DEFS = {
    "kv_reserve": "(int pool, Tensor(a!) meta, int layer, Tensor seq_ids, int n_new, Tensor? n_new_per_seq) -> ()",
    "kv_append": "(int pool, Tensor(a!) pages, Tensor(b!) meta, int layer, Tensor seq_ids, Tensor k_new, Tensor v_new, "
                 "Tensor? n_new_per_seq) -> ()",
    "kv_append_layers": "(int pool, Tensor(a!) pages, Tensor(b!) meta, int layer_begin, int layer_end, Tensor seq_ids, "
                        "Tensor? k_all, Tensor? v_all, int n_new=1, Tensor? n_new_per_seq=None) -> ()",
    "kv_append_rope": "(int pool, Tensor(a!) pages, Tensor(b!) meta, int layer, Tensor seq_ids, Tensor q, Tensor k, "
                      "Tensor v, Tensor(c!) q_out, Tensor table_row, Tensor cos, Tensor sin, int rotary_dim, "
                      "bool gptj_pairs, Tensor? n_new_per_seq, Tensor(d!)? k_stage, Tensor(e!)? v_stage) -> ()",
    "kv_truncate": "(int pool, Tensor(a!) meta, int layer_begin, int layer_end, Tensor seq_ids, int remove_len, "
                   "Tensor? remove_per_seq) -> ()",
    "kv_gather": "(int pool, Tensor(a!) meta, Tensor seq_ids, Tensor beam_idx) -> ()",
    "pard_accept": "(Tensor drafts, Tensor target_next, Tensor n_target, Tensor? forced, Tensor(a!) keep, "
                   "Tensor(b!) target_remove, Tensor(c!) draft_remove, Tensor(d!) kept) -> ()",
    "kv_read_dense": "(int pool, Tensor pages, int layer, Tensor seq_ids, Tensor(a!) k_out, Tensor(b!) v_out) -> ()",
}
_DEFS["linear_skinny"] = "(Tensor x, Tensor weight, Tensor(a!) out, Tensor(b!) workspace) -> ()"
# layers of hybrid decoders; a step is named by the address of its pace_step_t (``Step.handle``)
_DEFS.update({
    "residual_norm": "(int step, Tensor(a!) x, Tensor? y, Tensor? w_post, Tensor? embed, Tensor? w_next, Tensor(b!)? h, "
                     "float eps, bool restart, float weight_offset, float embed_scale=1.0, int top=0, Tensor? slot_expert=None, "
                     "Tensor? slot_rank=None, Tensor? slot_weight=None, Tensor? expert_count=None, Tensor? identity=None, "
                     "Tensor? add=None, Tensor? y_bias=None, Tensor? embed_norm=None, Tensor? w_next2=None, Tensor(c!)? h2=None, "
                     "float y_mul=1.0) -> ()",
    "kv_append_norm": "(int pool, Tensor(a!) pages, int layer, int step, Tensor qkv, Tensor? q_norm, Tensor? k_norm, "
                      "Tensor(b!) q_out, int dim, int vdim, float eps, float q_mul, float temp_coef, float temp_every, "
                      "bool per_head=False) -> ()",
    "attn_span": "(int pool, Tensor pages, int layer, int step, Tensor q, Tensor(a!) out, Tensor? slopes, Tensor? sinks, int dim, "
                 "int vdim, float scale, int span, int span_size, int entry_begin, int entry_end, int max_tokens, int max_keys, "
                 "float softcap=0.0, int out_row=0) -> ()",
    "attn_span_prefill": "(int pool, Tensor? pages, int layer, int step, Tensor q, Tensor(a!) out, Tensor? slopes, Tensor? sinks, "
                         "int dim, int vdim, float scale, int span, int span_size, int entry_begin, int entry_end, int max_tokens, "
                         "int max_keys, Tensor? k, Tensor? k2, Tensor? v, Tensor? key_cu, Tensor? key_pos, "
                         "float softcap=0.0, int out_row=0) -> bool",
    "latent_append": "(int pool, Tensor(a!) pages, int layer, int step, Tensor down, Tensor? q_norm, Tensor kv_norm, Tensor? cos, "
                     "Tensor? sin, Tensor(b!)? cq, int rot_dim, float eps) -> ()",
    "rotate_heads": "(int step, Tensor src, Tensor(a!) dst, Tensor cos, Tensor sin, int token_begin, int token_end, int pad_dim) -> ()",
    "latent_gather": "(int pool, Tensor pages, int layer, Tensor slot, Tensor pos, Tensor(a!) out) -> ()",
    "glu": "(Tensor x, Tensor(a!) out, int act, bool gated=True) -> ()",
    "soft_cap": "(Tensor(a!) x, float cap) -> ()",
    "part_norm_gate": "(Tensor o, Tensor gate, Tensor w, Tensor(a!) out, int part, int gate_mode, float eps) -> ()",
    "kv_append_conv": "(int pool, Tensor(a!) pages, int layer, int step, Tensor qkv, Tensor taps, Tensor(b!) ring, Tensor q_norm, "
                      "Tensor k_norm, Tensor? cos, Tensor? sin, Tensor(c!) q_out, int dim, int vdim, float eps, float v_mul, "
                      "bool store_ring) -> ()",
    "conv_store": "(int step, Tensor x, Tensor(a!) ring) -> ()",
    "ssd_prefill": "(int step, Tensor xbc, Tensor dt_raw, Tensor dt_bias, Tensor neg_a, Tensor d_skip, Tensor(a!) state, "
                   "Tensor(b!) out, int groups) -> ()",
    "ssd_step": "(int step, Tensor xbc, Tensor dt_raw, Tensor dt_bias, Tensor neg_a, Tensor d_skip, Tensor(a!) state, "
                "Tensor(b!) out, int groups, Tensor taps, Tensor? conv_bias, Tensor(c!) ring) -> ()",
    "delta_prefill": "(int step, Tensor qkv, Tensor a_raw, Tensor b_raw, Tensor dt_bias, Tensor neg_a, Tensor(a!) state, "
                     "Tensor(b!) out, int kv_heads, float unit_eps, float q_scale) -> ()",
    "delta_step": "(int step, Tensor qkv, Tensor a_raw, Tensor b_raw, Tensor dt_bias, Tensor neg_a, Tensor(a!) state, "
                  "Tensor(b!) out, int kv_heads, float unit_eps, float q_scale, Tensor taps, Tensor(c!) ring) -> ()",
    "gla_prefill": "(int step, Tensor qkv, Tensor z, Tensor z_bias, Tensor(a!) state, Tensor(b!) out, float inv_tau, float q_scale) -> ()",
    "gla_step": "(int step, Tensor qkv, Tensor z, Tensor z_bias, Tensor(a!) state, Tensor(b!) out, float inv_tau, float q_scale, "
                "Tensor norm, Tensor gate, float eps) -> ()",
    "kv_append_rotate": "(int pool, Tensor(a!) pages, int layer, int blocks, Tensor(b!)? block_pages, int block_layer, int step, Tensor qkv, "
                        "Tensor? cos, Tensor? sin, Tensor(c!) q_out, int dim, int vdim, bool halves, int block, bool block_now) -> ()",
    "attn_pooled": "(int pool, Tensor pages, int layer, int blocks, Tensor? block_pages, int block_layer, int step, Tensor q, "
                   "Tensor(a!) out, Tensor? gate, Tensor? sinks, Tensor? mix, int dim, int vdim, float scale, int window, int block, "
                   "int token_begin, int token_end, int max_keys) -> ()",
    "attn_pooled_prompt": "(int pool, Tensor pages, int layer, int blocks, Tensor? block_pages, int block_layer, int step, Tensor q, "
                          "Tensor(a!) out, Tensor? gate, Tensor? sinks, Tensor? mix, int dim, int vdim, float scale, int window, int block, "
                          "int entry_begin, int entry_end, int max_tokens, int max_keys) -> bool",
    "shift_norm": "(int step, Tensor x_in, Tensor(a!) x_out, Tensor? y, Tensor? y_bias, Tensor? w_post, Tensor? add, Tensor w_next, "
                  "Tensor shift, Tensor state, Tensor(b!) state_out, Tensor(c!) h, float eps) -> ()",
    "embed_pairs": "(int step, Tensor(a!) x, Tensor embed, float scale, Tensor? pairs, Tensor(b!)? last_token, int mul_prev, int mul_cur, "
                   "bool store_last) -> ()",
    "state_commit": "(int step, Tensor source, Tensor(a!) target, Tensor(b!)? last_token) -> ()",
    "gate_per_head": "(Tensor(a!) x, Tensor gate) -> ()",
    "moe_route": "(Tensor logits, Tensor? correction, Tensor(a!) slot_expert, Tensor(b!) slot_rank, Tensor(c!) slot_weight, "
                 "Tensor(d!) expert_count, Tensor(e!) expert_list, bool softmax=False, float? weight_scale=None) -> ()",
    "moe_experts": "(Tensor x, Tensor gate_up, Tensor down, Tensor(a!) hidden, Tensor(b!) y, Tensor(d!)? scratch, "
                   "Tensor expert_count, Tensor expert_list, Tensor slot_expert, Tensor slot_rank, Tensor(c!)? status, int act, "
                   "bool gated=True) -> ()",
    "attn_general": "(int pool, Tensor pages, int layer, int step, Tensor q, Tensor(a!) out, int dim, int vdim, "
                    "float scale) -> ()",
    "gate_heads": "(int step, Tensor attn, Tensor gate, Tensor(a!) out, int vdim) -> ()",
    "norm_gate": "(Tensor o, Tensor weight, Tensor gate, Tensor(a!) out, float eps) -> ()",
    "relu_squared": "(Tensor(a!) x) -> ()",
    "causal_conv": "(int step, Tensor x, Tensor taps, Tensor? bias, Tensor conv_state, Tensor(a!) out, bool silu=False) -> ()",
    "rglru_scan": "(int step, Tensor yx, Tensor u, Tensor gates, Tensor ra_bias, Tensor ri_bias, Tensor decay_base, "
                  "Tensor(a!) state, Tensor(b!) conv_state, Tensor(c!) out, int blocks) -> ()",
    "rglru_step": "(int step, Tensor yx, Tensor gate_w, Tensor taps, Tensor conv_bias, Tensor ra_bias, Tensor ri_bias, "
                  "Tensor decay_base, Tensor(a!) state, Tensor(b!) conv_state, Tensor(c!) out, int blocks) -> ()",
    "lightning_prefill": "(int step, Tensor qkv, Tensor decay, Tensor(a!) state, Tensor(b!) out) -> ()",
    "lightning_step": "(int step, Tensor qkv, Tensor decay, Tensor(a!) state, Tensor(b!) out) -> ()",
    "step_decode": "(Tensor(a!) token, Tensor(b!) tok_pos, Tensor(c!) start, Tensor next_token, Tensor position) -> ()",
})
_ATTN = ("(int pool, Tensor(a!) pages, int layer, Tensor q, Tensor(b!) out, Tensor? seq_ids, Tensor? kv_start, "
         "Tensor? q_lens, Tensor(c!) workspace, float scale, int flags, Tensor? k_pending, Tensor? v_pending, "
         "int max_ctas) -> ()")
for _n in ("attn_decode", "attn_decode_cuda_cores", "attn_verify", "attn_prefill"):
    _DEFS[_n] = _ATTN
for _n, _sig in _DEFS.items():
    _lib.define(_n + _sig)


def _pool(handle: int):
    return C.byref(_C.KVPoolStruct.from_address(handle))


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _stream(t: torch.Tensor) -> int:
    return torch.cuda.current_stream(t.device).cuda_stream


def _kv_reserve(pool, meta, layer, seq_ids, n_new, n_new_per_seq=None):
    with torch.cuda.device(meta.device):
        _C.check(_C.lib.pace_kv_reserve(_pool(pool), layer, seq_ids.data_ptr(), seq_ids.numel(), n_new,
                                        _ptr(n_new_per_seq), _stream(meta)), "pace_kv_reserve")


def _kv_append(pool, pages, meta, layer, seq_ids, k_new, v_new, n_new_per_seq=None):
    B, _, n, _ = k_new.shape
    sb, sh, st, _ = k_new.stride()
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append(_pool(pool), layer, seq_ids.data_ptr(), B, n, _ptr(n_new_per_seq),
                                       k_new.data_ptr(), v_new.data_ptr(), sb, sh, st, _stream(pages)), "pace_kv_append")


def _kv_append_layers(pool, pages, meta, layer_begin, layer_end, seq_ids, k_all=None, v_all=None, n_new=1,
                      n_new_per_seq=None):
    sl = sb = sh = st = 0
    if k_all is not None:
        sl, sb, sh, st, _ = k_all.stride()
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append_layers(_pool(pool), layer_begin, layer_end, seq_ids.data_ptr(), seq_ids.numel(), n_new,
                                              _ptr(n_new_per_seq), _ptr(k_all), _ptr(v_all), sl, sb, sh, st, _stream(pages)),
                 "pace_kv_append_layers")


def _kv_append_rope(pool, pages, meta, layer, seq_ids, q, k, v, q_out, table_row, cos, sin, rotary_dim, gptj_pairs,
                    n_new_per_seq=None, k_stage=None, v_stage=None):
    B, n, Hq, _ = q.shape
    a = _C.RopeArgs()
    a.q, (a.q_stride_b, a.q_stride_t, a.q_stride_h) = q.data_ptr(), q.stride()[:3]
    a.k, (a.k_stride_b, a.k_stride_t, a.k_stride_h) = k.data_ptr(), k.stride()[:3]
    a.v, (a.v_stride_b, a.v_stride_t, a.v_stride_h) = v.data_ptr(), v.stride()[:3]
    a.q_out, (a.o_stride_b, a.o_stride_t, a.o_stride_h) = q_out.data_ptr(), q_out.stride()[:3]
    a.table_row, a.row_stride_b = table_row.data_ptr(), table_row.stride(0)
    a.cos_table, a.sin_table, a.table_rows = cos.data_ptr(), sin.data_ptr(), cos.shape[0]
    a.rotary_dim, a.gptj_pairs, a.n_q_heads = rotary_dim, int(gptj_pairs), Hq
    if k_stage is not None:      # staged rows [B, H, n, D]: the pool is left as it is
        a.k_stage, a.v_stage = k_stage.data_ptr(), v_stage.data_ptr()
        a.stage_stride_b, a.stage_stride_h, a.stage_stride_t = k_stage.stride()[:3]
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append_rope(_pool(pool), layer, seq_ids.data_ptr(), B, n, _ptr(n_new_per_seq),
                                            C.byref(a), _stream(pages)), "pace_kv_append_rope")


def _kv_truncate(pool, meta, layer_begin, layer_end, seq_ids, remove_len, remove_per_seq=None):
    with torch.cuda.device(meta.device):
        _C.check(_C.lib.pace_kv_truncate(_pool(pool), layer_begin, layer_end, seq_ids.data_ptr(), seq_ids.numel(),
                                         remove_len, _ptr(remove_per_seq), _stream(meta)), "pace_kv_truncate")


def _kv_gather(pool, meta, seq_ids, beam_idx):
    with torch.cuda.device(meta.device):
        _C.check(_C.lib.pace_kv_gather(_pool(pool), seq_ids.data_ptr(), beam_idx.data_ptr(), seq_ids.numel(),
                                       _stream(meta)), "pace_kv_gather")


def _pard_accept(drafts, target_next, n_target, forced, keep, target_remove, draft_remove, kept):
    B, d = drafts.shape
    with torch.cuda.device(drafts.device):
        _C.check(_C.lib.pace_pard_accept(drafts.data_ptr(), target_next.data_ptr(), n_target.data_ptr(), _ptr(forced), B, d,
                                         keep.data_ptr(), target_remove.data_ptr(), draft_remove.data_ptr(),
                                         kept.data_ptr(), _stream(drafts)), "pace_pard_accept")


def _linear_skinny(x, weight, out, workspace):
    M, K = x.shape
    N = weight.shape[0]
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_linear_skinny(x.data_ptr(), x.stride(0), weight.data_ptr(), weight.stride(0), out.data_ptr(),
                                           out.stride(0), M, N, K, workspace.data_ptr(), workspace.numel(), None,
                                           _stream(x)), "pace_linear_skinny")


def _kv_read_dense(pool, pages, layer, seq_ids, k_out, v_out):
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_read_dense(_pool(pool), layer, seq_ids.data_ptr(), seq_ids.numel(), k_out.data_ptr(),
                                           v_out.data_ptr(), k_out.shape[2], _stream(pages)), "pace_kv_read_dense")


def _step(handle: int):
    return C.byref(_C.StepStruct.from_address(handle))


def _dtype(t: torch.Tensor) -> int:
    if t.dtype == torch.bfloat16:
        return _C.DTYPE_BF16
    if t.dtype == torch.float32:
        return _C.DTYPE_FP32
    raise TypeError(f"activations must be bfloat16 or float32, got {t.dtype}")


def _residual_norm(step, x, y, w_post, embed, w_next, h, eps, restart, weight_offset, embed_scale=1.0, top=0,
                   slot_expert=None, slot_rank=None, slot_weight=None, expert_count=None, identity=None, add=None, y_bias=None,
                   embed_norm=None, w_next2=None, h2=None, y_mul=1.0):
    a = _C.ResidualNormArgs()
    a.x, a.y, a.w_post, a.embed, a.w_next, a.h = x.data_ptr(), _ptr(y), _ptr(w_post), _ptr(embed), _ptr(w_next), _ptr(h)
    a.width, a.restart, a.eps, a.weight_offset = x.shape[1], int(restart), eps, weight_offset
    a.embed_scale, a.top = embed_scale, top
    if top:
        a.n_experts = expert_count.numel()      # (identity experts are not counted here)
        a.slot_expert, a.slot_rank = slot_expert.data_ptr(), slot_rank.data_ptr()
        a.slot_weight, a.expert_count = slot_weight.data_ptr(), expert_count.data_ptr()
    a.identity, a.add, a.y_bias, a.embed_norm = _ptr(identity), _ptr(add), _ptr(y_bias), _ptr(embed_norm)
    a.w_next2, a.h2, a.y_mul = _ptr(w_next2), _ptr(h2), y_mul
    a.add_stride = add.stride(0) if add is not None else 0
    a.y_stride = y.stride(0) if y is not None else x.shape[1]
    a.vocab = embed.shape[0] if embed is not None else 0
    a.dtype = _dtype(next(t for t in (h, y, embed) if t is not None))
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_residual_norm(_step(step), C.byref(a), _stream(x)), "pace_residual_norm")


def _kv_append_norm(pool, pages, layer, step, qkv, q_norm, k_norm, q_out, dim, vdim, eps, q_mul, temp_coef, temp_every,
                    per_head=False):
    a = _C.AppendNormArgs()
    a.qkv, a.qkv_stride = qkv.data_ptr(), qkv.stride(0)
    a.q_norm, a.k_norm, a.q_out = _ptr(q_norm), _ptr(k_norm), q_out.data_ptr()
    a.n_q_heads, a.dim, a.vdim, a.dtype = q_out.shape[1], dim, vdim, _dtype(qkv)
    a.eps, a.q_mul, a.temp_coef, a.temp_every, a.per_head = eps, q_mul, temp_coef, temp_every, int(per_head)
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append_norm(_pool(pool), layer, _step(step), C.byref(a), _stream(pages)),
                 "pace_kv_append_norm")


def _attn_general(pool, pages, layer, step, q, out, dim, vdim, scale):
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_attn_general(_pool(pool), layer, _step(step), q.data_ptr(), out.data_ptr(), q.shape[1], dim,
                                          vdim, scale, _dtype(q), _stream(pages)), "pace_attn_general")


def _span_args(a, q, out, slopes, sinks, dim, vdim, scale, span, span_size, entry_begin, entry_end, max_tokens, max_keys, softcap=0.0, out_row=0):
    a.softcap, a.out_row = softcap, out_row
    a.q, a.out, a.slopes, a.sinks = q.data_ptr(), out.data_ptr(), _ptr(slopes), _ptr(sinks)
    a.n_q_heads, a.dim, a.vdim, a.dtype = q.shape[1], dim, vdim, _dtype(q)
    a.q_elems, a.out_elems = q.shape[2], out.shape[2]
    a.entry_begin, a.entry_end, a.max_tokens, a.max_keys = entry_begin, entry_end, max_tokens, max_keys
    a.span, a.span_size, a.scale = span, span_size, scale
    return a


def _attn_span(pool, pages, layer, step, q, out, *rule):
    a = _span_args(_C.AttnSpanArgs(), q, out, *rule)
    with torch.cuda.device(q.device):
        _C.check(_C.lib.pace_attn_span(_pool(pool), layer, _step(step), C.byref(a), _stream(q)), "pace_attn_span")


def _attn_span_prefill(pool, pages, layer, step, q, out, slopes, sinks, dim, vdim, scale, span, span_size, entry_begin, entry_end,
                       max_tokens, max_keys, k=None, k2=None, v=None, key_cu=None, key_pos=None, softcap=0.0, out_row=0):
    """False: the kernel does not take these shapes and nothing was launched."""
    a = _C.AttnSpanPrefillArgs()
    _span_args(a.a, q, out, slopes, sinks, dim, vdim, scale, span, span_size, entry_begin, entry_end, max_tokens, max_keys, softcap,
               out_row)
    if k is not None:
        a.k, a.k_row, a.k_head, a.k_dim = k.data_ptr(), k.stride(0), k.stride(1), k.shape[2]
        a.v, a.v_row, a.v_head = v.data_ptr(), v.stride(0), v.stride(1)
        a.n_rows, a.n_kv_heads = k.shape[:2]
        a.key_cu, a.key_pos = key_cu.data_ptr(), key_pos.data_ptr()
        if k2 is not None:
            a.k2, a.k2_row, a.k2_dim = k2.data_ptr(), k2.stride(0), k2.shape[1]
    with torch.cuda.device(q.device):
        rc = _C.lib.pace_attn_span_prefill(_pool(pool), layer, _step(step), C.byref(a), _stream(q))
        if rc != _C.PACE_ERR_UNSUPPORTED:
            _C.check(rc, "pace_attn_span_prefill")
    return rc == _C.PACE_OK


def _latent_append(pool, pages, layer, step, down, q_norm, kv_norm, cos, sin, cq, rot_dim, eps):
    a = _C.LatentAppendArgs()
    a.down, a.down_stride, a.q_norm, a.kv_norm = down.data_ptr(), down.stride(0), _ptr(q_norm), kv_norm.data_ptr()
    a.cq, a.q_rank, a.kv_rank, a.rot_dim = _ptr(cq), 0 if q_norm is None else q_norm.numel(), kv_norm.numel(), rot_dim
    if cos is not None:
        a.cos_table, a.sin_table, (a.table_rows, a.rot_pairs) = cos.data_ptr(), sin.data_ptr(), cos.shape
    a.dtype, a.eps = _dtype(down), eps
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_latent_append(_pool(pool), layer, _step(step), C.byref(a), _stream(pages)), "pace_latent_append")


def _rotate_heads(step, src, dst, cos, sin, token_begin, token_end, pad_dim):
    a = _C.RotateArgs()
    a.src, a.dst = src.data_ptr(), dst.data_ptr()
    a.src_row, a.src_head, a.dst_row, a.dst_head = src.stride(0), src.stride(1), dst.stride(0), dst.stride(1)
    a.cos_table, a.sin_table, a.token_begin, a.token_end = cos.data_ptr(), sin.data_ptr(), token_begin, token_end
    a.n_heads, a.rot_dim, a.rot_pairs, a.pad_dim = src.shape[1], src.shape[2], cos.shape[1], pad_dim
    a.table_rows, a.dtype = cos.shape[0], _dtype(src)
    with torch.cuda.device(src.device):
        _C.check(_C.lib.pace_rotate_heads(_step(step), C.byref(a), _stream(src)), "pace_rotate_heads")


def _latent_gather(pool, pages, layer, slot, pos, out):
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_latent_gather(_pool(pool), layer, slot.data_ptr(), pos.data_ptr(), pos.numel(), out.data_ptr(),
                                           _stream(pages)), "pace_latent_gather")


def _glu(x, out, act, gated=True):
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_glu(x.data_ptr(), x.stride(0), out.data_ptr(), out.stride(0), out.shape[0], out.shape[1], act,
                                 int(gated), _dtype(x), _stream(x)), "pace_glu")


def _soft_cap(x, cap):
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_soft_cap(x.data_ptr(), x.numel(), cap, _stream(x)), "pace_soft_cap")


def _part_norm_gate(o, gate, w, out, part, gate_mode, eps):
    a = _C.PartNormGateArgs()
    a.o, a.gate, a.w, a.out = o.data_ptr(), gate.data_ptr(), w.data_ptr(), out.data_ptr()
    a.o_stride, a.gate_stride, a.out_stride = o.stride(0), gate.stride(0), out.stride(0)
    a.n_tokens, a.n, a.part, a.w_period, a.gate_mode, a.dtype, a.eps = *o.shape, part, w.numel(), gate_mode, _dtype(o), eps
    with torch.cuda.device(o.device):
        _C.check(_C.lib.pace_part_norm_gate(C.byref(a), _stream(o)), "pace_part_norm_gate")


def _moe_route(logits, correction, slot_expert, slot_rank, slot_weight, expert_count, expert_list, softmax=False, weight_scale=None):
    a = _C.MoeRouteArgs()
    a.softmax, a.normalise, a.weight_scale = int(softmax), int(weight_scale is not None), weight_scale or 0.0
    a.logits, a.correction, a.slot_expert, a.slot_rank = logits.data_ptr(), _ptr(correction), slot_expert.data_ptr(), slot_rank.data_ptr()
    a.slot_weight, a.expert_count, a.expert_list = slot_weight.data_ptr(), expert_count.data_ptr(), expert_list.data_ptr()
    (a.n_tokens, a.n_experts), a.top = logits.shape, slot_expert.shape[1]
    with torch.cuda.device(logits.device):
        _C.check(_C.lib.pace_moe_route(C.byref(a), _stream(logits)), "pace_moe_route")


def _moe_experts(x, gate_up, down, hidden, y, scratch, expert_count, expert_list, slot_expert, slot_rank, status, act, gated=True):
    a = _C.MoeExpertsArgs()
    a.gated = int(gated)
    a.x, a.gate_up, a.down, a.hidden, a.y = x.data_ptr(), gate_up.data_ptr(), down.data_ptr(), hidden.data_ptr(), y.data_ptr()
    a.expert_count, a.expert_list, a.status = expert_count.data_ptr(), expert_list.data_ptr(), _ptr(status)
    a.scratch, a.slot_expert, a.slot_rank = _ptr(scratch), slot_expert.data_ptr(), slot_rank.data_ptr()
    a.n_tokens, a.width = x.shape
    a.n_experts, _, a.ff = down.shape
    a.top, a.act, a.dtype = slot_expert.shape[1], act, _dtype(x)
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_moe_experts(C.byref(a), _stream(x)), "pace_moe_experts")


def _gate_heads(step, attn, gate, out, vdim):
    with torch.cuda.device(out.device):
        _C.check(_C.lib.pace_gate_heads(_step(step), attn.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(),
                                        attn.shape[1], vdim, attn.shape[2], _dtype(attn), _stream(out)), "pace_gate_heads")


def _norm_gate(o, weight, gate, out, eps):
    with torch.cuda.device(out.device):
        _C.check(_C.lib.pace_norm_gate(o.data_ptr(), weight.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(),
                                       o.shape[0], o.shape[1], eps, _dtype(o), _stream(out)), "pace_norm_gate")


def _relu_squared(x):
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_relu_squared(x.data_ptr(), x.numel(), _dtype(x), _stream(x)), "pace_relu_squared")


def _causal_conv(step, x, taps, bias, conv_state, out, silu=False):
    a = _C.CausalConvArgs()
    a.in_, a.in_stride, a.taps, a.bias = x.data_ptr(), x.stride(0), taps.data_ptr(), _ptr(bias)
    a.conv_state, a.out, a.out_stride = conv_state.data_ptr(), out.data_ptr(), out.stride(0)
    (a.n_taps, a.channels), a.ring_rows, a.ring_stride = taps.shape, conv_state.shape[1], conv_state.stride(1)
    a.silu, a.dtype = int(silu), _dtype(x)
    with torch.cuda.device(out.device):
        _C.check(_C.lib.pace_causal_conv(_step(step), C.byref(a), _stream(out)), "pace_causal_conv")


def _conv_store(step, x, ring):
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_conv_store(_step(step), x.data_ptr(), x.stride(0), ring.data_ptr(), ring.shape[1], ring.stride(1),
                                        ring.shape[2], _dtype(x), _stream(x)), "pace_conv_store")


def _kv_append_conv(pool, pages, layer, step, qkv, taps, ring, q_norm, k_norm, cos, sin, q_out, dim, vdim, eps, v_mul, store_ring):
    a = _C.AppendConvArgs()
    a.qkv, a.qkv_stride, a.taps, a.ring = qkv.data_ptr(), qkv.stride(0), taps.data_ptr(), ring.data_ptr()
    a.q_norm, a.k_norm, a.q_out = q_norm.data_ptr(), k_norm.data_ptr(), q_out.data_ptr()
    if cos is not None:
        a.cos_table, a.sin_table, (a.table_rows, a.rot_pairs) = cos.data_ptr(), sin.data_ptr(), cos.shape
    a.n_q_heads, a.dim, a.vdim, a.n_taps = q_out.shape[1], dim, vdim, taps.shape[0]
    a.ring_rows, a.ring_stride, a.store_ring, a.dtype = ring.shape[1], ring.stride(1), int(store_ring), _dtype(qkv)
    a.eps, a.v_mul = eps, v_mul
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append_conv(_pool(pool), layer, _step(step), C.byref(a), _stream(pages)), "pace_kv_append_conv")


def _workspace(a, nbytes: int, device) -> Optional[torch.Tensor]:
    """Scratch of one launch (stream ordered: the allocator hands it out again only behind it)."""
    if not nbytes:
        return None
    ws = torch.empty(nbytes, dtype=torch.uint8, device=device)
    a.workspace, a.workspace_bytes = ws.data_ptr(), nbytes
    return ws


def _ssd(entry: str):
    fn = getattr(_C.lib, entry)

    def impl(step, xbc, dt_raw, dt_bias, neg_a, d_skip, state, out, groups, taps=None, conv_bias=None, ring=None):
        a = _C.SsdArgs()
        a.xbc, a.xbc_stride, a.dt_raw, a.dt_stride = xbc.data_ptr(), xbc.stride(0), dt_raw.data_ptr(), dt_raw.stride(0)
        a.dt_bias, a.neg_a, a.d_skip = dt_bias.data_ptr(), neg_a.data_ptr(), d_skip.data_ptr()
        a.s_state, a.out, a.out_stride = state.data_ptr(), out.data_ptr(), out.stride(0)
        (_, a.heads, a.state, a.vdim), a.groups, a.dtype = state.shape, groups, _dtype(xbc)
        if taps is not None:
            a.taps, a.conv_bias, a.ring, a.n_taps = taps.data_ptr(), _ptr(conv_bias), ring.data_ptr(), taps.shape[0]
            a.ring_rows, a.ring_stride = ring.shape[1], ring.stride(1)
        with torch.cuda.device(out.device):
            st = _C.StepStruct.from_address(step)
            ws = None
            if taps is None and a.dtype == _C.DTYPE_BF16:
                ws = _workspace(a, _C.lib.pace_ssd_workspace_bytes(st.n_entries, st.max_count, a.heads, a.state, a.vdim), out.device)
            _C.check(fn(_step(step), C.byref(a), _stream(out)), entry)
            del ws
    return impl


def _delta(entry: str):
    fn = getattr(_C.lib, entry)

    def impl(step, qkv, a_raw, b_raw, dt_bias, neg_a, state, out, kv_heads, unit_eps, q_scale, taps=None, ring=None):
        a = _C.DeltaArgs()
        a.qkv, a.qkv_stride, a.a_raw, a.a_stride = qkv.data_ptr(), qkv.stride(0), a_raw.data_ptr(), a_raw.stride(0)
        a.b_raw, a.b_stride, a.dt_bias, a.neg_a = b_raw.data_ptr(), b_raw.stride(0), dt_bias.data_ptr(), neg_a.data_ptr()
        a.s_state, a.out, a.out_stride = state.data_ptr(), out.data_ptr(), out.stride(0)
        (_, a.heads, a.dim, a.vdim), a.kv_heads, a.dtype = state.shape, kv_heads, _dtype(qkv)
        a.unit_eps, a.q_scale = unit_eps, q_scale
        if taps is not None:
            a.taps, a.ring, a.n_taps, a.ring_rows, a.ring_stride = taps.data_ptr(), ring.data_ptr(), taps.shape[0], ring.shape[1], ring.stride(1)
        with torch.cuda.device(out.device):
            st = _C.StepStruct.from_address(step)
            ws = None
            if taps is None:
                ws = _workspace(a, _C.lib.pace_delta_workspace_bytes(st.n_entries, st.max_count, a.heads, a.dim, a.vdim, a.dtype),
                                out.device)
            _C.check(fn(_step(step), C.byref(a), _stream(out)), entry)
            del ws
    return impl


def _gla(entry: str):
    fn = getattr(_C.lib, entry)

    def impl(step, qkv, z, z_bias, state, out, inv_tau, q_scale, norm=None, gate=None, eps=0.0):
        a = _C.GlaArgs()
        a.qkv, a.qkv_stride, a.z, a.z_stride = qkv.data_ptr(), qkv.stride(0), z.data_ptr(), z.stride(0)
        a.z_bias, a.s_state, a.out, a.out_stride = z_bias.data_ptr(), state.data_ptr(), out.data_ptr(), out.stride(0)
        (_, a.heads, a.dim, a.vdim), a.dtype = state.shape, _dtype(qkv)
        a.inv_tau, a.q_scale, a.eps = inv_tau, q_scale, eps
        if norm is not None:
            a.norm, a.gate, a.gate_stride = norm.data_ptr(), gate.data_ptr(), gate.stride(0)
        with torch.cuda.device(out.device):
            st = _C.StepStruct.from_address(step)
            ws = None
            if norm is None:
                ws = _workspace(a, _C.lib.pace_gla_workspace_bytes(st.n_entries, st.max_count, a.heads, a.dim, a.dtype), out.device)
            _C.check(fn(_step(step), C.byref(a), _stream(out)), entry)
            del ws
    return impl


def _kv_append_rotate(pool, pages, layer, blocks, block_pages, block_layer, step, qkv, cos, sin, q_out, dim, vdim, halves, block, block_now):
    a = _C.AppendRotateArgs()
    a.qkv, a.qkv_stride, a.q_out = qkv.data_ptr(), qkv.stride(0), q_out.data_ptr()
    if cos is not None:
        a.cos_table, a.sin_table, (a.table_rows, a.rot_pairs) = cos.data_ptr(), sin.data_ptr(), cos.shape
    a.n_q_heads, a.dim, a.vdim, a.halves = q_out.shape[1], dim, vdim, int(halves)
    a.block, a.block_now, a.dtype = block, int(block_now), _dtype(qkv)
    with torch.cuda.device(pages.device):
        _C.check(_C.lib.pace_kv_append_rotate(_pool(pool), layer, _pool(blocks) if block else None, block_layer, _step(step), C.byref(a),
                                              _stream(pages)), "pace_kv_append_rotate")


def _pooled_args(q, out, gate, sinks, mix, dim, vdim, scale, window, block, max_keys):
    a = _C.AttnPooledArgs()
    a.q, a.out, a.sinks, a.mix, a.out_stride = q.data_ptr(), out.data_ptr(), _ptr(sinks), _ptr(mix), out.stride(0)
    if gate is not None:
        a.gate, a.gate_stride = gate.data_ptr(), gate.stride(0)
    (_, a.n_q_heads, a.q_elems), a.dim, a.vdim, a.dtype = q.shape, dim, vdim, _dtype(q)
    a.window, a.block, a.max_keys, a.scale = window, block, max_keys, scale
    return a


def _attn_pooled(pool, pages, layer, blocks, block_pages, block_layer, step, q, out, gate, sinks, mix, dim, vdim, scale, window, block,
                 token_begin, token_end, max_keys):
    a = _pooled_args(q, out, gate, sinks, mix, dim, vdim, scale, window, block, max_keys)
    a.token_begin, a.token_end = token_begin, token_end
    with torch.cuda.device(q.device):
        _C.check(_C.lib.pace_attn_pooled(_pool(pool), layer, _pool(blocks) if block else None, block_layer, _step(step), C.byref(a),
                                         _stream(q)), "pace_attn_pooled")


def _attn_pooled_prompt(pool, pages, layer, blocks, block_pages, block_layer, step, q, out, gate, sinks, mix, dim, vdim, scale, window,
                        block, entry_begin, entry_end, max_tokens, max_keys):
    """False: the kernel does not take these shapes and nothing was launched."""
    a = _pooled_args(q, out, gate, sinks, mix, dim, vdim, scale, window, block, max_keys)
    a.entry_begin, a.entry_end, a.max_tokens = entry_begin, entry_end, max_tokens
    with torch.cuda.device(q.device):
        ws = _workspace(a, _C.lib.pace_attn_pooled_prompt_workspace_bytes(
            entry_end - entry_begin, max_tokens, q.shape[1], _C.KVPoolStruct.from_address(pool).n_kv_heads, vdim, int(mix is not None)), q.device)
        rc = _C.lib.pace_attn_pooled_prompt(_pool(pool), layer, _pool(blocks) if block else None, block_layer, _step(step), C.byref(a),
                                            _stream(q))
        if rc != _C.PACE_ERR_UNSUPPORTED:
            _C.check(rc, "pace_attn_pooled_prompt")
        del ws
    return rc == _C.PACE_OK


def _shift_norm(step, x_in, x_out, y, y_bias, w_post, add, w_next, shift, state, state_out, h, eps):
    a = _C.ShiftNormArgs()
    a.x_in, a.x_out, a.w_next, a.shift, a.h = x_in.data_ptr(), x_out.data_ptr(), w_next.data_ptr(), shift.data_ptr(), h.data_ptr()
    a.state, a.state_out, a.state_stride = state.data_ptr(), state_out.data_ptr(), state.stride(0)
    a.y_bias, a.w_post, a.add = _ptr(y_bias), _ptr(w_post), _ptr(add)
    if y is not None:
        a.y, a.y_stride = y.data_ptr(), y.stride(0)
    a.width, a.dtype, a.eps = x_in.shape[1], _dtype(h), eps
    with torch.cuda.device(h.device):
        _C.check(_C.lib.pace_shift_norm(_step(step), C.byref(a), _stream(h)), "pace_shift_norm")


def _embed_pairs(step, x, embed, scale, pairs, last_token, mul_prev, mul_cur, store_last):
    a = _C.EmbedPairsArgs()
    a.x, a.embed, a.pairs, a.last_token = x.data_ptr(), embed.data_ptr(), _ptr(pairs), _ptr(last_token)
    a.mul_prev, a.mul_cur, (a.vocab, a.width), a.store_last = mul_prev, mul_cur, embed.shape, int(store_last)
    a.buckets, a.dtype, a.scale = pairs.shape[0] - 1 if pairs is not None else 0, _dtype(embed), scale
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_embed_pairs(_step(step), C.byref(a), _stream(x)), "pace_embed_pairs")


def _state_commit(step, source, target, last_token=None):
    with torch.cuda.device(target.device):
        _C.check(_C.lib.pace_state_commit(_step(step), source.data_ptr(), target.data_ptr(), source[0].numel(), source.stride(0),
                                          _ptr(last_token), _stream(target)), "pace_state_commit")


def _gate_per_head(x, gate):
    with torch.cuda.device(x.device):
        _C.check(_C.lib.pace_gate_per_head(x.data_ptr(), gate.data_ptr(), gate.stride(0), *x.shape, _dtype(x), _stream(x)),
                 "pace_gate_per_head")


def _rglru_args(yx, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks):
    a = _C.RglruArgs()
    a.yx, a.yx_stride = yx.data_ptr(), yx.stride(0)
    a.ra_bias, a.ri_bias, a.decay_base = ra_bias.data_ptr(), ri_bias.data_ptr(), decay_base.data_ptr()
    a.state, a.conv_state, a.out = state.data_ptr(), conv_state.data_ptr(), out.data_ptr()
    a.width, a.blocks, a.n_taps, a.dtype = out.shape[1], blocks, conv_state.shape[1], _dtype(yx)
    return a


def _rglru_scan(step, yx, u, gates, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks):
    a = _rglru_args(yx, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks)
    a.u, a.gates = u.data_ptr(), gates.data_ptr()
    with torch.cuda.device(out.device):
        _C.check(_C.lib.pace_rglru_scan(_step(step), C.byref(a), _stream(out)), "pace_rglru_scan")


def _rglru_step(step, yx, gate_w, taps, conv_bias, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks):
    a = _rglru_args(yx, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks)
    a.gate_w, a.taps, a.conv_bias = gate_w.data_ptr(), taps.data_ptr(), conv_bias.data_ptr()
    with torch.cuda.device(out.device):
        _C.check(_C.lib.pace_rglru_step(_step(step), C.byref(a), _stream(out)), "pace_rglru_step")


def _lightning(entry: str):
    fn = getattr(_C.lib, entry)

    def impl(step, qkv, decay, state, out):
        a = _C.LightningArgs()
        a.qkv, a.qkv_stride, a.decay = qkv.data_ptr(), qkv.stride(0), decay.data_ptr()
        a.state, a.out = state.data_ptr(), out.data_ptr()
        _, a.heads, a.dim, a.vdim = state.shape
        a.dtype = _dtype(qkv)
        with torch.cuda.device(out.device):
            st = _C.StepStruct.from_address(step)
            n = 0 if st.max_count == 1 else _C.lib.pace_lightning_workspace_bytes(st.n_entries, st.max_count, a.heads, a.dim,
                                                                                  a.vdim)
            if n:        # (stream ordered: the allocator hands it out again only behind this launch)
                ws = torch.empty(n // 4, dtype=torch.float32, device=out.device)
                a.workspace, a.workspace_bytes = ws.data_ptr(), n
            _C.check(fn(_step(step), C.byref(a), _stream(out)), entry)
    return impl


def _step_decode(token, tok_pos, start, next_token, position):
    with torch.cuda.device(token.device):
        _C.check(_C.lib.pace_step_decode(token.data_ptr(), tok_pos.data_ptr(), start.data_ptr(), next_token.data_ptr(),
                                         position.data_ptr(), token.numel(), _stream(token)), "pace_step_decode")


def _attn(entry: str):
    fn = getattr(_C.lib, entry)

    def impl(pool, pages, layer, q, out, seq_ids, kv_start, q_lens, workspace, scale, flags, k_pending, v_pending,
             max_ctas):
        B, Hq, S, D = q.shape
        a = _C.AttnArgs()
        a.pool = C.pointer(_C.KVPoolStruct.from_address(pool))
        a.layer, a.batch, a.n_q_heads, a.q_len = layer, B, Hq, S
        a.seq_ids, a.kv_start, a.q_lens = _ptr(seq_ids), _ptr(kv_start), _ptr(q_lens)
        a.q = q.data_ptr()
        a.q_stride_b, a.q_stride_h, a.q_stride_s = q.stride(0), q.stride(1), q.stride(2)
        a.out = out.data_ptr()
        a.o_stride_b, a.o_stride_h, a.o_stride_s = out.stride(0), out.stride(1), out.stride(2)
        a.scale = float(scale) if scale > 0 else 1.0 / math.sqrt(D)
        a.workspace, a.workspace_bytes = workspace.data_ptr(), workspace.numel()
        a.flags, a.max_ctas = int(flags), int(max_ctas)
        if k_pending is not None:
            a.k_pending, a.v_pending = k_pending.data_ptr(), v_pending.data_ptr()
            a.pending_stride_b, a.pending_stride_h = k_pending.stride(0), k_pending.stride(1)
        with torch.cuda.device(q.device):
            _C.check(fn(C.byref(a), _stream(q)), entry)
    return impl


_IMPLS = {"kv_reserve": _kv_reserve, "kv_append": _kv_append, "kv_append_layers": _kv_append_layers,
          "kv_append_rope": _kv_append_rope, "kv_truncate": _kv_truncate, "kv_gather": _kv_gather,
          "kv_read_dense": _kv_read_dense, "pard_accept": _pard_accept, "linear_skinny": _linear_skinny, "attn_decode": _attn("pace_attn_decode"),
          "attn_decode_cuda_cores": _attn("pace_attn_decode_cuda_cores"), "attn_verify": _attn("pace_attn_verify"),
          "attn_prefill": _attn("pace_attn_prefill"), "residual_norm": _residual_norm, "kv_append_norm": _kv_append_norm,
          "attn_general": _attn_general, "gate_heads": _gate_heads, "norm_gate": _norm_gate, "relu_squared": _relu_squared,
          "causal_conv": _causal_conv, "rglru_scan": _rglru_scan, "rglru_step": _rglru_step,
          "lightning_prefill": _lightning("pace_lightning_prefill"), "lightning_step": _lightning("pace_lightning_step"),
          "step_decode": _step_decode, "attn_span": _attn_span, "attn_span_prefill": _attn_span_prefill,
          "latent_append": _latent_append, "rotate_heads": _rotate_heads, "latent_gather": _latent_gather, "glu": _glu,
          "moe_route": _moe_route, "moe_experts": _moe_experts, "soft_cap": _soft_cap, "part_norm_gate": _part_norm_gate,
          "kv_append_conv": _kv_append_conv, "conv_store": _conv_store, "ssd_prefill": _ssd("pace_ssd_prefill"),
          "ssd_step": _ssd("pace_ssd_step"), "delta_prefill": _delta("pace_delta_prefill"), "delta_step": _delta("pace_delta_step"),
          "gla_prefill": _gla("pace_gla_prefill"), "gla_step": _gla("pace_gla_step"), "kv_append_rotate": _kv_append_rotate,
          "attn_pooled": _attn_pooled, "attn_pooled_prompt": _attn_pooled_prompt, "shift_norm": _shift_norm, "embed_pairs": _embed_pairs, "state_commit": _state_commit,
          "gate_per_head": _gate_per_head}
for _n, _f in _IMPLS.items():
    _lib.impl(_n, _f, "CUDA")
    # shape propagation for tracers: nothing is returned, nothing to compute
    _lib.impl(_n, (lambda *a, **k: None), "Meta")

OPS = tuple(_DEFS)
