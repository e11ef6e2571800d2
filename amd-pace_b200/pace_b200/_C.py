"""ctypes binding of libpace_b200.so (C ABI: include/pace_b200.h).

Plays the role of the reference's compiled extension module `pace._C`
(csrc/torch_extension_bindings.cpp): the Python layer above never touches CUDA
directly, it hands raw device pointers, sizes and the current stream to these
functions.
"""
import ctypes as C
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "libpace_b200.so")

if not os.path.exists(LIB_PATH):
    raise ImportError(
        f"{LIB_PATH} is missing: build it with `python amd-pace_b200/build.py` "
        "(there is no CPU or PyTorch fallback for these ops)")

lib = C.CDLL(LIB_PATH)

PACE_OK, PACE_ERR_INVALID, PACE_ERR_CUDA, PACE_ERR_UNSUPPORTED = 0, 1, 2, 3
DEV_POOL_EXHAUSTED, DEV_OVER_REMOVE, DEV_BAD_INDEX, DEV_TABLE_FULL, DEV_WAIT_TIMEOUT = 1, 2, 4, 8, 16
_DEV_NAMES = {1: "pool exhausted", 2: "over-removal", 4: "bad slot/page index", 8: "block table full",
              16: "in-kernel wait timed out"}


class KVPoolStruct(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_layers", "n_kv_heads", "head_dim", "page_tokens", "n_pages",
                                          "max_seqs", "max_pages_per_seq", "owns_memory")] + \
               [(n, C.c_void_p) for n in ("pages", "block_table", "seq_len", "seq_pages", "page_ref",
                                          "free_stack", "counters", "status", "table_tmp")] + \
               [("row_format", C.c_int32), ("row_tokens", C.c_int32)]


ROWS_BF16, ROWS_OPAQUE, ROWS_SHARED = 0, 1, 2   # PACE_ROWS_*
DTYPE_BF16, DTYPE_FP32 = 0, 1   # PACE_DTYPE_*
SPAN_ALL, SPAN_WINDOW, SPAN_CHUNK = 0, 1, 2   # PACE_SPAN_*
ACT_SILU, ACT_GELU_TANH, ACT_GELU_ERF = 0, 1, 2  # PACE_ACT_*
GATE_SIGMOID, GATE_SILU_FIRST, GATE_SILU = 0, 1, 2  # PACE_GATE_*

ATTN_WHOLE_UNITS = 1      # PACE_ATTN_WHOLE_UNITS
ATTN_PENDING_ROW = 2      # PACE_ATTN_PENDING_ROW
ATTN_NO_EARLY_KV = 4      # PACE_ATTN_NO_EARLY_KV
ATTN_ONE_CTA_PER_SM = 8   # PACE_ATTN_ONE_CTA_PER_SM
ATTN_SPLIT_WEIGHTS = 16   # PACE_ATTN_SPLIT_WEIGHTS


class AttnArgs(C.Structure):
    _fields_ = [("pool", C.POINTER(KVPoolStruct)), ("layer", C.c_int32), ("batch", C.c_int32),
                ("n_q_heads", C.c_int32), ("q_len", C.c_int32), ("seq_ids", C.c_void_p),
                ("kv_start", C.c_void_p), ("q_lens", C.c_void_p), ("q", C.c_void_p),
                ("q_stride_b", C.c_int64), ("q_stride_h", C.c_int64), ("q_stride_s", C.c_int64),
                ("out", C.c_void_p), ("o_stride_b", C.c_int64), ("o_stride_h", C.c_int64),
                ("o_stride_s", C.c_int64), ("scale", C.c_float), ("workspace", C.c_void_p),
                ("workspace_bytes", C.c_uint64), ("flags", C.c_uint32),
                ("k_pending", C.c_void_p), ("v_pending", C.c_void_p),
                ("pending_stride_b", C.c_int64), ("pending_stride_h", C.c_int64), ("max_ctas", C.c_int32)]


class RopeArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("q_stride_b", C.c_int64), ("q_stride_t", C.c_int64), ("q_stride_h", C.c_int64),
                ("k", C.c_void_p), ("k_stride_b", C.c_int64), ("k_stride_t", C.c_int64), ("k_stride_h", C.c_int64),
                ("v", C.c_void_p), ("v_stride_b", C.c_int64), ("v_stride_t", C.c_int64), ("v_stride_h", C.c_int64),
                ("q_out", C.c_void_p), ("o_stride_b", C.c_int64), ("o_stride_t", C.c_int64),
                ("o_stride_h", C.c_int64), ("table_row", C.c_void_p), ("row_stride_b", C.c_int64),
                ("cos_table", C.c_void_p), ("sin_table", C.c_void_p), ("table_rows", C.c_int32),
                ("rotary_dim", C.c_int32), ("gptj_pairs", C.c_int32), ("n_q_heads", C.c_int32),
                ("k_stage", C.c_void_p), ("v_stage", C.c_void_p), ("stage_stride_b", C.c_int64),
                ("stage_stride_h", C.c_int64), ("stage_stride_t", C.c_int64)]


class StepStruct(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_tokens", "n_entries", "max_count", "reserved")] + \
               [(n, C.c_void_p) for n in ("token", "tok_entry", "tok_pos", "q_row", "cu", "start", "slot")]


class ResidualNormArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x", "y", "w_post", "embed", "w_next", "h")] + [("y_stride", C.c_int64)] + \
               [(n, C.c_int32) for n in ("width", "vocab", "restart", "dtype")] + \
               [("eps", C.c_float), ("weight_offset", C.c_float), ("embed_scale", C.c_float), ("top", C.c_int32),
                ("n_experts", C.c_int32)] + \
               [(n, C.c_void_p) for n in ("slot_expert", "slot_rank", "slot_weight", "expert_count", "identity", "add")] + \
               [("add_stride", C.c_int64)] + [(n, C.c_void_p) for n in ("y_bias", "embed_norm", "w_next2", "h2")] + \
               [("y_mul", C.c_float)]


class AppendNormArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("q_norm", "k_norm", "q_out")] + \
               [(n, C.c_int32) for n in ("n_q_heads", "dim", "vdim", "dtype")] + \
               [("eps", C.c_float), ("q_mul", C.c_float), ("temp_coef", C.c_float), ("temp_every", C.c_double),
                ("per_head", C.c_int32)]


class AttnSpanArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "out", "slopes", "sinks")] + \
               [(n, C.c_int32) for n in ("n_q_heads", "dim", "vdim", "dtype", "q_elems", "out_elems", "entry_begin", "entry_end",
                                         "max_tokens", "max_keys", "span", "span_size")] + \
               [("scale", C.c_float), ("softcap", C.c_float), ("out_row", C.c_int64)]


class AttnSpanPrefillArgs(C.Structure):
    _fields_ = [("a", AttnSpanArgs)] + [(n, C.c_void_p) for n in ("k", "k2", "v")] + \
               [(n, C.c_int64) for n in ("k_row", "k_head", "k2_row", "v_row", "v_head")] + \
               [(n, C.c_int32) for n in ("k_dim", "k2_dim", "n_kv_heads", "n_rows")] + \
               [("key_cu", C.c_void_p), ("key_pos", C.c_void_p)]


class LatentAppendArgs(C.Structure):
    _fields_ = [("down", C.c_void_p), ("down_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("q_norm", "kv_norm", "cos_table", "sin_table", "cq")] + \
               [(n, C.c_int32) for n in ("q_rank", "kv_rank", "rot_dim", "rot_pairs", "table_rows", "dtype")] + \
               [("eps", C.c_float)]


class RotateArgs(C.Structure):
    _fields_ = [("src", C.c_void_p), ("dst", C.c_void_p)] + \
               [(n, C.c_int64) for n in ("src_row", "src_head", "dst_row", "dst_head")] + \
               [("cos_table", C.c_void_p), ("sin_table", C.c_void_p)] + \
               [(n, C.c_int32) for n in ("token_begin", "token_end", "n_heads", "rot_dim", "rot_pairs", "pad_dim", "table_rows",
                                         "dtype")]


class MoeRouteArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("logits", "correction", "slot_expert", "slot_rank", "slot_weight", "expert_count",
                                          "expert_list")] + \
               [(n, C.c_int32) for n in ("n_tokens", "n_experts", "top", "softmax", "normalise")] + [("weight_scale", C.c_float)]


class MoeExpertsArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x", "gate_up", "down", "hidden", "y", "scratch", "expert_count", "expert_list", "slot_expert",
                                          "slot_rank", "status")] + \
               [(n, C.c_int32) for n in ("n_tokens", "n_experts", "top", "width", "ff", "act", "dtype", "gated")]


class RglruArgs(C.Structure):
    _fields_ = [("yx", C.c_void_p), ("yx_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("u", "gates", "gate_w", "taps", "conv_bias", "ra_bias", "ri_bias", "decay_base",
                                          "state", "conv_state", "out")] + \
               [(n, C.c_int32) for n in ("width", "blocks", "n_taps", "dtype")]


class LightningArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64), ("decay", C.c_void_p), ("state", C.c_void_p),
                ("out", C.c_void_p), ("workspace", C.c_void_p), ("workspace_bytes", C.c_uint64)] + \
               [(n, C.c_int32) for n in ("heads", "dim", "vdim", "dtype")]


class CausalConvArgs(C.Structure):
    _fields_ = [("in_", C.c_void_p), ("in_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("taps", "bias", "conv_state", "out")] + [("out_stride", C.c_int64)] + \
               [(n, C.c_int32) for n in ("n_taps", "channels", "ring_rows", "ring_stride", "silu", "dtype")]


class AppendConvArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("taps", "ring", "q_norm", "k_norm", "cos_table", "sin_table", "q_out")] + \
               [(n, C.c_int32) for n in ("n_q_heads", "dim", "vdim", "n_taps", "ring_rows", "ring_stride", "rot_pairs", "table_rows",
                                         "store_ring", "dtype")] + [("eps", C.c_float), ("v_mul", C.c_float)]


class PartNormGateArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("o", "gate", "w", "out")] + \
               [(n, C.c_int64) for n in ("o_stride", "gate_stride", "out_stride")] + \
               [(n, C.c_int32) for n in ("n_tokens", "n", "part", "w_period", "gate_mode", "dtype")] + [("eps", C.c_float)]


class SsdArgs(C.Structure):
    _fields_ = [("xbc", C.c_void_p), ("xbc_stride", C.c_int64), ("dt_raw", C.c_void_p), ("dt_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("dt_bias", "neg_a", "d_skip", "s_state", "out")] + [("out_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("taps", "conv_bias", "ring", "workspace")] + [("workspace_bytes", C.c_uint64)] + \
               [(n, C.c_int32) for n in ("heads", "groups", "state", "vdim", "n_taps", "ring_rows", "ring_stride", "dtype")]


class DeltaArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64), ("a_raw", C.c_void_p), ("a_stride", C.c_int64),
                ("b_raw", C.c_void_p), ("b_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("dt_bias", "neg_a", "s_state", "out")] + [("out_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("taps", "ring", "workspace")] + [("workspace_bytes", C.c_uint64)] + \
               [(n, C.c_int32) for n in ("heads", "kv_heads", "dim", "vdim", "n_taps", "ring_rows", "ring_stride", "dtype")] + \
               [("unit_eps", C.c_float), ("q_scale", C.c_float)]


class GlaArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64), ("z", C.c_void_p), ("z_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("z_bias", "s_state", "out")] + [("out_stride", C.c_int64)] + \
               [("norm", C.c_void_p), ("gate", C.c_void_p), ("gate_stride", C.c_int64), ("workspace", C.c_void_p),
                ("workspace_bytes", C.c_uint64)] + \
               [(n, C.c_int32) for n in ("heads", "dim", "vdim", "dtype")] + [(n, C.c_float) for n in ("inv_tau", "q_scale", "eps")]


class AppendRotateArgs(C.Structure):
    _fields_ = [("qkv", C.c_void_p), ("qkv_stride", C.c_int64)] + [(n, C.c_void_p) for n in ("cos_table", "sin_table", "q_out")] + \
               [(n, C.c_int32) for n in ("n_q_heads", "dim", "vdim", "rot_pairs", "halves", "table_rows", "block", "block_now", "dtype")]


class AttnPooledArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("q", "out", "gate", "sinks", "mix")] + [("out_stride", C.c_int64), ("gate_stride", C.c_int64)] + \
               [(n, C.c_int32) for n in ("n_q_heads", "dim", "vdim", "dtype", "q_elems", "window", "block", "token_begin", "token_end",
                                         "entry_begin", "entry_end", "max_tokens", "max_keys")] + \
               [("scale", C.c_float), ("workspace", C.c_void_p), ("workspace_bytes", C.c_uint64)]


class ShiftNormArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x_in", "x_out", "y")] + [("y_stride", C.c_int64)] + \
               [(n, C.c_void_p) for n in ("y_bias", "w_post", "add", "w_next", "shift", "state", "state_out")] + \
               [("state_stride", C.c_int64), ("h", C.c_void_p), ("width", C.c_int32), ("dtype", C.c_int32), ("eps", C.c_float)]


class EmbedPairsArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x", "embed", "pairs", "last_token")] + [("mul_prev", C.c_int64), ("mul_cur", C.c_int64)] + \
               [(n, C.c_int32) for n in ("width", "vocab", "buckets", "store_last", "dtype")] + [("scale", C.c_float)]


byref = C.byref
_S = C.POINTER(StepStruct)
_P = C.POINTER(KVPoolStruct)
_SIGS = {
    "pace_last_cuda_error": (C.c_char_p, []),
    "pace_version": (C.c_char_p, []),
    "pace_kv_pool_bytes": (C.c_int, [_P, C.POINTER(C.c_uint64), C.POINTER(C.c_uint64)]),
    "pace_kv_pool_bind": (C.c_int, [_P, C.c_void_p, C.c_void_p]),
    "pace_kv_pool_create": (C.c_int, [_P]),
    "pace_kv_pool_destroy": (C.c_int, [_P]),
    "pace_kv_pool_reset": (C.c_int, [_P, C.c_void_p]),
    "pace_kv_pool_query": (C.c_int, [_P, C.POINTER(C.c_int32 * 4), C.c_void_p]),
    "pace_kv_pool_clear_status": (C.c_int, [_P, C.c_void_p]),
    "pace_selftest_wait_timeout": (C.c_int, [_P, C.c_int32, C.c_void_p]),
    "pace_kv_seq_release": (C.c_int, [_P, C.c_void_p, C.c_int32, C.c_void_p]),
    "pace_kv_reserve": (C.c_int, [_P, C.c_int32, C.c_void_p, C.c_int32, C.c_int32, C.c_void_p, C.c_void_p]),
    "pace_kv_append": (C.c_int, [_P, C.c_int32, C.c_void_p, C.c_int32, C.c_int32, C.c_void_p, C.c_void_p,
                                 C.c_void_p, C.c_int64, C.c_int64, C.c_int64, C.c_void_p]),
    "pace_kv_append_layers": (C.c_int, [_P, C.c_int32, C.c_int32, C.c_void_p, C.c_int32, C.c_int32, C.c_void_p,
                                        C.c_void_p, C.c_void_p, C.c_int64, C.c_int64, C.c_int64, C.c_int64,
                                        C.c_void_p]),
    "pace_kv_append_rope": (C.c_int, [_P, C.c_int32, C.c_void_p, C.c_int32, C.c_int32, C.c_void_p,
                                      C.POINTER(RopeArgs), C.c_void_p]),
    "pace_kv_truncate": (C.c_int, [_P, C.c_int32, C.c_int32, C.c_void_p, C.c_int32, C.c_int32, C.c_void_p,
                                   C.c_void_p]),
    "pace_pard_accept": (C.c_int, [C.c_void_p] * 4 + [C.c_int32, C.c_int32] + [C.c_void_p] * 5),
    "pace_kv_gather": (C.c_int, [_P, C.c_void_p, C.c_void_p, C.c_int32, C.c_void_p]),
    "pace_kv_read_dense": (C.c_int, [_P, C.c_int32, C.c_void_p, C.c_int32, C.c_void_p, C.c_void_p, C.c_int32,
                                     C.c_void_p]),
    "pace_attn_workspace_bytes": (C.c_uint64, [C.c_int32] * 5),
    "pace_attn_decode": (C.c_int, [C.POINTER(AttnArgs), C.c_void_p]),
    "pace_attn_decode_cuda_cores": (C.c_int, [C.POINTER(AttnArgs), C.c_void_p]),
    "pace_attn_decode_static": (C.c_int, [C.POINTER(AttnArgs), C.c_void_p]),
    "pace_attn_verify": (C.c_int, [C.POINTER(AttnArgs), C.c_void_p]),
    "pace_attn_prefill": (C.c_int, [C.POINTER(AttnArgs), C.c_void_p]),
    "pace_profile_enabled": (C.c_int, []),
    "pace_profile_flush": (C.c_int, []),
    "pace_linear_workspace_bytes": (C.c_uint64, [C.c_int32]),
    "pace_linear_skinny": (C.c_int, [C.c_void_p, C.c_int64, C.c_void_p, C.c_int64, C.c_void_p, C.c_int64, C.c_int32,
                                     C.c_int32, C.c_int32, C.c_void_p, C.c_uint64, C.c_void_p, C.c_void_p]),
    "pace_residual_norm": (C.c_int, [_S, C.POINTER(ResidualNormArgs), C.c_void_p]),
    "pace_kv_append_norm": (C.c_int, [_P, C.c_int32, _S, C.POINTER(AppendNormArgs), C.c_void_p]),
    "pace_attn_general": (C.c_int, [_P, C.c_int32, _S, C.c_void_p, C.c_void_p, C.c_int32, C.c_int32, C.c_int32, C.c_float,
                                    C.c_int32, C.c_void_p]),
    "pace_attn_span": (C.c_int, [_P, C.c_int32, _S, C.POINTER(AttnSpanArgs), C.c_void_p]),
    "pace_attn_span_prefill": (C.c_int, [_P, C.c_int32, _S, C.POINTER(AttnSpanPrefillArgs), C.c_void_p]),
    "pace_latent_append": (C.c_int, [_P, C.c_int32, _S, C.POINTER(LatentAppendArgs), C.c_void_p]),
    "pace_rotate_heads": (C.c_int, [_S, C.POINTER(RotateArgs), C.c_void_p]),
    "pace_latent_gather": (C.c_int, [_P, C.c_int32, C.c_void_p, C.c_void_p, C.c_int32, C.c_void_p, C.c_void_p]),
    "pace_glu": (C.c_int, [C.c_void_p, C.c_int64, C.c_void_p, C.c_int64] + [C.c_int32] * 5 + [C.c_void_p]),
    "pace_soft_cap": (C.c_int, [C.c_void_p, C.c_int64, C.c_float, C.c_void_p]),
    "pace_part_norm_gate": (C.c_int, [C.POINTER(PartNormGateArgs), C.c_void_p]),
    "pace_kv_append_conv": (C.c_int, [_P, C.c_int32, _S, C.POINTER(AppendConvArgs), C.c_void_p]),
    "pace_ssd_workspace_bytes": (C.c_uint64, [C.c_int32] * 5),
    "pace_ssd_prefill": (C.c_int, [_S, C.POINTER(SsdArgs), C.c_void_p]),
    "pace_ssd_step": (C.c_int, [_S, C.POINTER(SsdArgs), C.c_void_p]),
    "pace_delta_workspace_bytes": (C.c_uint64, [C.c_int32] * 6),
    "pace_delta_prefill": (C.c_int, [_S, C.POINTER(DeltaArgs), C.c_void_p]),
    "pace_delta_step": (C.c_int, [_S, C.POINTER(DeltaArgs), C.c_void_p]),
    "pace_gla_workspace_bytes": (C.c_uint64, [C.c_int32] * 5),
    "pace_gla_prefill": (C.c_int, [_S, C.POINTER(GlaArgs), C.c_void_p]),
    "pace_gla_step": (C.c_int, [_S, C.POINTER(GlaArgs), C.c_void_p]),
    "pace_kv_append_rotate": (C.c_int, [_P, C.c_int32, _P, C.c_int32, _S, C.POINTER(AppendRotateArgs), C.c_void_p]),
    "pace_attn_pooled": (C.c_int, [_P, C.c_int32, _P, C.c_int32, _S, C.POINTER(AttnPooledArgs), C.c_void_p]),
    "pace_attn_pooled_prompt_workspace_bytes": (C.c_uint64, [C.c_int32] * 6),
    "pace_attn_pooled_prompt": (C.c_int, [_P, C.c_int32, _P, C.c_int32, _S, C.POINTER(AttnPooledArgs), C.c_void_p]),
    "pace_shift_norm": (C.c_int, [_S, C.POINTER(ShiftNormArgs), C.c_void_p]),
    "pace_embed_pairs": (C.c_int, [_S, C.POINTER(EmbedPairsArgs), C.c_void_p]),
    "pace_state_commit": (C.c_int, [_S, C.c_void_p, C.c_void_p, C.c_int64, C.c_int64, C.c_void_p, C.c_void_p]),
    "pace_gate_per_head": (C.c_int, [C.c_void_p, C.c_void_p, C.c_int64] + [C.c_int32] * 4 + [C.c_void_p]),
    "pace_moe_route": (C.c_int, [C.POINTER(MoeRouteArgs), C.c_void_p]),
    "pace_moe_experts": (C.c_int, [C.POINTER(MoeExpertsArgs), C.c_void_p]),
    "pace_gate_heads": (C.c_int, [_S, C.c_void_p, C.c_void_p, C.c_int64, C.c_void_p, C.c_int32, C.c_int32, C.c_int32,
                                  C.c_int32, C.c_void_p]),
    "pace_norm_gate": (C.c_int, [C.c_void_p, C.c_void_p, C.c_void_p, C.c_int64, C.c_void_p, C.c_int32, C.c_int32, C.c_float,
                                 C.c_int32, C.c_void_p]),
    "pace_relu_squared": (C.c_int, [C.c_void_p, C.c_int64, C.c_int32, C.c_void_p]),
    "pace_causal_conv": (C.c_int, [_S, C.POINTER(CausalConvArgs), C.c_void_p]),
    "pace_conv_store": (C.c_int, [_S, C.c_void_p, C.c_int64, C.c_void_p] + [C.c_int32] * 4 + [C.c_void_p]),
    "pace_rglru_scan": (C.c_int, [_S, C.POINTER(RglruArgs), C.c_void_p]),
    "pace_rglru_step": (C.c_int, [_S, C.POINTER(RglruArgs), C.c_void_p]),
    "pace_lightning_workspace_bytes": (C.c_uint64, [C.c_int32] * 5),
    "pace_lightning_prefill": (C.c_int, [_S, C.POINTER(LightningArgs), C.c_void_p]),
    "pace_lightning_step": (C.c_int, [_S, C.POINTER(LightningArgs), C.c_void_p]),
    "pace_step_decode": (C.c_int, [C.c_void_p] * 5 + [C.c_int32, C.c_void_p]),
    "pace_attention_dense": (C.c_int, [C.c_void_p] * 4 + [C.c_int32, C.c_int32, C.c_void_p] + [C.c_int32] * 6 +
                             [C.c_void_p, C.c_uint64, C.c_void_p]),
}
EXPORTS = tuple(_SIGS)
for _name, (_res, _args) in _SIGS.items():
    _fn = getattr(lib, _name)   # AttributeError here = the library does not export what the header declares
    _fn.restype, _fn.argtypes = _res, _args


class PaceError(RuntimeError):
    pass


def check(rc: int, what: str) -> None:
    if rc == PACE_OK:
        return
    if rc == PACE_ERR_INVALID:
        raise ValueError(f"{what}: invalid argument")
    if rc == PACE_ERR_UNSUPPORTED:
        raise NotImplementedError(f"{what}: shape not supported by the sm_100a kernels")
    raise PaceError(f"{what}: {lib.pace_last_cuda_error().decode()}")


def describe_status(bits: int) -> str:
    return ", ".join(v for k, v in _DEV_NAMES.items() if bits & k) or "ok"
