"""Operators of hybrid decoders over a packed ``Step``: fused residual norms, attention with normalised keys,
gated linear recurrence, decayed linear attention.  Thin callers of the C ABI (include/pace_b200.h); every
constant of a model is an argument.  ``torch.float32`` activations run the same functions in full 32-bit."""
from typing import Optional

import torch
import torch.nn.functional as F

from pace_b200 import _C
from pace_b200.llm.step import Step
from pace_b200.ops.backends.b200 import even_lengths, workspace

_OPS = torch.ops.pace_b200


def residual_norm(step: Step, x: torch.Tensor, y: Optional[torch.Tensor] = None, w_post: Optional[torch.Tensor] = None,
                  embed: Optional[torch.Tensor] = None, w_next: Optional[torch.Tensor] = None, eps: float = 1e-6,
                  restart: bool = False, weight_offset: float = 0.0, dtype: Optional[torch.dtype] = None):
    """x (fp32, in place) takes ``rms(y) * w_post`` and, with ``embed``, the tokens' embedding rows; returns
    ``rms(x) * w_next`` in the activations' dtype (None without ``w_next``)."""
    h = None
    if w_next is not None:
        h = torch.empty(x.shape, dtype=dtype or (y if y is not None else embed).dtype, device=x.device)
    _OPS.residual_norm(step.handle, x, y, w_post, embed, w_next, h, eps, restart, weight_offset)
    return h


def step_attention(step: Step, cache, qkv: torch.Tensor, heads: int, dim: int, vdim: int, scale: float,
                   q_norm: Optional[torch.Tensor] = None, k_norm: Optional[torch.Tensor] = None, eps: float = 1e-6,
                   temp_coef: float = 0.0, temp_every: float = 1.0) -> torch.Tensor:
    """Norms, query temperature, append to the pages and causal attention.  ``qkv`` [T, >= ...]: projection rows
    (q, k, v); ``cache`` one layer of a paged pool whose lengths already count the step's tokens.  Returns the
    heads' outputs in the step's staging rows, ``[rows, heads, row elements]`` (columns beyond ``vdim`` zero).

    bf16 rows of 64 or 128: entries of one token go to the decode kernel, the others to the verify / prefill
    kernels (two launches at most); other row formats: the general kernel."""
    pool = cache.pool
    fast = pool.desc.row_format == _C.ROWS_BF16
    row = pool.head_dim * 2 // qkv.element_size()
    q = torch.empty(step.staging_rows, heads, row, dtype=qkv.dtype, device=qkv.device)
    out = torch.empty_like(q)
    q_mul = 1.0
    if fast and not scale > 0:              # the tensor-core kernels take positive scales only
        q_mul, scale = scale, 1.0
    _OPS.kv_append_norm(pool.handle, pool.pages, cache.layer, step.handle, qkv, q_norm, k_norm, q, dim, vdim, eps, q_mul,
                        temp_coef, temp_every)
    if not fast:
        _OPS.attn_general(pool.handle, pool.pages, cache.layer, step.handle, q, out, dim, vdim, scale)
        return out
    Ed, E, n = step.n_decode, step.n_entries, step.max_count
    for lo, hi, S, qs, os in ((0, Ed, 1, q[:Ed].unsqueeze(2), out[:Ed].unsqueeze(2)),
                              (Ed, E, n, q[Ed:].view(-1, n, heads, row).transpose(1, 2),
                               out[Ed:].view(-1, n, heads, row).transpose(1, 2))):
        if lo == hi:
            continue
        ws = workspace(q.device, _C.lib.pace_attn_workspace_bytes(hi - lo, heads, pool.n_kv_heads, row, S))
        flags, q_lens = _C.ATTN_SPLIT_WEIGHTS, None      # weights stay in 32-bit up to the product with V
        if S == 1:
            lens = [step.starts[i] + 1 for i in range(lo, hi)] if not cache.manager.static_launch else cache._lens
            if even_lengths(lens, pool.n_kv_heads, row, pool.page_tokens, q.device):
                flags |= _C.ATTN_WHOLE_UNITS
        elif any(c != n for c in step.counts[lo:hi]):
            q_lens = step.count[lo:hi]
        op = _OPS.attn_decode if S == 1 else _OPS.attn_verify if S <= 64 else _OPS.attn_prefill
        op(pool.handle, pool.pages, cache.layer, qs, os, step.slot[lo:hi], None, q_lens, ws, scale, flags, None, None, 0)
    return out


def gate_heads(step: Step, attn: torch.Tensor, gate: torch.Tensor, vdim: int) -> torch.Tensor:
    """Concatenated heads times sigmoid(gate), back in token order: ``[T, heads * vdim]``."""
    out = torch.empty(step.n_tokens, attn.shape[1] * vdim, dtype=attn.dtype, device=attn.device)
    _OPS.gate_heads(step.handle, attn, gate, out, vdim)
    return out


def norm_gate(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float) -> torch.Tensor:
    """rms(o) * weight * sigmoid(gate) over whole rows."""
    out = torch.empty_like(o)
    _OPS.norm_gate(o, weight, gate, out, eps)
    return out


def relu_squared_(x: torch.Tensor) -> torch.Tensor:
    _OPS.relu_squared(x)
    return x


def rglru(step: Step, yx: torch.Tensor, gate_w: torch.Tensor, taps: torch.Tensor, conv_bias: torch.Tensor,
          ra_bias: torch.Tensor, ri_bias: torch.Tensor, decay_base: torch.Tensor, state: torch.Tensor,
          conv_state: torch.Tensor) -> torch.Tensor:
    """Real-gated linear recurrence behind a short causal convolution, times its gelu branch.  ``yx`` [T, 2 width]
    holds both branches' projections (y first), ``gate_w`` [blocks, 2, n, n] the block-diagonal gates (r, i; rows
    are outputs).  One token per entry: one launch.  Otherwise convolution, gate products (fp32 results) and scan."""
    T, W = yx.shape[0], yx.shape[1] // 2
    blocks, n = gate_w.shape[0], gate_w.shape[2]
    out = torch.empty(T, W, dtype=yx.dtype, device=yx.device)
    if step.decode_only and 96 * (n + 32) * yx.element_size() <= 200 * 1024:      # what the launch keeps in shared memory
        _OPS.rglru_step(step.handle, yx, gate_w, taps, conv_bias, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks)
        return out
    u = torch.empty(T, W, dtype=yx.dtype, device=yx.device)
    _OPS.causal_conv(step.handle, yx[:, W:], taps, conv_bias, conv_state, u)
    ub, wb = u.view(T, blocks, n).transpose(0, 1), gate_w.view(blocks, 2 * n, n).transpose(1, 2)
    gates = torch.bmm(ub, wb) if yx.dtype == torch.float32 else torch.bmm(ub, wb, out_dtype=torch.float32)
    _OPS.rglru_scan(step.handle, yx, u, gates, ra_bias, ri_bias, decay_base, state, conv_state, out, blocks)
    return out


def lightning(step: Step, qkv: torch.Tensor, decay: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """Linear attention with a fixed decay per head; ``qkv`` rows are the projections before their silu, ``state``
    fp32 ``[slots, heads, dim, vdim]``.  Returns ``[T, heads * vdim]``."""
    out = torch.empty(step.n_tokens, state.shape[1] * state.shape[3], dtype=qkv.dtype, device=qkv.device)
    op = _OPS.lightning_step if step.decode_only else _OPS.lightning_prefill
    op(step.handle, qkv, decay, state, out)
    return out


def linear_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """x W^T with an fp32 result (logits)."""
    if x.dtype == torch.float32:
        return F.linear(x, weight)
    return torch.mm(x, weight.t(), out_dtype=torch.float32)
