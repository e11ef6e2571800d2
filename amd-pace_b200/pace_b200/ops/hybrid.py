"""Operators of hybrid decoders over a packed ``Step``: fused residual norms, attention with normalised keys, with windows, with pooled
blocks, over latents, gated linear recurrence, decayed and gated linear attention, state-space recurrence, gated delta rule, mixtures
of experts.  Thin callers of the C ABI (include/pace_b200.h); every constant of a model is an argument.  ``torch.float32`` activations run the same functions in full 32-bit."""
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from pace_b200 import _C
from pace_b200.llm.step import Step
from pace_b200.ops.backends.b200 import even_lengths, workspace

_OPS = torch.ops.pace_b200


@dataclass
class Routed:
    """What a router chose and what the experts made of it: ``slot_*`` [T, top], ``count`` [experts], ``experts`` lists
    the tokens of every expert, ``y`` the experts' results by expert (``moe_experts``)."""
    top: int
    slot_expert: torch.Tensor
    slot_rank: torch.Tensor
    slot_weight: torch.Tensor
    count: torch.Tensor          # experts with weights, without the identity experts behind them
    lists: torch.Tensor
    y: Optional[torch.Tensor] = None
    identity: Optional[torch.Tensor] = None    # the rows identity experts hand on


def residual_norm(step: Step, x: torch.Tensor, y: Optional[torch.Tensor] = None, w_post: Optional[torch.Tensor] = None,
                  embed: Optional[torch.Tensor] = None, w_next: Optional[torch.Tensor] = None, eps: float = 1e-6,
                  restart: bool = False, weight_offset: float = 0.0, dtype: Optional[torch.dtype] = None,
                  embed_scale: float = 1.0, plain: bool = False, routed: Optional[Routed] = None, bias: Optional[torch.Tensor] = None,
                  y_mul: float = 1.0, embed_norm: Optional[torch.Tensor] = None, w_next2: Optional[torch.Tensor] = None):
    """x (fp32, in place) takes ``rms(y) * w_post`` (without w_post ``y_mul * y``) and, with ``embed``, the tokens' embedding rows
    times ``embed_scale`` or normalised (``embed_norm``); returns ``rms(x) * w_next`` in the activations' dtype (None without
    ``w_next``; with ``plain`` x itself, rounded), with ``w_next2`` a pair of two such norms of the same x.  ``bias`` (fp32)
    belongs to y.  ``routed``: the weighted sum of the experts' rows is (with y: is added to) the output, taken up on the way."""
    h = h2 = add = None
    if routed is not None:
        y, add = routed.y, y
    if w_next is not None or plain:
        h = torch.empty(x.shape, dtype=dtype or (y if y is not None else embed).dtype, device=x.device)
    if w_next2 is not None:
        h2 = torch.empty_like(h)
    more = (add, bias, embed_norm, w_next2, h2, y_mul)
    if routed is None:
        _OPS.residual_norm(step.handle, x, y, w_post, embed, w_next, h, eps, restart, weight_offset, embed_scale, 0, None, None, None,
                           None, None, *more)
    else:
        _OPS.residual_norm(step.handle, x, y, w_post, embed, w_next, h, eps, restart, weight_offset, embed_scale, routed.top,
                           routed.slot_expert, routed.slot_rank, routed.slot_weight, routed.count, routed.identity, *more)
    return h if h2 is None else (h, h2)


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


def _pool_row(pool, dtype: torch.dtype) -> int:
    return pool.head_dim * 2 // dtype.itemsize


def _span(window: Optional[int], chunk: Optional[int]):
    if window is not None:
        return _C.SPAN_WINDOW, window
    return (_C.SPAN_CHUNK, chunk) if chunk is not None else (_C.SPAN_ALL, 0)


MOE_WIDE = 32           # tokens per expert from which wide token tiles are worth the copy
PROMPT_TOKENS = (256, 16)    # tokens of all prompt portions, and of the longest, from which pooled attention over tiles is faster
PROMPT_ROWS = 64        # query rows of an entry from which the tcgen05 prompt kernel is worth a launch


def span_attention(step: Step, cache, qkv: torch.Tensor, heads: int, dim: int, vdim: int, scale: float, eps: float,
                   window: Optional[int] = None, chunk: Optional[int] = None, slopes: Optional[torch.Tensor] = None,
                   sinks: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention with queries and keys normalised per head (no weights): append to the pages, then the softmax over a
    sliding window or a chunk (None: all), minus ``slopes[h]`` times the distance, with ``sinks[h]`` in the denominator.
    ``qkv`` [T, ...]: projection rows (q, k, v).  Returns ``[T, heads * vdim]``."""
    pool, T = cache.pool, step.n_tokens
    q = torch.empty(T, heads, _pool_row(pool, qkv.dtype), dtype=qkv.dtype, device=qkv.device)
    out = torch.empty(T, heads, vdim, dtype=qkv.dtype, device=qkv.device)
    _OPS.kv_append_norm(pool.handle, pool.pages, cache.layer, step.handle, qkv, None, None, q, dim, vdim, eps, 1.0, 0.0, 1.0,
                        True)
    _span_over_pages(step, cache, q, out, (slopes, sinks, dim, vdim, scale) + _span(window, chunk))
    return out.view(T, heads * vdim)


def _span_over_pages(step: Step, cache, q: torch.Tensor, out: torch.Tensor, rule: tuple, softcap: float = 0.0) -> None:
    """The span kernels over a step's entries: those of one token, then the others (tcgen05 where it is worth a launch)."""
    pool, Ed, E = cache.pool, step.n_decode, step.n_entries
    tail = (softcap, out.stride(0))
    if (E > Ed and q.dtype == torch.bfloat16 and pool.desc.row_format == _C.ROWS_BF16
            and step.max_count * (q.shape[1] // pool.n_kv_heads) >= PROMPT_ROWS
            and _OPS.attn_span_prefill(pool.handle, pool.pages, cache.layer, step.handle, q, out, *rule, Ed, E, step.max_count,
                                       step.max_keys, None, None, None, None, None, *tail)):
        E = Ed
    for lo, hi, n in ((0, Ed, 1), (Ed, E, step.max_count)):
        if lo < hi:
            _OPS.attn_span(pool.handle, pool.pages, cache.layer, step.handle, q, out, *rule, lo, hi, n, step.max_keys, *tail)


def conv_attention(step: Step, cache, qkv: torch.Tensor, taps: torch.Tensor, ring: torch.Tensor, q_norm: torch.Tensor,
                   k_norm: torch.Tensor, tables, heads: int, dim: int, vdim: int, scale: float, eps: float, softcap: float = 0.0,
                   v_mul: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention behind short convolutions: every channel of q, k and v is convolved over time, queries and keys are
    normalised per head (weights shared by the heads) and rotated by ``tables`` (None: not), then the softmax over capped
    scores.  ``qkv`` [T, >= ...]: projection rows (q, k, v); ``taps`` fp32 [taps, channels]; ``ring`` fp32 [slots, rows,
    channels]: the newest projections of every slot, stored here in a step of one token per entry and by ``conv_store``
    otherwise.  Values are cached times ``v_mul``.  ``out`` [T, heads * vdim] may have a row stride of its own."""
    pool, T = cache.pool, step.n_tokens
    q = torch.empty(T, heads, _pool_row(pool, qkv.dtype), dtype=qkv.dtype, device=qkv.device)
    if out is None:
        out = torch.empty(T, heads * vdim, dtype=qkv.dtype, device=qkv.device)
    _OPS.kv_append_conv(pool.handle, pool.pages, cache.layer, step.handle, qkv, taps, ring, q_norm, k_norm, *(tables or (None, None)),
                        q, dim, vdim, eps, v_mul, step.decode_only)
    _span_over_pages(step, cache, q, out.unflatten(1, (heads, vdim)), (None, None, dim, vdim, scale, _C.SPAN_ALL, 0), softcap)
    return out


def conv_store(step: Step, x: torch.Tensor, ring: torch.Tensor) -> None:
    """The newest rows of ``x`` [T, >= channels] of every entry into its ring, behind the launches that read the older ones."""
    _OPS.conv_store(step.handle, x, ring)


def latent_attention(step: Step, cache, down: torch.Tensor, q_norm: Optional[torch.Tensor], kv_norm: torch.Tensor,
                     q_up: Optional[torch.Tensor], kv_up: torch.Tensor, heads: int, dim: int, rot_dim: int, vdim: int, scale: float,
                     eps: float, tables, window: Optional[int] = None, sinks: Optional[torch.Tensor] = None,
                     q: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Latent attention.  ``down`` [T, q_rank + rank + rot_dim]: the down projections (query latent, key/value latent,
    rotated key part); the latents are normalised, the key part is rotated, and the row goes to its page.  ``q_up``
    [heads * (dim + rot_dim), q_rank] makes the queries, ``kv_up`` [heads * (dim + vdim), rank] the keys (first) and values
    of all heads.  ``tables``: cosines and sines of every position, [rows, pairs] (None: nothing turns).  Without a query latent
    (``q_norm`` and ``q_up`` None) ``q`` [T, heads * (dim + rot_dim)] holds the queries.  Two forms:

    absorbed  queries go through the key half of ``kv_up``, the heads read the cached rows themselves as one KV head, the
              weighted latents go through the value half (decoding, short portions, fp32);
    expanded  keys and values of the visible latents are made once per step (prompts, where that is less work)."""
    pool, T, R = cache.pool, step.n_tokens, kv_norm.numel()
    row, dt, dev = _pool_row(pool, down.dtype), down.dtype, down.device
    cq = torch.empty(T, q_norm.numel(), dtype=dt, device=dev) if q_norm is not None else None
    _OPS.latent_append(pool.handle, pool.pages, cache.layer, step.handle, down, q_norm, kv_norm, *(tables or (None, None)), cq, rot_dim,
                       eps)
    q = (F.linear(cq, q_up) if q is None else q).unflatten(1, (heads, dim + rot_dim))
    out = torch.empty(T, heads, vdim, dtype=dt, device=dev)
    Ed, E = step.n_decode, step.n_entries
    rule = (scale,) + _span(window, None)
    uk, uv = kv_up[: heads * dim].view(heads, dim, R), kv_up[heads * dim:].view(heads, vdim, R)
    if E > Ed and expand_pays(step, dt, heads, dim, rot_dim, vdim, R, window) and scale > 0:
        keys = step.key_rows(window, Ed)
        lat = torch.empty(keys.total, row, dtype=dt, device=dev)
        _OPS.latent_gather(pool.handle, pool.pages, cache.layer, keys.slot, keys.pos, lat)
        kv = F.linear(lat[:, :R], kv_up)
        k, v = kv[:, : heads * dim].view(-1, heads, dim), kv[:, heads * dim:].view(-1, heads, vdim)
        q = q.contiguous()
        if tables is not None:
            _OPS.rotate_heads(step.handle, q[:, :, dim:], q[:, :, dim:], *tables, Ed, T, rot_dim)
        if not _OPS.attn_span_prefill(pool.handle, pool.pages, cache.layer, step.handle, q, out, None, sinks, dim + rot_dim, vdim,
                                      *rule, Ed, E, step.max_count, step.max_keys, k, lat[:, R: R + rot_dim] if rot_dim else None, v,
                                      keys.cu, keys.first_pos):
            raise RuntimeError("prompt attention refused sizes that expand_pays() lets through")
        E = Ed
    n = T if E > Ed else Ed            # tokens of the absorbed form: all, or those of decoding entries
    if n:
        qa = torch.empty(n, heads, row, dtype=dt, device=dev)
        torch.bmm(q[:n, :, :dim].transpose(0, 1), uk, out=qa[:, :, :R].transpose(0, 1))
        if tables is not None:
            _OPS.rotate_heads(step.handle, q[:, :, dim:], qa[:, :, R:], *tables, 0, n, row - R)
        elif row > R:
            qa[:, :, R: R + rot_dim] = q[:n, :, dim:]
            qa[:, :, R + rot_dim:].zero_()
        mixed = torch.empty(n, heads, R, dtype=dt, device=dev)
        for lo, hi, m in ((0, Ed, 1), (Ed, E, step.max_count)):
            if lo < hi:
                _OPS.attn_span(pool.handle, pool.pages, cache.layer, step.handle, qa, mixed, None, sinks, R + rot_dim, R, *rule,
                               lo, hi, m, step.max_keys)
        torch.bmm(mixed.transpose(0, 1), uv.transpose(1, 2), out=out[:n].transpose(0, 1))
    return out.view(T, heads * vdim)


def pooled_attention(step: Step, cache, blocks, qkv: torch.Tensor, tables, heads: int, dim: int, vdim: int, scale: float, window: int,
                     block: int, sinks: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None,
                     gate: Optional[torch.Tensor] = None, halves: bool = True) -> torch.Tensor:
    """Attention over the last ``window`` tokens and the means of whole blocks of ``block`` tokens in front of them: the first elements
    of queries and keys are rotated by ``tables`` (None: not; ``halves``: element i with element i + pairs, else neighbours), keys and
    values go to their pages, completed blocks to those of ``blocks``; then one softmax over tokens and blocks (``sinks``: scores
    without values), the weights mixed over the heads by ``mix`` [heads, heads], outputs times sigmoid(``gate``).  ``qkv``
    [T, >= ...]: projection rows (q, k, v).  Returns ``[T, heads * vdim]``."""
    pool, bp, T = cache.pool, blocks.pool, step.n_tokens
    q = torch.empty(T, heads, _pool_row(pool, qkv.dtype), dtype=qkv.dtype, device=qkv.device)
    out = torch.empty(T, heads * vdim, dtype=qkv.dtype, device=qkv.device)
    where = (pool.handle, pool.pages, cache.layer, bp.handle, bp.pages, blocks.layer, step.handle)
    _OPS.kv_append_rotate(*where, qkv, *(tables or (None, None)), q, dim, vdim, halves, block, step.decode_only)
    rule = (q, out, gate, sinks, mix, dim, vdim, scale, window, block)
    Ed, E = step.n_decode, step.n_entries
    if (E > Ed and q.dtype == torch.bfloat16 and T - Ed >= PROMPT_TOKENS[0] and step.max_count >= PROMPT_TOKENS[1]
            and _OPS.attn_pooled_prompt(*where, *rule, Ed, E, step.max_count, step.max_keys)):
        T = Ed
    if T:
        _OPS.attn_pooled(*where, *rule, 0, T, step.max_keys)
    return out


def expand_pays(step: Step, dtype: torch.dtype, heads: int, dim: int, rot_dim: int, vdim: int, rank: int,
                window: Optional[int]) -> bool:
    """Whether a step's prompt portions are less work with expanded keys and values, in sizes the prompt kernel takes."""
    up = lambda n: (n + 63) // 64      # noqa: E731
    if dtype != torch.bfloat16 or any(n % 8 for n in (dim, rot_dim, vdim, rank)) or vdim > 128 or up(dim) + up(rot_dim) > 4:
        return False
    expanded = absorbed = 0.0
    for s, c in zip(step.starts[step.n_decode:], step.counts[step.n_decode:]):
        seen = min(s + c, window + c - 1 if window else s + c)
        pairs = c * min(s + c / 2.0, float(window or s + c))
        expanded += seen * rank * (dim + vdim) + pairs * (dim + rot_dim + vdim)
        absorbed += c * rank * (dim + vdim) + pairs * (2 * rank + rot_dim)
    return step.max_count >= 32 and expanded < absorbed


def glu(x: torch.Tensor, act: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """act(gate) * up of rows ``[T, 2 n]`` (gate first); ``out`` may have a row stride of its own."""
    if out is None:
        out = torch.empty(x.shape[0], x.shape[1] // 2, dtype=x.dtype, device=x.device)
    _OPS.glu(x, out, act)
    return out


def activate(x: torch.Tensor, act: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """act(x) of rows ``[T, n]``; ``out`` may have a row stride of its own."""
    out = torch.empty_like(x) if out is None else out
    _OPS.glu(x, out, act, False)
    return out


def moe_route(h: torch.Tensor, router: torch.Tensor, correction: Optional[torch.Tensor], top: int, softmax: bool = False,
              weight_scale: Optional[float] = None, identity: int = 0) -> Routed:
    """Sigmoid (or softmax) scores of every router output in fp32, the ``top`` largest by score + ``correction``, weighted by
    their scores (``weight_scale``: made to sum to that).  The last ``identity`` outputs are experts that hand on ``h`` itself."""
    logits = linear_f32(h, router)
    T, E = logits.shape
    ints = torch.empty(2 * T * top + E + E * T, dtype=torch.int32, device=h.device)
    a, b = T * top, 2 * T * top
    r = Routed(top, ints[:a].view(T, top), ints[a:b].view(T, top), torch.empty(T, top, dtype=torch.float32, device=h.device),
               ints[b: b + E - identity], ints[b + E:].view(E, T), identity=h if identity else None)
    _OPS.moe_route(logits, correction, r.slot_expert, r.slot_rank, r.slot_weight, ints[b: b + E], r.lists, softmax, weight_scale)
    return r


def moe_experts(h: torch.Tensor, routed: Routed, gate_up: torch.Tensor, down: torch.Tensor, act: int,
                status: Optional[torch.Tensor] = None, gated: bool = True) -> Routed:
    """The chosen experts' feed-forwards (gated: ``gate_up`` holds gate and up rows), left by expert in ``routed.y``
    (``residual_norm`` sums them up)."""
    n = h.shape[0] * routed.top
    hidden = torch.empty(n, down.shape[2], dtype=h.dtype, device=h.device)
    routed.y = torch.empty(n, down.shape[1], dtype=h.dtype, device=h.device)
    # many tokens per expert: wide tiles, over rows that are copied into expert order first
    scratch = torch.empty(n, h.shape[1], dtype=h.dtype, device=h.device) if n > MOE_WIDE * down.shape[0] else None
    _OPS.moe_experts(h, gate_up, down, hidden, routed.y, scratch, routed.count, routed.lists, routed.slot_expert, routed.slot_rank,
                     status, act, gated)
    return routed


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


def part_norm_gate(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, part: int, eps: float, gate_first: bool = False,
                   out: Optional[torch.Tensor] = None, silu: bool = False) -> torch.Tensor:
    """rms over every ``part`` elements of a row: ``rms(o) * weight * sigmoid(gate)`` (``silu``: times silu(gate)), or with the gate in
    front ``rms(o * silu(gate)) * weight``; the weight repeats along the row.  ``out`` may have a row stride of its own."""
    out = torch.empty_like(o) if out is None else out
    mode = _C.GATE_SILU_FIRST if gate_first else _C.GATE_SILU if silu else _C.GATE_SIGMOID
    _OPS.part_norm_gate(o, gate, weight, out, part, mode, eps)
    return out


def soft_cap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """cap * tanh(x / cap) in place (fp32)."""
    if x.numel():
        _OPS.soft_cap(x, cap)
    return x


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


def ssd(step: Step, xbc: torch.Tensor, dt_raw: torch.Tensor, taps: torch.Tensor, conv_bias: Optional[torch.Tensor],
        dt_bias: torch.Tensor, neg_a: torch.Tensor, d_skip: torch.Tensor, groups: int, state: torch.Tensor,
        ring: torch.Tensor) -> torch.Tensor:
    """State-space recurrence behind a short convolution with silu.  ``xbc`` [T, >= channels]: projections x (heads x vdim),
    b and c (groups x state each); ``dt_raw`` [T, heads]; ``state`` fp32 [slots, heads, state, vdim]; ``ring`` as in
    ``conv_attention``.  Returns [T, heads * vdim].  One token per entry: one launch, which also stores the ring."""
    T, inner = step.n_tokens, state.shape[1] * state.shape[3]
    out = torch.empty(T, inner, dtype=xbc.dtype, device=xbc.device)
    if step.decode_only:
        _OPS.ssd_step(step.handle, xbc, dt_raw, dt_bias, neg_a, d_skip, state, out, groups, taps, conv_bias, ring)
        return out
    u = torch.empty(T, (taps.shape[1] + 7) // 8 * 8, dtype=xbc.dtype, device=xbc.device)
    _OPS.causal_conv(step.handle, xbc, taps, conv_bias, ring, u, True)
    _OPS.ssd_prefill(step.handle, u, dt_raw, dt_bias, neg_a, d_skip, state, out, groups)
    return out


def delta_rule(step: Step, qkv: torch.Tensor, a_raw: torch.Tensor, b_raw: torch.Tensor, taps: torch.Tensor, dt_bias: torch.Tensor,
               neg_a: torch.Tensor, kv_heads: int, state: torch.Tensor, ring: torch.Tensor, unit_eps: float,
               q_scale: float) -> torch.Tensor:
    """Gated delta rule with a decay per key channel behind a short convolution with silu.  ``qkv`` [T, >= channels]: projections
    q, k (kv_heads x dim each) and v (heads x vdim); ``a_raw`` [T, heads * dim], ``b_raw`` [T, heads]; ``state`` fp32 [slots,
    heads, dim, vdim]; ``ring`` as in ``conv_attention``.  Returns [T, heads * vdim].  One token per entry: one launch, which
    also stores the ring."""
    T = step.n_tokens
    out = torch.empty(T, state.shape[1] * state.shape[3], dtype=qkv.dtype, device=qkv.device)
    if step.decode_only:
        _OPS.delta_step(step.handle, qkv, a_raw, b_raw, dt_bias, neg_a, state, out, kv_heads, unit_eps, q_scale, taps, ring)
        return out
    u = torch.empty(T, (taps.shape[1] + 7) // 8 * 8, dtype=qkv.dtype, device=qkv.device)
    _OPS.causal_conv(step.handle, qkv, taps, None, ring, u, True)
    _OPS.delta_prefill(step.handle, u, a_raw, b_raw, dt_bias, neg_a, state, out, kv_heads, unit_eps, q_scale)
    return out


def gla(step: Step, qkv: torch.Tensor, z: torch.Tensor, z_bias: torch.Tensor, state: torch.Tensor, norm: torch.Tensor,
        gate: torch.Tensor, tau: float, q_scale: float, eps: float) -> torch.Tensor:
    """Gated linear attention, decay per head and key channel sigmoid(z + z_bias)^(1 / tau); outputs normalised per head (``norm``
    [vdim]) and times silu(gate).  ``qkv`` [T, >= ...]: projections q, k (heads x dim each) and v (heads x vdim); ``z`` [T, heads * dim],
    ``gate`` [T, heads * vdim]; ``state`` fp32 [slots, heads, dim, vdim].  Returns [T, heads * vdim].  One token per entry: one
    launch."""
    T, heads, vdim = step.n_tokens, state.shape[1], state.shape[3]
    out = torch.empty(T, heads * vdim, dtype=qkv.dtype, device=qkv.device)
    if step.decode_only:
        _OPS.gla_step(step.handle, qkv, z, z_bias, state, out, 1.0 / tau, q_scale, norm, gate, eps)
        return out
    _OPS.gla_prefill(step.handle, qkv, z, z_bias, state, out, 1.0 / tau, q_scale)
    return part_norm_gate(out, norm, gate, vdim, eps, out=out, silu=True)


def embed_pairs(step: Step, embed: torch.Tensor, scale: float, pairs: Optional[torch.Tensor] = None,
                last_token: Optional[torch.Tensor] = None, mul_prev: int = 0, mul_cur: int = 0) -> torch.Tensor:
    """fp32 rows ``embed[token] * scale``, plus the row of ``pairs`` that (previous token, token) hash to.  ``last_token`` int32
    [slots]: every slot's newest token, stored here in a step of one token per entry and by ``state_commit`` otherwise."""
    x = torch.empty(step.n_tokens, embed.shape[1], dtype=torch.float32, device=embed.device)
    _OPS.embed_pairs(step.handle, x, embed, scale, pairs, last_token, mul_prev, mul_cur, step.decode_only and last_token is not None)
    return x


def shift_norm(step: Step, x: torch.Tensor, w_next: torch.Tensor, shift: torch.Tensor, state: torch.Tensor, state_out: torch.Tensor,
               eps: float, dtype: torch.dtype, y: Optional[torch.Tensor] = None, y_bias: Optional[torch.Tensor] = None,
               w_post: Optional[torch.Tensor] = None, add: Optional[torch.Tensor] = None, spare: Optional[torch.Tensor] = None):
    """(new stream, mixer input): the fp32 stream x takes ``rms(y + y_bias) * w_post`` and the vector ``add``; its norm ``n = rms(x) *
    w_next`` moves to ``n + (n' - n) * shift`` with n' the previous token's.  ``state`` [slots, width]: every slot's newest n; those
    of this step go to ``state_out`` (one token per entry: may be the same).  The new stream lies in ``spare`` (None: a new buffer;
    with one token per entry in x itself)."""
    x_out = x if step.decode_only else torch.empty_like(x) if spare is None else spare
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    _OPS.shift_norm(step.handle, x, x_out, y, y_bias, w_post, add, w_next, shift, state, state_out, h, eps)
    return x_out, h


def state_commit(step: Step, source: torch.Tensor, target: torch.Tensor, last_token: Optional[torch.Tensor] = None) -> None:
    """``target`` [slots, ...] takes the rows of the step's slots from ``source``, ``last_token`` the entries' last tokens."""
    _OPS.state_commit(step.handle, source, target, last_token)


def gate_per_head_(x: torch.Tensor, gate: torch.Tensor, heads: int) -> torch.Tensor:
    """Heads of rows ``[T, heads * vdim]`` times sigmoid(``gate`` [T, heads]), in place."""
    _OPS.gate_per_head(x.view(x.shape[0], heads, -1), gate)
    return x


def linear_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """x W^T with an fp32 result (logits)."""
    if x.dtype == torch.float32:
        return F.linear(x, weight)
    return torch.mm(x, weight.t(), out_dtype=torch.float32)
