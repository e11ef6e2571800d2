"""The Garupel model on the GPU against the plain implementation: every mechanism alone, then whole models,
prompts, portions, decoding, batches, reuse of pages and slots, and generation through the framework's loops."""
import json
import math
import os
import subprocess

import pytest
import torch

import garupel_models as gm
from oracle import garupel_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF16, FP32 = torch.bfloat16, torch.float32
TOL = {BF16: 0.06, FP32: 1e-4}
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))


def build(cfg, dtype, seed=0):
    from pace_b200.llm.registry import build_model
    w = gm.weights(cfg, seed)
    model = build_model(cfg, dtype, DEV)
    model.load_weights(w)
    return model, w


def batcher(model, slots=4, pool_tokens=64 * 20, max_len=64 * 12, **kw):
    from pace_b200.llm.serving import ContinuousBatcher
    return ContinuousBatcher(model, pool_tokens=pool_tokens, max_batch=slots, max_seq_len=max_len, **kw)


def prompt(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed))


def feed(b, slot, tokens, sizes):
    """All logits of a sequence fed in portions of the given sizes (the last one repeated)."""
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        out.append(b.step({slot: tokens[at: at + n]}, {slot: range(n)}).float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


# ---- mechanisms alone ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("kind,mixer,ff", [
    ("attention", gm.att(6, 2, 20, 28, every=3), None), ("attention", gm.att(5, 5, 130, 33), None),
    ("attention", gm.att(34, 1, 8, 16, scale=0.7, coef=-0.2), None), ("rglru", gm.lru(39, 3, 4), None),
    ("rglru", gm.lru(96, 2, 2), None), ("lightning", gm.lin(3, 12, 20, [0.1, 0.8, 0.999]), None),
    ("lightning", gm.lin(2, 64, 128, [0.99, 1.0]), None), ("lightning", gm.lin(1, 300, 70, [0.9]), None),
    ("rglru", gm.lru(16, 16, 1), 21)])
def test_one_layer_models(kind, mixer, ff, dtype):
    cfg = gm.config([gm.layer(kind, mixer, ff)], 44)
    model, w = build(cfg, dtype, 5)
    toks = prompt(cfg, 90, 1)
    want = ref.Sequence(cfg, w).run(toks)
    b = batcher(model)
    for sizes in ([90], [2, 3, 64, 5], [70, 1]):
        slot = b.open()
        assert gm.error(feed(b, slot, toks, sizes), want) < TOL[dtype], sizes
        b.close(slot)
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width", [64, 44, 37, 2200])
def test_residual_norm(width, dtype):
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(width)
    T, eps = 5, 1e-3
    toks = torch.tensor([3, 0, 8, 8, 1])
    step = Step([5], [0], [0], toks, 9, DEV)
    x, y, e = (torch.randn(n, width, generator=g) for n in (T, T, 9))
    y, e = y.to(dtype), e.to(dtype)
    wp, wn = torch.randn(width, generator=g), torch.randn(width, generator=g)
    xd = x.to(DEV)
    for offset in (0.0, 1.0):
        got = hybrid.residual_norm(step, xd.copy_(x), y.to(DEV), wp.to(DEV), e.to(DEV), wn.to(DEV), eps, weight_offset=offset)
        want_x = x.double() + ref.rms_norm(y.double(), wp.double() + offset, eps) + e.double()[toks]
        torch.testing.assert_close(xd.double().cpu(), want_x, rtol=2e-6, atol=2e-6)
        want_h = ref.rms_norm(want_x, wn.double() + offset, eps)
        torch.testing.assert_close(got.double().cpu(), want_h, rtol=(1e-2 if dtype == BF16 else 5e-6), atol=1e-5)
    hybrid.residual_norm(step, xd, embed=e.to(DEV), restart=True)
    assert torch.equal(xd.cpu(), e.float()[toks])
    hybrid.residual_norm(step, xd, y.to(DEV))           # no norm behind, none in front
    assert torch.equal(xd.cpu(), e.float()[toks] + y.float())


def _attention_case(dtype, heads, kv, dim, vdim, n, seed=0):
    """Random projections of n tokens and the cache of one attention layer for two rows."""
    from pace_b200.llm.hybrid_cache import HybridCacheManager, KVSpec
    g = torch.Generator().manual_seed(seed)
    qkv = torch.randn(n, heads * dim + kv * (dim + vdim), generator=g).to(dtype)
    cache = HybridCacheManager([KVSpec(kv, dim, vdim)], 2, 64 * 16, 64 * 8, dtype, DEV)
    return qkv, cache


def _attend(qkv, cache, row, counts, heads, dim, vdim, scale, **kw):
    from pace_b200.ops import hybrid
    out, at = [], 0
    for n in counts:
        c = [0, 0]
        c[row] = n
        step = cache.step(c, torch.zeros(n, dtype=torch.long), 1)
        cache.begin_step(step)
        o = hybrid.step_attention(step, cache[0], qkv[at: at + n].to(DEV), heads, dim, vdim, scale, **kw)
        out.append(o[step.q_row.long(), :, :vdim].double().cpu())
        at += n
    cache.pool.check_status()
    return torch.cat(out)


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim", [(BF16, 10, 2, 88, 104), (BF16, 8, 4, 33, 64), (BF16, 2, 2, 144, 40),
                                                     (FP32, 6, 2, 40, 24), (FP32, 3, 3, 128, 128)])
def test_one_key_far_away_at_every_page_border(dtype, heads, kv, dim, vdim):
    """One key stands out for one query; whatever the place of either (first token, last of a page, first of the
    next, the query itself) and however the tokens came, the output is that key's value, and one place later in
    the future it is not."""
    n, scale = 140, 1.0
    for j, t in ((0, 139), (0, 64), (63, 64), (64, 65), (63, 139), (64, 128), (127, 128), (127, 127), (128, 127), (100, 99)):
        qkv, cache = _attention_case(dtype, heads, kv, dim, vdim, n, seed=j)
        qkv = qkv.float() * 0.05
        u = torch.zeros(dim)
        u[j % dim] = 8.0
        qkv[t, : heads * dim] += u.repeat(heads)
        qkv[j, heads * dim: (heads + kv) * dim] += u.repeat(kv)
        qkv[:, (heads + kv) * dim:] *= 20.0
        qkv = qkv.to(dtype)
        v = qkv[j, (heads + kv) * dim:].double().view(kv, vdim).repeat_interleave(heads // kv, 0)
        for row, counts in ((0, [n]), (1, [t, 1] + [1] * (n - t - 1)), (0, [50, 2, 40, n - 92])):
            got = _attend(qkv, cache, row, counts, heads, dim, vdim, scale)[t]
            gap = float((got - v).abs().max())
            assert (gap < 0.02) if j <= t else (gap > 0.3), (j, t, counts, gap)
            cache.recycle([row])


@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 1, 128, 128), (12, 1, 64, 64), (20, 1, 96, 80), (2, 1, 64, 64)])
def test_softmax_weights_are_not_rounded_to_bf16(heads, kv, dim, vdim):
    """Every key but the first has a weight half way between two bf16 values: rounded, all of them would be off in
    the same direction by 2^-8 of themselves, and half of the outputs would land on another bf16 value than the exact
    result does."""
    p = 0.5 + 2.0 ** -9 * 0.98
    n = 500
    for counts in ([n], [n - 1, 1], [n - 2, 2], [n - 3, 3], [n - 40, 40]):
        qkv, cache = _attention_case(BF16, heads, kv, dim, vdim, n, 11)
        v = (1.0 + torch.rand(n, kv * vdim, generator=torch.Generator().manual_seed(1))).to(BF16)
        qkv[:, : (heads + kv) * dim] = 0
        qkv[:, : heads * dim: dim] = 1
        qkv[0, heads * dim: (heads + kv) * dim: dim] = 1
        qkv[:, (heads + kv) * dim:] = v
        got = _attend(qkv, cache, 0, counts, heads, dim, vdim, -math.log(p))[n - counts[-1]:]
        w = torch.cat([torch.ones(1, dtype=torch.float64), torch.full((n - 1,), p, dtype=torch.float64)])
        same = []
        for i in range(0, counts[-1], 97):
            t = n - counts[-1] + i
            if t >= 300:
                want = (w[: t + 1] @ v[: t + 1].double()) / w[: t + 1].sum()
                same.append((got[i] == want.view(kv, vdim).to(BF16).double()).double().mean())
        assert float(min(same)) > 0.9, (counts, same)


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_norms_and_temperature_of_queries_and_keys(dtype):
    heads, kv, dim, vdim, n, eps = 4, 2, 24, 40, 70, 0.05
    qkv, cache = _attention_case(dtype, heads, kv, dim, vdim, n, 3)
    g = torch.Generator().manual_seed(4)
    qn, kn = torch.rand(heads * dim, generator=g) * 2, torch.rand(kv * dim, generator=g) * 2
    x = qkv.double()
    q = ref.rms_norm(x[:, : heads * dim], qn.double(), eps).view(n, heads, dim)
    k = ref.rms_norm(x[:, heads * dim: (heads + kv) * dim], kn.double(), eps).view(n, kv, dim)
    v = x[:, (heads + kv) * dim:].view(n, kv, vdim)
    temp = torch.tensor([ref.query_temperature(t, 0.8, 7) for t in range(n)], dtype=torch.float64)
    q, k = (q * temp[:, None, None]).to(dtype).double(), k.to(dtype).double()      # as the products take them

    def read(t, h, scale):
        return ref.softmax_read(q[t, h], k[: t + 1, h // 2], v[: t + 1, h // 2], scale)
    want = torch.stack([torch.stack([read(t, h, 0.4) for h in range(heads)]) for t in range(n)])
    kw = dict(q_norm=qn.to(DEV), k_norm=kn.to(DEV), eps=eps, temp_coef=0.8, temp_every=7.0)
    got = _attend(qkv, cache, 1, [33, 1, 36], heads, dim, vdim, 0.4, **kw)
    tol = 0.03 if dtype == BF16 else 2e-5
    assert float((got - want).abs().max()) < tol
    if dtype == BF16:      # a scale the tensor-core kernels do not take by themselves
        cache.recycle([1])
        neg = _attend(qkv, cache, 1, [n], heads, dim, vdim, -0.5, **kw)      # (a power of two: the same rounding of q)
        w = torch.stack([read(69, h, -0.5) for h in range(heads)])
        assert float((neg[69] - w).abs().max()) < tol


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("heads,dim,vdim", [(3, 20, 36), (2, 128, 128), (1, 64, 256), (2, 96, 80), (1, 7, 5)])
def test_decayed_linear_attention_remembers_exactly(dtype, heads, dim, vdim):
    """One token is large among silent ones: what later queries read of it is decay^distance, across portions,
    chunk edges and single tokens.  Distances run over several chunk lengths."""
    from pace_b200.llm.hybrid_cache import HybridCacheManager, StateSpec
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(dim)
    n, decay = 300, [0.9995, 0.97, 0.5][:heads]
    x = torch.randn(n, heads * (2 * dim + vdim), generator=g)
    for t in (0, 63, 64, 127, 128, 200):
        x[t] *= 4.0
    x = x.to(dtype)
    silu = lambda z: torch.nn.functional.silu(z.double()).to(dtype).double()     # noqa: E731
    q, k, v = (silu(x[:, a: b]).view(n, heads, -1) for a, b in ((0, heads * dim), (heads * dim, 2 * heads * dim),
                                                                (2 * heads * dim, x.shape[1])))
    S, want = torch.zeros(heads, dim, vdim, dtype=torch.float64), []
    dec = torch.tensor(decay, dtype=torch.float32).double()
    for t in range(n):
        S, o = ref.lightning_step(S, q[t], k[t], v[t], dec)
        want.append(o)
    want = torch.stack(want)
    cache = HybridCacheManager([StateSpec((("S", (heads, dim, vdim)),))], 3, 64, 4096, dtype, DEV)
    cache[0]["S"].fill_(float("nan"))                # a used slot: must not be read by a sequence that starts
    for row, counts in ((2, [n]), (1, [2, 61, 1, 1, 65, 128, 42]), (0, [200] + [1] * 100), (1, [64, 64, 172])):
        cache.recycle([row])
        at, got = 0, []
        for c in counts:
            cs = [0, 0, 0]
            cs[row] = c
            step = cache.step(cs, torch.zeros(c, dtype=torch.long), 1)
            cache.begin_step(step)
            got.append(hybrid.lightning(step, x[at: at + c].to(DEV), torch.tensor(decay).to(DEV), cache[0]["S"]).cpu())
            at += c
        got = torch.cat(got).double().view(n, heads, vdim)
        rel = (got - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-3)
        assert float(rel.max()) < (0.012 if dtype == BF16 else 2e-5), counts
        state = cache[0]["S"][row].double().cpu()
        assert float((state - S).abs().max() / S.abs().max()) < 2e-5, counts      # fp32 states with either dtype


@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 128), (64, 32, 40), (3, 128, 136)])
def test_decayed_linear_attention_over_long_prompts(heads, dim, vdim):
    """Prompts long enough to be cut into segments that run side by side, of unequal lengths in one batch, in front
    of them a state from earlier tokens (or none)."""
    from pace_b200.llm.hybrid_cache import HybridCacheManager, StateSpec
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(heads)
    lens = [1500, 70, 900, 1]
    decay = torch.linspace(0.9, 0.9999, heads)
    dec = decay.double()[:, None, None]
    xs = [torch.randn(n, heads * (2 * dim + vdim), generator=g).to(BF16) for n in lens]
    cache = HybridCacheManager([StateSpec((("S", (heads, dim, vdim)),))], 4, 64, 4096, BF16, DEV)
    cache[0]["S"].fill_(float("nan"))
    at = [0] * 4
    outs = [[] for _ in lens]

    def go(counts):
        x = torch.cat([xs[b][at[b]: at[b] + c] for b, c in enumerate(counts)])
        step = cache.step(counts, torch.zeros(sum(counts), dtype=torch.long), 1)
        cache.begin_step(step)
        order = torch.cat([torch.arange(sum(counts[:b]), sum(counts[:b + 1])) for b in step.rows])
        o = hybrid.lightning(step, x[order].to(DEV), decay.to(DEV), cache[0]["S"]).double().cpu()
        for b in step.rows:
            outs[b].append(o[step.first_row[b]: step.first_row[b] + counts[b]])
            at[b] += counts[b]
    go([0, 0, 65, 0])
    go([1, 0, 30, 0])
    go([1499, 70, 805, 1])
    silu = lambda z: torch.nn.functional.silu(z.double()).to(BF16).double()     # noqa: E731
    for b, n in enumerate(lens):
        q, k, v = (silu(xs[b][:, a: z]).view(n, heads, -1) for a, z in ((0, heads * dim), (heads * dim, 2 * heads * dim),
                                                                        (2 * heads * dim, xs[b].shape[1])))
        S, want = torch.zeros(heads, dim, vdim, dtype=torch.float64), []
        for t in range(n):
            S = dec * S + k[t, :, :, None] * v[t, :, None, :]
            want.append(torch.einsum("hdv,hd->hv", S, q[t]))
        want, got = torch.stack(want), torch.cat(outs[b]).view(n, heads, vdim)
        rel = (got - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-3)
        assert float(rel.max()) < 0.012, b
        assert float((cache[0]["S"][b].double().cpu() - S).abs().max() / S.abs().max()) < 2e-5, b


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width,blocks,taps", [(60, 3, 3), (66, 2, 4), (128, 1, 1), (240, 5, 6), (33, 3, 2)])
def test_gated_recurrence(dtype, width, blocks, taps):
    from pace_b200.llm.hybrid_cache import HybridCacheManager, StateSpec
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(width)
    n, m = 270, width // blocks
    yx = torch.randn(n, 2 * width, generator=g).to(dtype)
    yx[::37] *= 5
    gw = (torch.randn(blocks, 2, m, m, generator=g) / math.sqrt(m)).to(dtype)
    tp, cb = torch.randn(width, taps, generator=g) * 0.6, torch.randn(width, generator=g) * 0.2
    ra, ri = torch.randn(width, generator=g), torch.randn(width, generator=g)
    lam = torch.linspace(-12, 1, width).double()     # from hardly any decay per token to almost all
    S, past, want = torch.zeros(width, dtype=torch.float64), [], []
    gd = gw.double()
    for t in range(n):
        u = ref.causal_conv_token(yx[t, width:].double(), tp.double(), cb.double(), past).to(dtype).double()
        r, i = ref.rglru_gates(u, gd[:, 0], ra.double().view(blocks, m), gd[:, 1], ri.double().view(blocks, m))
        S = ref.rglru_step(S, u, r, i, lam)
        want.append(S * ref.gelu_tanh(yx[t, :width].double()))
    want = torch.stack(want)
    base = (-8 * torch.nn.functional.softplus(lam)).float()
    args = [z.to(DEV) for z in (gw, tp.t().contiguous(), cb, ra, ri, base)]
    cache = HybridCacheManager([StateSpec((("S", (width,)), ("conv", (taps, width))))], 3, 64, 4096, dtype, DEV)
    for a in cache[0].arrays.values():
        a.fill_(float("nan"))
    for row, counts in ((1, [n]), (0, [2, 2, 3, 120, 1, 1, 1, 2, 138]), (2, [1] * 40 + [230]), (1, [128, 142])):
        cache.recycle([row])
        at, got = 0, []
        for c in counts:
            cs = [0, 0, 0]
            cs[row] = c
            step = cache.step(cs, torch.zeros(c, dtype=torch.long), 1)
            cache.begin_step(step)
            got.append(hybrid.rglru(step, yx[at: at + c].to(DEV), *args, cache[0]["S"], cache[0]["conv"]).cpu())
            at += c
        got = torch.cat(got).double()
        scale = want.abs().max()
        assert float((got - want).abs().max() / scale) < (0.01 if dtype == BF16 else 1e-5), counts
        assert float((cache[0]["S"][row].double().cpu() - S).abs().max() / S.abs().max()) < (0.01 if dtype == BF16 else 1e-5)


def test_gates_and_activation():
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(0)
    for dtype, tol in ((BF16, 2e-2), (FP32, 1e-5)):
        for H, vd, row in ((3, 16, 64), (5, 7, 64), (2, 128, 128)):
            step = Step([1, 4, 0, 2], [3, 0, 0, 5], [0, 1, 2, 3], torch.zeros(7, dtype=torch.long), 1, DEV)
            a = torch.randn(step.staging_rows, H, row, generator=g).to(dtype)
            gate = (torch.randn(7, H * vd + 3, generator=g) * 30).to(dtype)
            got = hybrid.gate_heads(step, a.to(DEV), gate.to(DEV)[:, 3:], vd).double().cpu()
            want = a[step.q_row.cpu().long()][:, :, :vd].reshape(7, -1).double() * torch.sigmoid(gate[:, 3:].double())
            torch.testing.assert_close(got, want, rtol=tol, atol=1e-6)
        for n in (48, 37):
            o, gate, w = torch.randn(5, n, generator=g).to(dtype), torch.randn(5, n, generator=g).to(dtype), torch.randn(n, generator=g)
            got = hybrid.norm_gate(o.to(DEV), w.to(DEV), gate.to(DEV), 1e-2).double().cpu()
            torch.testing.assert_close(got, ref.rms_norm(o.double(), w.double(), 1e-2) * torch.sigmoid(gate.double()), rtol=tol, atol=1e-5)
            got = hybrid.relu_squared_(o.to(DEV).clone()).double().cpu()
            torch.testing.assert_close(got, torch.relu(o.double()) ** 2, rtol=tol, atol=1e-6)


# ---- whole models ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("name", list(gm.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    cfg = gm.CONFIGS[name]
    model, w = build(cfg, dtype)
    toks = prompt(cfg, 150, 2)
    want = ref.Sequence(cfg, w).run(toks)
    b = batcher(model)
    whole = None
    for sizes in ([150], [1], [2], [7, 64, 2, 33], [130, 1], [64], [63, 2, 1]):
        slot = b.open()
        got = feed(b, slot, toks, sizes)
        b.close(slot)
        assert gm.error(got, want) < TOL[dtype], sizes
        whole = got if whole is None else whole
        assert gm.error(got, whole) < TOL[dtype], sizes
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_unequal_requests_in_one_batch(dtype):
    """Prompts, portions and decoded tokens of several requests share steps; slots and pages go round: the pool
    holds fewer tokens than all requests together, rows are freed and taken in another order."""
    cfg = gm.CONFIGS["mixed"]
    model, w = build(cfg, dtype, 7)
    lens = [140, 9, 75, 66, 1, 130, 64, 20]
    toks = [prompt(cfg, n, 20 + i) for i, n in enumerate(lens)]
    want = [ref.Sequence(cfg, w).run(t) for t in toks]
    b = batcher(model, slots=3, pool_tokens=64 * 7, max_len=64 * 4)
    rng = torch.Generator().manual_seed(1)
    live, todo, got = {}, list(range(len(lens))), [[] for _ in lens]
    while live or todo:
        while todo and len(live) < 3:
            live[todo.pop(0)] = [b.open(), 0]
        step, take = {}, {}
        for i, (slot, at) in live.items():
            r = int(torch.randint(0, 5, (1,), generator=rng))
            n = min([1, 2, 1, 17, 64][r], lens[i] - at)
            if len(live) > 1 and r == 2 and step:
                continue                    # left out of this step
            step[slot], take[i] = toks[i][at: at + n], n
        logits = b.step(step, {live[i][0]: range(n) for i, n in take.items()}).float().cpu()
        off = 0
        for i, n in take.items():
            got[i].append(logits[off: off + n])
            off += n
            live[i][1] += n
        for i in [i for i, (s, at) in live.items() if at == lens[i]]:
            b.close(live.pop(i)[0])
    for i in range(len(lens)):
        assert gm.error(torch.cat(got[i]), want[i]) < TOL[dtype], i
    bits, free = b.pool.query()
    assert bits == 0 and free == b.pool.n_pages


def test_long_decoding_keeps_its_precision():
    cfg = gm.config([gm.layer("lightning", gm.lin(2, 16, 16, [0.999, 0.9]), 24), gm.layer("rglru", gm.lru(24, 2, 4), 24),
                     gm.layer("attention", gm.att(2, 1, 16, 16, every=50))], 32)
    model, w = build(cfg, FP32, 9)
    toks = prompt(cfg, 600, 3)
    want = ref.Sequence(cfg, w).run(toks)
    b = batcher(model, slots=1)
    got = feed(b, b.open(), toks, [5, 1])
    assert gm.error(got[-100:], want[-100:]) < 1e-4


# ---- generation through the framework's loops ----------------------------------------------------------------
def greedy(cfg, w, toks, n):
    s = ref.Sequence(cfg, w)
    logits, out = s.run(toks)[-1], []
    for _ in range(n):
        out.append(int(logits.argmax()))
        logits = s.token(out[-1])
    return out


def test_greedy_generation():
    from pace_b200.llm.configs import SamplingConfig
    from pace_b200.llm.device_loop import GreedyDeviceLoop
    from pace_b200.llm.generator import Generator
    cfg = gm.CONFIGS["mixed"]
    model, w = build(cfg, FP32, 11)
    toks = [prompt(cfg, n, 40 + i) for i, n in enumerate((70, 3, 129, 20, 64))]
    want = [greedy(cfg, w, t, 12) for t in toks]
    b = batcher(model, slots=2, pool_tokens=64 * 8, prefill_chunk=48)
    for _ in range(2):                                  # the second run reuses slots and pages
        outs, stats = b.run(toks, 12)
        assert outs == want and stats.output_tokens == 60
    even = torch.stack([prompt(cfg, 30, 50), prompt(cfg, 30, 51)])
    want = [greedy(cfg, w, t, 9) for t in even]
    out = Generator(model).generate(even, SamplingConfig(max_new_tokens=9)).output_token_ids
    assert out[:, 30:].tolist() == want
    # device-resident loop: one recorded step per token
    cache = model.new_cache(2, 64 * 8, 200)
    with torch.inference_mode():
        last = model.forward_ragged(even.to(DEV), [30, 30], cache).logits[:, -1].argmax(-1)
        loop = GreedyDeviceLoop(model, cache, last, torch.full((2,), 30, device=DEV), max_new_tokens=80)
        loop.run()
    assert [[int(f)] + r[:8] for f, r in zip(last, loop.tokens.tolist())] == want
    assert loop.tokens[0, :79].tolist() == greedy(cfg, w, even[0], 80)[1:80]        # across page borders


def test_beam_search_follows_the_states():
    from pace_b200.llm.configs import SamplingConfig
    from pace_b200.llm.generator import Generator
    cfg = gm.config([gm.layer("lightning", gm.lin(2, 12, 12, [0.9, 0.99]), 24), gm.layer("rglru", gm.lru(24, 2, 3)),
                     gm.layer("attention", gm.att(2, 1, 16, 16), 24)], 32)
    model, w = build(cfg, FP32, 13)
    p = prompt(cfg, 66, 60)
    got = Generator(model).generate(p[None], SamplingConfig(max_new_tokens=6, num_beams=3)).output_token_ids[0, 66:].tolist()

    def score(seq):
        lp = torch.log_softmax(ref.Sequence(cfg, w).run(torch.cat([p, torch.tensor(seq)])), -1)
        return sum(float(lp[65 + i, t]) for i, t in enumerate(seq))
    beams = [([], 0.0)]
    for _ in range(6):
        cand = []
        for seq, s in beams:
            lp = torch.log_softmax(ref.Sequence(cfg, w).run(torch.cat([p, torch.tensor(seq, dtype=torch.long)]))[-1], -1)
            cand += [(seq + [t], s + float(lp[t])) for t in range(cfg["vocab"])]
        beams = sorted(cand, key=lambda c: -c[1])[:3]
    assert got == beams[0][0] and abs(score(got) - beams[0][1]) < 1e-6


def test_pool_limits_and_refusals():
    from pace_b200.llm.serving import WaveServer
    cfg = gm.CONFIGS["ones"]
    model, _ = build(cfg, BF16)
    b = batcher(model, slots=1, pool_tokens=128, max_len=128)
    s = b.open()
    b.step({s: prompt(cfg, 128, 0)})
    with pytest.raises(RuntimeError, match="max_seq_len"):
        b.step({s: prompt(cfg, 1, 0)})
    with pytest.raises(RuntimeError, match="slots are taken"):
        b.open()
    b.close(s)
    with pytest.raises(ValueError, match="token ids"):
        b.step({b.open(): torch.tensor([cfg["vocab"]])})
    with pytest.raises(NotImplementedError, match="rolled back"):
        b.manager.remove_cache(1)
    with pytest.raises(TypeError, match="ContinuousBatcher"):
        WaveServer(model, 128, 1, 128)


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_trace_replay_program(tmp_path, dtype):
    from pace_b200.llm.weights import write_safetensors
    cfg = gm.CONFIGS["mixed"]
    w = gm.weights(cfg, 15)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    a, c = prompt(cfg, 70, 1), prompt(cfg, 12, 2)
    wa, wc = ref.Sequence(cfg, w).run(a), ref.Sequence(cfg, w).run(c)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66].tolist(), "want": [0, 65]},
                                     {"id": "c", "tokens": c[:1].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "c", "tokens": c[1:3].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "c", "tokens": c[3:].tolist(), "want": [8, 2]},
                                     {"id": "a", "tokens": a[66:67].tolist(), "want": [0]}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "c2", "tokens": c.tolist(), "want": [11]}], "end": ["a", "c2"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", str(dtype)[6:],
                          "--out", str(tmp_path), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]

    def out(i):
        raw = (tmp_path / f"{i}.f32").read_bytes()
        return torch.frombuffer(bytearray(raw), dtype=torch.float32).view(-1, cfg["vocab"])
    assert gm.error(out(0), wa[[0, 65]]) < TOL[dtype] and not (tmp_path / "1.f32").exists()
    assert gm.error(out(2), torch.stack([wc[11], wc[5], wa[66]])) < TOL[dtype]
    assert gm.error(out(3), wc[[11]]) < TOL[dtype]
