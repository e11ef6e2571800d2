"""The Kibotar model on the GPU against the plain implementation: every mechanism alone, then whole models, prompts, portions,
decoding, batches, reuse of pages and slots, and generation through the framework's loops."""
import json
import math
import os
import subprocess

import pytest
import torch

import kibotar_models as km
from oracle import kibotar_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF16, FP32 = torch.bfloat16, torch.float32
TOL = {BF16: 0.06, FP32: 1e-4}
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))


@pytest.fixture(params=[(1, 2), None], ids=["tiles", "tokens"])
def form(request, monkeypatch):
    """Prompt portions take the tile form of pooled attention whatever their size, or token by token."""
    from pace_b200.ops import hybrid
    monkeypatch.setattr(hybrid, "PROMPT_TOKENS", request.param or (1 << 30, 2))


def build(cfg, dtype, seed=0):
    from pace_b200.llm.registry import build_model
    w = km.weights(cfg, seed)
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


def manager(specs, dtype, rows=2, tokens=1024):
    from pace_b200.llm.hybrid_cache import HybridCacheManager
    c = HybridCacheManager(specs, rows, rows * tokens, tokens, dtype, DEV)
    for s in c.states:                       # a state is never cleared: what a slot holds must not matter
        for x in s.arrays.values():
            x.fill_(float("nan") if x.dtype == FP32 else -7)
    return c


def over_portions(cache, row, counts, fn):
    """``fn(step, lo, hi)`` for every portion of one sequence; the outputs back to back."""
    out, at = [], 0
    for n in counts:
        c = [0] * cache.batch
        c[row] = n
        step = cache.step(c, torch.zeros(n, dtype=torch.long), 1)
        cache.begin_step(step)
        out.append(fn(step, at, at + n).cpu())
        at += n
    cache.pool.check_status()
    return torch.cat(out).double()


def row_error(got, want):
    """Largest error of a row over the rms of all of them."""
    return float((got - want).flatten(1).pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt())


# ---- attention over a window and pooled blocks, with mixed heads -----------------------------------------------------------
def pooled_cache(m, dtype, tokens=1024, rows=2):
    from pace_b200.llm.hybrid_cache import BlockSpec, JointSpec, KVSpec
    sizes = (m["kv_heads"], m["dim"], m["vdim"])
    return manager([JointSpec((KVSpec(*sizes), BlockSpec(*sizes, m["mask"]["pool"])))], dtype, rows, tokens)


def operands(m, n, dtype, seed=0):
    g = torch.Generator().manual_seed(seed)
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    qkv = torch.randn(n, H * d + G * (d + vd), generator=g)
    qkv[:, : H * d] *= 1.5
    return qkv.to(dtype), torch.randn(n, H * vd, generator=g).to(dtype), torch.eye(H) + torch.randn(H, H, generator=g) * 0.5


def attend(m, qkv, gate, mix, cache, row, counts, sinks=True, tables=True):
    from pace_b200.ops import RotaryEmbedding, hybrid
    H, rot = m["heads"], m["rot"]["dims"] if tables else 0
    tb = RotaryEmbedding({"rope_type": "precise"}, rot, 8192, m["rot"]["base"]).device_tables(DEV) if rot else None
    zero = torch.zeros(H, device=DEV) if sinks else None
    mix = mix.float().to(DEV) if mix is not None else None

    def run(step, lo, hi):
        p = torch.cat([qkv[lo:hi], gate[lo:hi]], 1).to(DEV) if gate is not None else qkv[lo:hi].to(DEV)
        return hybrid.pooled_attention(step, *cache[0], p, tb, H, m["dim"], m["vdim"], m["scale"], m["mask"]["size"], m["mask"]["pool"], zero,
                                       mix, p[:, qkv.shape[1]:] if gate is not None else None)
    return over_portions(cache, row, counts, run).view(len(qkv), H, m["vdim"])


def plain(m, qkv, gate, mix, sinks=True, tables=True):
    n, H, G, d, vd = len(qkv), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = torch.split(qkv.double(), [H * d, G * d, G * vd], -1)
    q, k, v = q.view(n, H, d), k.reshape(n, G, d), v.reshape(n, G, vd)
    if tables:
        q, k = (ref.rotate_half(x, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
    size, window = m["mask"]["pool"], m["mask"]["size"]
    if sinks:
        p = ref.pooled_weights(q, k, m["scale"], window, size)
    else:
        keys, unseen = torch.cat([k, ref.block_means(k, size)]), ~ref.pooled_mask(n, window, size)
        p = torch.stack([torch.softmax(((q[:, h] @ keys[:, h // (H // G)].T) * m["scale"]).masked_fill(unseen, -math.inf), -1)
                         for h in range(H)])
    o = ref.mixed_heads(p, v, mix.double() if mix is not None else torch.eye(H).double(), size)
    return o * ref.sigmoid(gate.double()).view(n, H, vd) if gate is not None else o


SHAPES = [(BF16, 6, 2, 40, 24, 37, 5, 24), (BF16, 10, 5, 64, 120, 100, 16, 32), (BF16, 32, 8, 128, 128, 70, 8, 64), (BF16, 8, 8, 48, 64, 64, 64, 48),
          (BF16, 3, 1, 22, 13, 19, 7, 6), (BF16, 4, 2, 136, 72, 33, 4, 136), (BF16, 2, 2, 16, 16, 1, 1, 2), (BF16, 40, 2, 32, 56, 130, 3, 2),
          (BF16, 12, 12, 72, 128, 50, 100, 24), (BF16, 7, 1, 64, 64, 200, 32, 64), (BF16, 33, 1, 64, 64, 40, 6, 8),
          (FP32, 6, 2, 40, 24, 37, 5, 24), (FP32, 3, 3, 22, 13, 1, 2, 22), (FP32, 4, 1, 136, 160, 64, 16, 8)]


@pytest.mark.parametrize("dtype,H,G,d,vd,window,block,rot", SHAPES)
def test_pooled_attention_at_every_position(dtype, H, G, d, vd, window, block, rot, form):
    """Prompts, portions and decoding against the plain form; blocks are completed inside portions, across them and by
    decoded tokens."""
    n = 330
    m = km.att(H, G, d, vd, window, block, rot, 1e3)
    qkv, gate, mix = operands(m, n, dtype, H)
    want = plain(m, qkv, gate, mix)
    cache = pooled_cache(m, dtype)
    for row, counts in ((1, [n]), (0, [1] * 130 + [2] * 40 + [3, 20, 15, 82]), (1, [64, 63, 1, 2, 130, 17, 16, 1, 36]), (0, [15, 1, 300, 14])):
        got = attend(m, qkv, gate, mix, cache, row, counts)
        assert row_error(got, want) < (0.03 if dtype == BF16 else 1e-5), counts[:4]
        cache.recycle([row])


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("with_mix,with_gate,sinks", [(False, False, False), (True, False, True), (False, True, True)])
def test_pooled_attention_without_its_parts(dtype, with_mix, with_gate, sinks, form):
    m = km.att(8, 4, 32, 40, 45, 6, 16)
    qkv, gate, mix = operands(m, 200, dtype, 1)
    gate, mix = gate if with_gate else None, mix if with_mix else None
    want = plain(m, qkv, gate, mix, sinks)
    for counts in ([200], [100] + [1] * 100):
        got = attend(m, qkv, gate, mix, pooled_cache(m, dtype), 0, counts, sinks)
        assert row_error(got, want) < (0.03 if dtype == BF16 else 1e-5)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("window,block", [(70, 12), (64, 64), (65, 5), (33, 24), (1, 8), (130, 1)])
@pytest.mark.parametrize("tail", [[200], [1] * 200, [7, 1, 50, 2, 140]])
def test_a_key_that_stands_out(dtype, window, block, tail, form):
    """One key has nearly all the weight where it is seen: just inside and just outside the window, between window and block, and
    in the mean of its block from the first position that sees it.  Its value is recognised in every output."""
    H, G, d = 4, 2, 64
    m = km.att(H, G, d, d, window, block, 2, scale=1.0)
    n, at = 300, 83
    qkv, _, _ = operands(m, n, dtype, 3)
    q, k, v = qkv[:, : H * d].view(n, H, d), qkv[:, H * d: H * d + G * d].view(n, G, d), qkv[:, -G * d:].view(n, G, d)
    q.mul_(0.05), k.mul_(0.05), v.mul_(0.1)
    q[:, :, 0] = 6.0
    k[:, :, 0] = 0.0
    k[at, :, 0], v[at] = 2.0 * block, 8.0           # score 12 as a part of its block's mean, 12 x block as a token
    want = plain(m, qkv, None, None, tables=False)
    token = [i for i in range(n) if 0 <= i - at < window]
    last = at // block * block + block - 1
    pooled = [i for i in range(n) if i - window >= last]
    big = (want[:, 0, 0] > 8.0 / block / 2).nonzero().flatten().tolist()
    assert big == sorted(token + pooled)            # (the case shows what it should)
    got = attend(m, qkv, None, None, pooled_cache(m, dtype), 0, [100] + tail, tables=False)
    assert float((got - want).abs().max()) < (0.05 if dtype == BF16 else 1e-4)


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_one_in_the_denominator(dtype, form):
    """With scores far below 0 hardly any weight is left; with scores far above 0 the one does not matter."""
    for level in (-6.0, 0.0, 30.0):
        m = km.att(4, 2, 64, 64, 20, 4, 2, scale=1.0)
        qkv, _, mix = operands(m, 120, dtype, 5)
        qkv[:, : 4 * 64] = 0.01 * qkv[:, : 4 * 64]
        qkv[:, : 4 * 64: 64] = level
        qkv[:, 4 * 64: 6 * 64: 64] = 1.0
        want = plain(m, qkv, None, mix, tables=False)
        for counts in ([120], [60] + [1] * 60):
            got = attend(m, qkv, None, mix, pooled_cache(m, dtype), 0, counts, tables=False)
            assert row_error(got, want) < (0.03 if dtype == BF16 else 1e-4), level


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_mixing_crosses_kv_heads(dtype, form):
    """A permutation of the heads: head h takes another head's weights to its own values."""
    m = km.att(6, 3, 32, 16, 30, 4, 8)
    qkv, gate, _ = operands(m, 150, dtype, 6)
    mix = torch.eye(6)[[5, 3, 0, 4, 1, 2]]
    want = plain(m, qkv, gate, mix)
    for counts in ([150], [50] + [1] * 100):
        assert row_error(attend(m, qkv, gate, mix, pooled_cache(m, dtype), 0, counts), want) < (0.03 if dtype == BF16 else 1e-5)


def test_weights_keep_more_than_bf16(form):
    """Two keys with nearly the same weight whose values nearly cancel: what is left shows the weights' rounding."""
    m = km.att(2, 1, 64, 64, 64, 64, 2, scale=1.0)
    n = 33
    qkv = torch.zeros(n, 2 * 64 + 64 + 64)
    qkv[:, 0] = qkv[:, 64] = 1.0                     # both query heads
    qkv[:, 128] = -40.0
    qkv[0, 128], qkv[1, 128] = 4.0, 4.03125
    qkv[0, 192:], qkv[1, 192:] = 1.0, -1.0
    qkv = qkv.to(BF16)
    want = plain(m, qkv, None, torch.eye(2), tables=False)[1:]
    for counts in ([n], [2] + [1] * (n - 2)):
        got = attend(m, qkv, None, torch.eye(2), pooled_cache(m, BF16), 0, counts, tables=False)[1:]
        assert float(((got - want).abs() / want.abs()).max()) < 0.02


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_thousands_of_keys(dtype, form):
    """Far blocks stand out among a thousand; decoding shares a token's keys over a cluster."""
    m = km.att(4, 2, 64, 64, 90, 3, 64)
    n = 3300
    qkv, gate, mix = operands(m, n, dtype, 8)
    qkv[10:13, 4 * 64: 5 * 64] = qkv[3290, :64] * 3
    want = plain(m, qkv, gate, mix)
    got = attend(m, qkv, gate, mix, pooled_cache(m, dtype, 3400, 1), 0, [2000, 1270] + [1] * 25 + [5])
    assert row_error(got[1500:], want[1500:]) < (0.03 if dtype == BF16 else 1e-5)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("d,rot", [(64, 64), (40, 24), (22, 6), (24, 0)])
def test_rotation_pairs(dtype, d, rot):
    """Pairs of halves and of neighbours; the queries' staging rows."""
    from pace_b200.ops import RotaryEmbedding
    m = km.att(3, 1, d, d, 16, 4, rot, 50.0)
    qkv, _, _ = operands(m, 40, dtype, 9)
    x = qkv[:, : 3 * d].double().view(40, 3, d)
    swap = torch.tensor(list(range(0, rot, 2)) + list(range(1, rot, 2)) + list(range(rot, d)))
    for halves in (True, False):
        want = ref.rotate_half(x, rot, 50.0) if halves else torch.empty_like(x)
        if not halves:
            want[..., swap] = ref.rotate_half(x[..., swap], rot, 50.0)
        cache = pooled_cache(m, dtype)
        tb = RotaryEmbedding({"rope_type": "precise"}, rot, 64, 50.0).device_tables(DEV) if rot else (None, None)
        step = cache.step([0, 40], torch.zeros(40, dtype=torch.long), 1)
        cache.begin_step(step)
        kv, bl = cache[0]
        row = kv.pool.head_dim * 2 // dtype.itemsize
        q = torch.full((40, 3, row), 7.0, dtype=dtype, device=DEV)
        torch.ops.pace_b200.kv_append_rotate(kv.pool.handle, kv.pool.pages, kv.layer, bl.pool.handle, bl.pool.pages, bl.layer, step.handle,
                                             qkv.to(DEV), *tb, q, d, d, halves, 4, False)
        torch.testing.assert_close(q[:, :, :d].double().cpu(), want, rtol=1e-2 if dtype == BF16 else 1e-5, atol=1e-2 if dtype == BF16 else 1e-5)
        assert row == d or float(q[:, :, d:].abs().max()) == 0


# ---- gated linear attention -------------------------------------------------------------------------------------------------
def gla_case(dtype, H, d, vd, n, tau, low, high, seed=0):
    g = torch.Generator().manual_seed(seed)
    qkv = torch.randn(n, H * (2 * d + vd), generator=g).to(dtype)
    z = (torch.rand(n, H * d, generator=g) * (high - low) + low).to(dtype)
    bias = torch.randn(H * d, generator=g) * 0.5
    return qkv, z, bias, torch.randn(n, H * vd, generator=g).to(dtype), 1 + 0.3 * torch.randn(vd, generator=g)


def plain_gla(qkv, z, bias, gate, norm, H, d, vd, tau, eps):
    n = len(qkv)
    q, k, v = torch.split(qkv.double(), [H * d, H * d, H * vd], -1)
    alpha = ref.sigmoid(z.double() + bias.double()) ** (1.0 / tau)
    o = ref.gla_scan(q.view(n, H, d) * d ** -0.5, k.view(n, H, d), v.view(n, H, vd), alpha.view(n, H, d))
    return (ref.rms(o, eps) * norm.double()).reshape(n, H * vd) * ref.silu(gate.double())


GLA = [(BF16, 2, 64, 64, 16.0, -1, 6), (BF16, 3, 128, 136, 1.0, -4, 8), (BF16, 1, 24, 40, 4.0, -30, 2), (BF16, 2, 72, 16, 0.5, -30, 12),
       (BF16, 3, 13, 21, 5.5, -2, 4), (BF16, 1, 160, 72, 16.0, -2, 4), (BF16, 1, 8, 8, 2.0, -200, -100), (FP32, 2, 64, 64, 16.0, -1, 6),
       (FP32, 3, 24, 40, 0.7, -30, 12), (FP32, 1, 130, 33, 1.0, 0, 9), (FP32, 2, 1, 300, 3.0, 0, 4)]


@pytest.mark.parametrize("dtype,H,d,vd,tau,low,high", GLA)
def test_gated_linear_attention(dtype, H, d, vd, tau, low, high):
    """Decays from hardly any to whole rows per token; chunks, portions and single tokens; slots that held anything."""
    from pace_b200.llm.hybrid_cache import StateSpec
    from pace_b200.ops import hybrid
    n, eps = 300, 1e-4
    qkv, z, bias, gate, norm = gla_case(dtype, H, d, vd, n, tau, low, high, d)
    want = plain_gla(qkv, z, bias, gate, norm, H, d, vd, tau, eps)
    cache = manager([StateSpec((("S", (H, d, vd)),))], dtype)

    def run(step, lo, hi):
        return hybrid.gla(step, qkv[lo:hi].to(DEV), z[lo:hi].to(DEV), bias.to(DEV), cache[0]["S"], norm.to(DEV), gate[lo:hi].to(DEV), tau,
                          d ** -0.5, eps)
    for row, counts in ((1, [n]), (0, [1] * 90 + [2] * 15 + [64, 65, 51]), (1, [63, 1, 2, 130, 104])):
        got = over_portions(cache, row, counts, run)
        assert row_error(got, want) < (0.03 if dtype == BF16 else 2e-5), counts[:4]
        cache.recycle([row])


def test_small_additions_to_a_large_state():
    """Thousands of tokens with hardly any decay: the state keeps fp32."""
    from pace_b200.llm.hybrid_cache import StateSpec
    from pace_b200.ops import hybrid
    H, d, vd, n = 2, 64, 32, 2600
    qkv, z, bias, gate, norm = gla_case(BF16, H, d, vd, n, 16.0, 8, 12, 3)
    qkv[:, H * d:] = qkv[:, H * d:].abs()            # keys and values of one sign: a sum that grows
    want = plain_gla(qkv, z, bias, gate, norm, H, d, vd, 16.0, 1e-5)
    cache = manager([StateSpec((("S", (H, d, vd)),))], BF16, tokens=n)

    def run(step, lo, hi):
        return hybrid.gla(step, qkv[lo:hi].to(DEV), z[lo:hi].to(DEV), bias.to(DEV), cache[0]["S"], norm.to(DEV), gate[lo:hi].to(DEV), 16.0,
                          d ** -0.5, 1e-5)
    got = over_portions(cache, 0, [2500] + [1] * 100, run)
    assert row_error(got, want) < 0.02
    q, k, v = torch.split(qkv.double(), [H * d, H * d, H * vd], -1)
    alpha = (ref.sigmoid(z.double() + bias.double()) ** (1 / 16)).view(n, H, d)
    S = torch.zeros(H, d, vd).double()
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t].view(H, d)[:, :, None] * v[t].view(H, vd)[:, None, :]
    torch.testing.assert_close(cache[0]["S"][0].double().cpu(), S, rtol=1e-4, atol=1e-3)


# ---- latent attention without positions ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("H,d,vd,rank", [(4, 32, 48, 64), (3, 11, 9, 21), (16, 128, 128, 512), (2, 72, 120, 40), (1, 8, 8, 8)])
def test_latent_attention_without_positions(dtype, H, d, vd, rank):
    from pace_b200.llm.hybrid_cache import LatentSpec
    from pace_b200.ops import hybrid
    n, eps, scale = 200, 1e-4, 1.3 / math.sqrt(d)
    g = torch.Generator().manual_seed(d)
    q, c, gate = torch.randn(n, H * d, generator=g) * 1.5, torch.randn(n, rank, generator=g), torch.randn(n, H, generator=g)
    q, c, gate = q.to(dtype), c.to(dtype), gate.to(dtype)
    w, norm = (torch.randn(H * (d + vd), rank, generator=g) / math.sqrt(rank)).to(dtype), 1 + 0.3 * torch.randn(rank, generator=g)
    lat = ref.rms(c.double(), eps) * norm.double()
    k, v = (lat @ w[: H * d].double().T).view(n, H, d), (lat @ w[H * d:].double().T).view(n, H, vd)
    want = ref.causal_softmax(q.double().view(n, H, d), k, v, scale) * ref.sigmoid(gate.double())[:, :, None]
    cache = manager([LatentSpec(rank, 0)], dtype)

    def run(step, lo, hi):
        down = torch.cat([c[lo:hi], gate[lo:hi]], 1).to(DEV)
        wide = torch.cat([q[lo:hi], q[lo:hi]], 1).to(DEV)[:, : H * d]         # (queries inside wider rows)
        o = hybrid.latent_attention(step, cache[0], down[:, :rank], None, norm.to(DEV), None, w.to(DEV), H, d, 0, vd, scale, eps, None, q=wide)
        return hybrid.gate_per_head_(o, down[:, rank:], H)
    for row, counts in ((1, [n]), (0, [70] + [1] * 30 + [2, 3, 95]), (1, [64, 63, 1, 2, 70])):
        got = over_portions(cache, row, counts, run).view(n, H, vd)
        assert row_error(got, want) < (0.03 if dtype == BF16 else 1e-5), counts[:4]
        cache.recycle([row])


# ---- shifted inputs and token pairs -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width,n", [(64, 40), (37, 21), (2200, 9), (256, 700), (136, 2600)])
def test_shifted_norms(dtype, width, n):
    """Two sequences side by side in portions: stream, norm and shift behind a sublayer's output, a bias and a vector."""
    from pace_b200.llm.hybrid_cache import StateSpec
    from pace_b200.ops import hybrid
    g, eps = torch.Generator().manual_seed(width), 1e-2
    xs, ys = [torch.randn(n, width, generator=g) for _ in range(2)], [torch.randn(n, width, generator=g).to(dtype) for _ in range(2)]
    wp, wn, bias, add = (torch.randn(width, generator=g) for _ in range(4))
    mix = torch.rand(width, generator=g)
    cache = manager([StateSpec((("h", (3, width)), ("next", (3, width))))], dtype, tokens=4096)
    cut = n // 2
    got = [[], []]
    for part in ((0, cut), (cut, n - 2), (n - 2, n - 1), (n - 1, n)):
        lo, hi = part
        counts = [int(lo == n - 1), hi - lo]           # the other sequence takes part in the last step only
        step = cache.step(counts, torch.zeros(sum(counts), dtype=torch.long), 1)
        cache.begin_step(step)
        rows = [(0, 0)] * counts[0] + [(1, i) for i in range(lo, hi)]
        x, y = torch.stack([xs[s][i] for s, i in rows]).to(DEV), torch.stack([ys[s][i] for s, i in rows]).to(DEV)
        before, after = cache[0]["h"][:, 1], cache[0]["h" if step.decode_only else "next"][:, 1]
        new, h = hybrid.shift_norm(step, x, wn.to(DEV), mix.to(DEV), before, after, eps, dtype, y, bias.to(DEV), wp.to(DEV), add.to(DEV))
        if not step.decode_only:
            hybrid.state_commit(step, cache[0]["next"], cache[0]["h"])
        for j, (s, i) in enumerate(rows):
            got[s].append((new[j].double().cpu(), h[j].double().cpu()))
    for s, m in ((1, n), (0, 1)):
        x = xs[s].double() + ref.rms(ys[s].double() + bias.double(), eps) * wp.double() + add.double()
        h = ref.token_shift(ref.rms(x, eps) * wn.double(), mix.double())
        torch.testing.assert_close(torch.stack([a for a, _ in got[s]]), x[:m], rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(torch.stack([b for _, b in got[s]]), h[:m], rtol=1e-2 if dtype == BF16 else 1e-5, atol=1e-2 if dtype == BF16 else 1e-5)
    # nothing taken up: the first layer
    cache.recycle([0])
    step = cache.step([3, 0], torch.zeros(3, dtype=torch.long), 1)
    x = xs[0][:3].to(DEV)
    new, h = hybrid.shift_norm(step, x, wn.to(DEV), mix.to(DEV), cache[0]["h"][:, 0], cache[0]["next"][:, 0], eps, dtype)
    assert torch.equal(new, x)
    want = ref.token_shift(ref.rms(xs[0][:3].double(), eps) * wn.double(), mix.double())
    torch.testing.assert_close(h.double().cpu(), want, rtol=1e-2 if dtype == BF16 else 1e-5, atol=1e-2 if dtype == BF16 else 1e-5)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("buckets,prev,cur", [(13, 7, 3), (1, 1, 1), (491, 2000003, 1999993)])
def test_embedding_of_token_pairs(dtype, buckets, prev, cur):
    """Products beyond 32 bits; a sequence's first token; the previous token across portions and in decoding."""
    from pace_b200.llm.hybrid_cache import StateSpec
    from pace_b200.ops import hybrid
    g, V, W = torch.Generator().manual_seed(buckets), 5000, 24
    e, b = torch.randn(V, W, generator=g).to(dtype), torch.randn(buckets + 1, W, generator=g).to(dtype)
    toks = torch.randint(0, V, (50,), generator=g)
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": buckets, "mul_prev": prev, "mul_cur": cur}}}
    want = ref.embed(toks, cfg, {"embed": e.double(), "bigram": b.double()})
    cache = manager([StateSpec((("token", ()),), torch.int32), StateSpec((("h", (2, 4)),))], dtype)
    token, h = cache[0]["token"], cache[1]["h"]
    for row, counts in ((1, [50]), (0, [1] * 9 + [2, 3, 1, 35]), (1, [20, 30])):
        at, got = 0, []
        for n in counts:
            c = [0, 0]
            c[row] = n
            step = cache.step(c, toks[at: at + n], V)
            cache.begin_step(step)
            got.append(hybrid.embed_pairs(step, e.to(DEV), 2.5, b.to(DEV), token, prev, cur).double().cpu())
            if not step.decode_only:
                hybrid.state_commit(step, h.clone(), h, token)
            at += n
        torch.testing.assert_close(torch.cat(got), want, rtol=1e-6, atol=1e-6)
        cache.recycle([row])


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("kind,mixer,ff", [
    (km.A, km.att(6, 2, 20, 28, 30, 4, 8, scaling=km.SCALING), None), (km.A, km.att(5, 5, 130, 33, 12, 9, 2), 40),
    (km.A, km.att(34, 1, 8, 16, 40, 8, 8, scale=-0.4), 21), (km.A, km.att(2, 2, 16, 16, 200, 64, 16), None),
    (km.G, km.gla(4, 24, 40, 2.0), None), (km.G, km.gla(5, 9, 33), 21), (km.L, km.lat(3, 20, 28, 36), None), (km.L, km.lat(2, 9, 130, 33), 40)])
def test_one_layer_models(kind, mixer, ff, dtype):
    cfg = km.config([km.layer(kind, mixer, ff)], 48, loop=(0, 1, 2))
    model, w = build(cfg, dtype, 5)
    toks = prompt(cfg, 110, 1)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    for sizes in ([110], [2, 3, 64, 5], [70, 1]):
        slot = b.open()
        assert km.error(feed(b, slot, toks, sizes), want) < TOL[dtype], sizes
        b.close(slot)
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype, form):
    cfg = km.CONFIGS[name]
    model, w = build(cfg, dtype)
    toks = prompt(cfg, 220, 2)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    whole = None
    for sizes in ([220], [1], [2], [7, 64, 2, 33], [200, 1], [64], [63, 2, 1], [3, 150, 2]):
        slot = b.open()
        got = feed(b, slot, toks, sizes)
        b.close(slot)
        assert km.error(got, want) < TOL[dtype], sizes
        whole = got if whole is None else whole
        assert km.error(got, whole) < TOL[dtype], sizes
    b.pool.check_status()


@pytest.mark.parametrize("loop,bigram", [(None, (5, 3, 2)), ((0, 2, 2), None), ((2, 3, 3), (31, 7, 11)), ((0, 3, 1), None)])
def test_loops_and_tables_of_pairs(loop, bigram):
    cfg = km.config([km.layer(km.L, km.lat(2, 16, 16, 24), 24), km.layer(km.A, km.att(2, 1, 16, 16, 20, 4, 8), None),
                     km.layer(km.G, km.gla(2, 16, 16), 24)], 32, loop=loop, bigram=bigram)
    model, w = build(cfg, FP32, 6)
    toks = prompt(cfg, 90, 4)
    b = batcher(model)
    assert km.error(feed(b, b.open(), toks, [60, 1]), ref.run(cfg, w, toks)) < 1e-4


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_unequal_requests_in_one_batch(dtype, form):
    """Prompts, portions and decoded tokens of several requests share steps; slots and pages go round: the pool holds
    fewer tokens than all requests together, rows are freed and taken in another order."""
    cfg = km.CONFIGS["mixed"]
    model, w = build(cfg, dtype, 7)
    lens = [140, 9, 75, 66, 1, 130, 64, 20, 200]
    toks = [prompt(cfg, n, 20 + i) for i, n in enumerate(lens)]
    want = [ref.run(cfg, w, t) for t in toks]
    b = batcher(model, slots=3, pool_tokens=64 * 8, max_len=64 * 4)
    for s in b.manager.states:
        for x in s.arrays.values():
            x.fill_(float("nan") if x.dtype == FP32 else -7)
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
        assert km.error(torch.cat(got[i]), want[i]) < TOL[dtype], i
    bits, free = b.pool.query()
    assert bits == 0 and free == b.pool.n_pages
    assert all(p.query()[1] == p.n_pages for p in b.pool.pools)      # the pages of blocks as well


def test_pages_of_blocks_follow_the_token_pages():
    """A pool that is full to the last token: every row's blocks have their pages, and new requests find them again."""
    cfg = km.config([km.layer(km.A, km.att(2, 1, 16, 16, 20, 3, 8), None), km.layer(km.A, km.att(2, 1, 16, 16, 9, 7, 8), None)], 32)
    model, w = build(cfg, FP32, 8)
    b = batcher(model, slots=4, pool_tokens=64 * 8, max_len=64 * 8)
    toks = [prompt(cfg, n, i) for i, n in enumerate((128, 128, 128, 128, 512, 64, 448))]
    for group in ((0, 1, 2, 3), (4,), (5, 6)):
        slots = {i: b.open() for i in group}
        logits = b.step({s: toks[i] for i, s in slots.items()}, {s: [len(toks[i]) - 1] for i, s in slots.items()}).cpu()
        for row, i in zip(logits, group):
            assert km.error(row[None], ref.run(cfg, w, toks[i])[-1:]) < 1e-4
        for s in slots.values():
            b.close(s)
    b.pool.check_status()


def test_long_decoding_keeps_its_precision():
    cfg = km.config([km.layer(km.A, km.att(4, 2, 16, 16, 50, 8, 8, scaling=km.SCALING), 24), km.layer(km.G, km.gla(2, 16, 24), None),
                     km.layer(km.L, km.lat(2, 16, 16, 24), 16)], 32, loop=(1, 2, 2))
    model, w = build(cfg, FP32, 9)
    toks = prompt(cfg, 700, 3)
    want = ref.run(cfg, w, toks)
    got = feed(batcher(model, slots=1), 0, toks, [5, 1])
    assert km.error(got[-100:], want[-100:]) < 1e-4


def test_a_step_in_which_nothing_is_wanted():
    model, w = build(km.CONFIGS["mixed"], BF16, 3)
    b = batcher(model)
    assert b.step({b.open(): prompt(km.CONFIGS["mixed"], 5, 1)}, {0: []}).shape == (0, 67)


# ---- generation through the framework's loops ---------------------------------------------------------------------------
def greedy(cfg, w, toks, n):
    seq = list(map(int, toks))
    for _ in range(n):
        seq.append(int(ref.run(cfg, w, seq)[-1].argmax()))
    return seq[len(toks):]


def test_greedy_generation():
    from pace_b200.llm.configs import SamplingConfig
    from pace_b200.llm.device_loop import GreedyDeviceLoop
    from pace_b200.llm.generator import Generator
    cfg = km.CONFIGS["mixed"]
    model, w = build(cfg, FP32, 11)
    toks = [prompt(cfg, n, 40 + i) for i, n in enumerate((70, 3, 129, 20, 64))]
    want = [greedy(cfg, w, t, 6) for t in toks]
    b = batcher(model, slots=2, pool_tokens=64 * 8, prefill_chunk=48)
    for _ in range(2):                                  # the second run reuses slots and pages
        outs, stats = b.run(toks, 6)
        assert outs == want and stats.output_tokens == 30
    even = torch.stack([prompt(cfg, 30, 50), prompt(cfg, 30, 51)])
    want = [greedy(cfg, w, t, 7) for t in even]
    out = Generator(model).generate(even, SamplingConfig(max_new_tokens=7)).output_token_ids
    assert out[:, 30:].tolist() == want
    # device-resident loop: one recorded step per token, across a page border and many blocks
    cache = model.new_cache(2, 64 * 8, 200)
    with torch.inference_mode():
        last = model.forward_ragged(even.to(DEV), [30, 30], cache).logits[:, -1].argmax(-1)
        loop = GreedyDeviceLoop(model, cache, last, torch.full((2,), 30, device=DEV), max_new_tokens=50)
        loop.run()
    assert [[int(f)] + r[:6] for f, r in zip(last, loop.tokens.tolist())] == want
    seq = even[0].tolist() + [int(last[0])] + loop.tokens[0].tolist()
    told = ref.run(cfg, w, seq[:-1])[29:].argmax(-1).tolist()
    assert told == seq[30:]


def test_recorded_decoding_in_bf16_follows_the_steps():
    """The recorded step (positions on the device) and steps made on the host give the same tokens."""
    from pace_b200.llm.device_loop import GreedyDeviceLoop
    cfg = km.CONFIGS["wide"]
    model, _ = build(cfg, BF16, 12)
    toks = torch.stack([prompt(cfg, 100, 1), prompt(cfg, 100, 2)])
    outs, _ = batcher(model).run(list(toks), 60)
    cache = model.new_cache(2, 64 * 8, 256)
    with torch.inference_mode():
        last = model.forward_ragged(toks.to(DEV), [100, 100], cache).logits[:, -1].argmax(-1)
        loop = GreedyDeviceLoop(model, cache, last, torch.full((2,), 100, device=DEV), max_new_tokens=60)
        got = loop.run()
    same = sum(([int(f)] + r[:59])[: 20] == o[: 20] for f, r, o in zip(last, got.tolist(), outs))
    assert same == 2


def test_beam_search_follows_the_states_and_rollback_is_refused():
    from pace_b200.llm.configs import SamplingConfig
    from pace_b200.llm.generator import Generator
    cfg = km.config([km.layer(km.A, km.att(2, 1, 16, 16, 9, 3, 8), 24), km.layer(km.G, km.gla(2, 16, 16), None),
                     km.layer(km.L, km.lat(2, 16, 16, 16), 24)], 32, loop=(0, 2, 2))
    model, w = build(cfg, FP32, 13)
    p = prompt(cfg, 66, 60)
    got = Generator(model).generate(p[None], SamplingConfig(max_new_tokens=7, num_beams=3)).output_token_ids[0, 66:].tolist()
    beams = [([], 0.0)]
    for _ in range(7):
        cand = []
        for seq, s in beams:
            lp = torch.log_softmax(ref.run(cfg, w, p.tolist() + seq)[-1], -1)
            cand += [(seq + [t], s + float(lp[t])) for t in range(cfg["vocab"])]
        beams = sorted(cand, key=lambda c: -c[1])[:3]
    assert got == beams[0][0]
    b = batcher(model, slots=1)
    feed(b, b.open(), prompt(cfg, 10, 9), [10])
    with pytest.raises(NotImplementedError):
        b.manager.remove_cache(7)


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_trace_replay_program(tmp_path, dtype):
    from pace_b200.llm.weights import write_safetensors
    cfg = km.CONFIGS["mixed"]
    w = km.weights(cfg, 15)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    a, c = prompt(cfg, 100, 1), prompt(cfg, 12, 2)
    wa, wc = ref.run(cfg, w, a), ref.run(cfg, w, c)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:96].tolist(), "want": [0, 95]},
                                     {"id": "c", "tokens": c[:1].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "c", "tokens": c[1:3].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "c", "tokens": c[3:].tolist(), "want": [8, 2]},
                                     {"id": "a", "tokens": a[96:97].tolist(), "want": [0]}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "c2", "tokens": c.tolist(), "want": [11]}], "end": ["a", "c2"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", str(dtype)[6:],
                          "--out", str(tmp_path), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]

    def out(i):
        raw = (tmp_path / f"{i}.f32").read_bytes()
        return torch.frombuffer(bytearray(raw), dtype=torch.float32).view(-1, cfg["vocab"])
    assert km.error(out(0), wa[[0, 95]]) < TOL[dtype] and not (tmp_path / "1.f32").exists()
    assert km.error(out(2), torch.stack([wc[11], wc[5], wa[96]])) < TOL[dtype]
    assert km.error(out(3), wc[[11]]) < TOL[dtype]
