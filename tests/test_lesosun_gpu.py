"""The Lesosun model on the GPU against the plain implementation: every mechanism alone, then whole models, prompts, portions,
decoding, batches, reuse of pages and slots, and generation through the framework's loops."""
import json
import math
import os
import subprocess

import pytest
import torch

import lesosun_models as lm
from oracle import lesosun_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF16, FP32 = torch.bfloat16, torch.float32
TOL = {BF16: 0.06, FP32: 1e-4}
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))


def build(cfg, dtype, seed=0):
    """bf16 models get corrections that settle the choice of experts: rounding then cannot flip one."""
    from pace_b200.llm.registry import build_model
    w = lm.weights(cfg, seed, decided=dtype == BF16)
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
            x.fill_(float("nan"))
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


# ---- attention behind convolutions, with capped scores ----------------------------------------------------------------
def attention_case(dtype, H, G, d, vd, conv, rot, n, scale, cap, seed=0, tokens=1024):
    from pace_b200.llm.hybrid_cache import KVSpec, StateSpec
    g = torch.Generator().manual_seed(seed)
    m = lm.left(H, G, d, vd, conv, rot, 1e4, scale, cap)
    ch = H * d + G * (d + vd)
    qkv = torch.randn(n, ch, generator=g).to(dtype)
    w = {"taps": torch.randn(ch, conv, generator=g) * 0.6, "q": 1 + torch.rand(d, generator=g), "k": 1 + torch.rand(d, generator=g)}
    cache = manager([KVSpec(G, d, vd), StateSpec((("conv", (max(conv, 1) + 1, ch + 8)),))], dtype, tokens=tokens)
    return m, w, qkv, cache


def attend(m, w, qkv, cache, row, counts, eps=1e-6, v_mul=1.0):
    from pace_b200.ops import RotaryEmbedding, hybrid
    rot, ch = m["rot"]["dims"], qkv.shape[1]
    tables = RotaryEmbedding({"rope_type": "precise"}, rot, 4096, m["rot"]["base"], is_neox_style=False).device_tables(DEV) if rot else None
    taps, qn, kn = w["taps"].t().contiguous().to(DEV), w["q"].to(DEV), w["k"].to(DEV)
    ring = cache[1]["conv"][:, :, :ch]

    def run(step, lo, hi):
        x = qkv[lo:hi].to(DEV)
        wide = torch.full((hi - lo, m["heads"] * m["vdim"] + 16), 7.0, dtype=qkv.dtype, device=DEV)
        out = wide[:, 8:-8]
        hybrid.conv_attention(step, cache[0], x, taps, ring, qn, kn, tables, m["heads"], m["dim"], m["vdim"], m["scale"], eps,
                              m["softcap"], v_mul, out)
        if not step.decode_only:
            hybrid.conv_store(step, x, ring)
        assert float((wide[:, :8] - 7).abs().max()) == 0 and float((wide[:, -8:] - 7).abs().max()) == 0
        return out.clone()
    return over_portions(cache, row, counts, run).view(len(qkv), m["heads"], m["vdim"])


def plain_attention(m, w, qkv, eps=1e-6):
    """``ref.capped_attention`` from given projections: they pass through identities."""
    ch, d = qkv.shape[1], m["dim"]
    eye, at, p = torch.eye(ch, dtype=torch.float64), 0, {}
    for x, c in (("q", m["heads"] * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * m["vdim"])):
        p[x], p[x + ".b"], p[x + ".conv"] = eye[at: at + c], torch.zeros(c).double(), w["taps"][at: at + c].double()
        at += c
    p.update({"q.norm": w["q"].double(), "k.norm": w["k"].double(), "o": torch.eye(m["heads"] * m["vdim"]).double(),
              "o.b": torch.zeros(m["heads"] * m["vdim"]).double()})
    return ref.capped_attention(qkv.double(), m, p, "", eps).view(len(qkv), m["heads"], m["vdim"])


SHAPES = [(BF16, 6, 2, 40, 24, 3, 16), (BF16, 10, 5, 64, 120, 4, 48), (BF16, 40, 2, 128, 64, 4, 32), (BF16, 3, 1, 22, 13, 5, 6),
          (BF16, 4, 2, 136, 72, 2, 136), (BF16, 2, 2, 16, 16, 1, 0), (FP32, 6, 2, 40, 24, 4, 16), (FP32, 3, 3, 22, 13, 2, 22),
          (FP32, 2, 1, 136, 160, 3, 8)]


@pytest.mark.parametrize("dtype,H,G,d,vd,conv,rot", SHAPES)
def test_conv_attention_against_plain(dtype, H, G, d, vd, conv, rot):
    """Every position of a prompt, of portions (also shorter than the taps) and of decoding."""
    n = 210
    m, w, qkv, cache = attention_case(dtype, H, G, d, vd, conv, rot, n, 0.15, 3.0, seed=H)
    want = plain_attention(m, w, qkv, 1e-3)
    for row, counts in ((0, [n]), (1, [129, 1, 1, 2, 3, 64, n - 200]), (0, [n - 40] + [1] * 40), (1, [1, 1, 2, 1, 2, 2, 3, n - 12])):
        got = attend(m, w, qkv, cache, row, counts, 1e-3)
        assert float((got - want).abs().max()) < (0.06 if dtype == BF16 else 3e-5), counts
        cache.recycle([row])
    got = attend(m, w, qkv, cache, 0, [n - 1, 1], 1e-3, v_mul=-1.25)
    assert float((got + 1.25 * want).abs().max()) < (0.08 if dtype == BF16 else 4e-5)


@pytest.mark.parametrize("dtype,H,G,d,vd,conv,rot", SHAPES)
def test_one_far_key_stands_out(dtype, H, G, d, vd, conv, rot):
    """A query finds the one key made for it, across page borders; capped, that key's weight is bounded by its closed form."""
    n = 260
    for t, j in ((259, 0), (64, 63), (128, 64), (191, 5), (255, 254), (127, 127)):
        m, w, qkv, cache = attention_case(dtype, H, G, d, vd, conv, rot, n, 1.0, 30.0, seed=t)
        w["taps"][:, :-1] = 0
        w["taps"][:, -1] = 1
        qkv[:, : (H + G) * d] = 0
        # the pair of dimensions behind the rotated ones, or the slowest pair, carries the match
        at = d - 2 if rot == d else rot
        at += (d - at) % 2 if rot == d else 0
        qkv[j, H * d + at: (H + G) * d: d] = 1
        qkv[t, at: H * d: d] = 1
        want = plain_attention(m, w, qkv)[t]
        value = qkv[j, (H + G) * d:].double().view(G, vd).repeat_interleave(H // G, 0)
        near = float((want - value).abs().max())
        if m["dim"] >= 40 and (rot < d):
            assert near < 1e-3                # 30 tanh(x / 30) leaves the match tens of units ahead
        for row, counts in ((0, [n]), (1, [t, 1] + [n - t - 1] * (t < n - 1)), (0, [50, 2, t - 53, 3, n - t - 2] if 55 < t < n - 2 else [n - 2, 2])):
            got = attend(m, w, qkv, cache, row, counts)[t]
            assert float((got - want).abs().max()) < (0.05 if dtype == BF16 else 1e-4), (t, j, counts)
            cache.recycle([row])


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("cap", [0.5, 8.0, 60.0])
def test_scores_are_capped(dtype, cap):
    """Scores far beyond the cap on either side: every weight is e^(+-cap) over their sum; without the cap one key would win."""
    H, G, d, vd, n = 4, 2, 32, 16, 150
    m, w, qkv, cache = attention_case(dtype, H, G, d, vd, 1, 0, n, 100.0, cap, seed=3)
    w["taps"][:] = 1
    w["q"][:], w["k"][:] = 1, 1
    qkv[:, : (H + G) * d] = 0
    qkv[:, : H * d: d] = 1
    signs = (torch.arange(n) % 3 == 0).to(dtype) * 2 - 1
    size = 1 + torch.rand(n, generator=torch.Generator().manual_seed(1))
    qkv[:, H * d: (H + G) * d: d] = (signs.float() * size)[:, None].to(dtype)     # (normalised: only the sign stays)
    x = qkv[:, (H + G) * d:].double().view(n, G, vd).repeat_interleave(H // G, 1)
    e = torch.exp(signs.double() * cap)
    for counts in ([n], [n - 1, 1], [60, 2, n - 62]):
        got = attend(m, w, qkv, cache, 0, counts)
        for t in (n - 1, n - 40, 3):
            want = (e[: t + 1, None, None] * x[: t + 1]).sum(0) / e[: t + 1].sum()
            if counts[0] > t or counts[-1] == 1 or counts[0] == 60:
                assert float((got[t] - want).abs().max()) < (0.01 if dtype == BF16 else 2e-6), (counts, t)
        cache.recycle([0])


def test_long_contexts_split_over_a_cluster():
    H, G, d, vd, n = 8, 1, 128, 128, 3000
    m, w, qkv, cache = attention_case(BF16, H, G, d, vd, 4, 32, n, 0.2, 20.0, tokens=4096)
    want = plain_attention(m, w, qkv)[-4:]
    for counts in ([n - 3, 1, 1, 1], [n - 2, 2]):
        got = attend(m, w, qkv, cache, 0, counts)
        assert float((got[-2:] - want[-2:]).abs().max()) < 0.03, counts
        cache.recycle([0])


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_convolutions_and_their_rings(dtype):
    """Every tap count, with and without bias and silu, in channels of a wider ring, over portions shorter than the taps."""
    from pace_b200.llm.hybrid_cache import StateSpec
    from pace_b200.ops import hybrid
    n = 60
    for taps in (1, 2, 3, 4, 7):
        for ch, off in ((48, 8), (37, 5)):
            g = torch.Generator().manual_seed(taps)
            x, tw, bias = torch.randn(n, ch, generator=g).to(dtype), torch.randn(ch, taps, generator=g), torch.randn(ch, generator=g)
            cache = manager([StateSpec((("conv", (taps + 1, ch + 2 * off)),))], dtype)
            ring = cache[0]["conv"][:, :, off: off + ch]
            for silu, b in ((True, bias), (False, None)):
                want = ref.short_conv(x.double(), tw.double(), None if b is None else b.double())
                want = ref.silu(want) if silu else want
                for row, counts in ((0, [n]), (1, [2] * 30), (0, [1, 1, 5, 1, 2, 50]), (1, [3, 57])):
                    def run(step, lo, hi):
                        out = torch.empty(hi - lo, ch + 3, dtype=dtype, device=DEV)[:, :ch]
                        torch.ops.pace_b200.causal_conv(step.handle, x[lo:hi].to(DEV), tw.t().contiguous().to(DEV),
                                                        None if b is None else b.to(DEV), ring, out, silu)
                        hybrid.conv_store(step, x[lo:hi].to(DEV), ring)
                        return out
                    got = over_portions(cache, row, counts, run)
                    torch.testing.assert_close(got, want, rtol=1e-2 if dtype == BF16 else 1e-5, atol=1e-2 if dtype == BF16 else 1e-5)
                    cache.recycle([row])
            assert bool(cache[0]["conv"][:, :, :off].isnan().all()) and bool(cache[0]["conv"][:, :, off + ch:].isnan().all())


# ---- state-space recurrence ---------------------------------------------------------------------------------------------
def ssd_run(dtype, m, w, xbc, dt, cache, row, counts):
    from pace_b200.ops import hybrid
    dev = {k: v.float().to(DEV) for k, v in w.items()}
    ring = cache[0]["conv"]

    def run(step, lo, hi):
        x = xbc[lo:hi].to(DEV)
        y = hybrid.ssd(step, x, dt[lo:hi].to(DEV), dev["conv"].t().contiguous(), dev["conv.b"], dev["dt_bias"], -dev["A_log"].double().exp().float(),
                       dev["D"], m["groups"], cache[0]["S"], ring)
        if not step.decode_only:
            hybrid.conv_store(step, x, ring)
        return y
    return over_portions(cache, row, counts, run)


def ssd_plain(dtype, m, w, xbc, dt):
    n, H, P, N, G = len(xbc), m["heads"], m["vdim"], m["state"], m["groups"]
    wd = {k: v.double() for k, v in w.items()}
    u = ref.silu(ref.short_conv(xbc.double(), wd["conv"], wd["conv.b"])).to(dtype).double()
    x, b, c = torch.split(u, [H * P, G * N, G * N], -1)
    b, c = (t.view(n, G, N).repeat_interleave(H // G, 1) for t in (b, c))
    return ref.ssd_scan(x.view(n, H, P), b, c, ref.softplus(dt.double() + wd["dt_bias"]), wd["A_log"], wd["D"]).reshape(n, -1)


SSD = [(BF16, 4, 2, 64, 64, 4), (BF16, 6, 3, 24, 16, 3), (BF16, 2, 1, 128, 128, 4), (BF16, 2, 2, 40, 136, 2), (BF16, 3, 3, 11, 7, 1),
       (BF16, 2, 1, 200, 64, 4), (FP32, 6, 2, 24, 16, 3), (FP32, 2, 1, 128, 64, 4), (FP32, 3, 1, 11, 37, 5)]


@pytest.mark.parametrize("dtype,H,G,N,P,conv", SSD)
@pytest.mark.parametrize("decay", ["weak", "mixed", "strong"])
def test_state_space_against_plain(dtype, H, G, N, P, conv, decay):
    """Decays from one in a hundred thousand per token to the whole state; chunk borders, portions, decoding, old slots."""
    from pace_b200.llm.hybrid_cache import StateSpec
    n = 330
    g = torch.Generator().manual_seed(N + P)
    m = lm.right(H, G, N, P, conv, 1)
    ch = H * P + 2 * G * N
    xbc, dt = torch.randn(n, ch, generator=g).to(dtype), torch.randn(n, H, generator=g).to(dtype)
    w = {"conv": torch.randn(ch, conv, generator=g) * 0.7, "conv.b": torch.randn(ch, generator=g) * 0.3, "D": torch.randn(H, generator=g),
         "dt_bias": torch.full((H,), {"weak": -3.0, "mixed": -1.0, "strong": 2.0}[decay]) + torch.randn(H, generator=g) * 0.3,
         "A_log": torch.full((H,), {"weak": -6.0, "mixed": 0.0, "strong": 3.0}[decay]) + torch.randn(H, generator=g)}
    want = ssd_plain(dtype, m, w, xbc, dt)
    cache = manager([StateSpec((("S", (H, N, P)), ("conv", (conv + 2, ch))))], dtype)
    scale = want.view(n, H, P).pow(2).mean(-1, keepdim=True).sqrt()
    scale = scale.clamp(min=0.2 * float(scale.mean()))
    for row, counts in ((0, [n]), (1, [129, 1, 1, 2, 3, 64, n - 200]), (0, [n - 40] + [1] * 40), (1, [63, 2, 64, 65, n - 194]), (0, [1] * 30 + [n - 30])):
        got = ssd_run(dtype, m, w, xbc, dt, cache, row, counts)
        err = float(((got - want).view(n, H, P) / scale).abs().max())
        assert err < (0.04 if dtype == BF16 else 1e-4), (counts, err)
        cache.recycle([row])


@pytest.mark.parametrize("N,P", [(64, 64), (128, 128), (200, 40)])
def test_state_space_keeps_small_additions(N, P):
    """A large state that hardly decays takes thousands of small additions; rounded to 16 bits it would not move.  Long prompts
    are cut into segments: their states are the same."""
    from pace_b200.llm.hybrid_cache import StateSpec
    n = 2600
    m = lm.right(1, 1, N, P, 1, 1)
    xbc = torch.zeros(n, P + 2 * N, dtype=BF16)
    xbc[0, :P], xbc[1:, :P] = 20.0, 0.5
    xbc[:, P], xbc[:, P + N] = 3.0, 3.0
    w = {"conv": torch.ones(P + 2 * N, 1), "conv.b": torch.zeros(P + 2 * N), "D": torch.zeros(1), "dt_bias": torch.full((1,), -5.0),
         "A_log": torch.full((1,), -9.0)}
    dt = torch.zeros(n, 1, dtype=BF16)
    want = ssd_plain(BF16, m, w, xbc, dt)
    cache = manager([StateSpec((("S", (1, N, P)), ("conv", (1, P + 2 * N))))], BF16, tokens=4096)
    for row, counts in ((0, [n]), (1, [1500, n - 1500]), (0, [n - 20] + [1] * 20)):
        got = ssd_run(BF16, m, w, xbc, dt, cache, row, counts)
        assert float(((got - want) / want.abs().clamp(min=1e-3)).abs()[-50:].max()) < 5e-3, counts
        cache.recycle([row])


# ---- delta rule -----------------------------------------------------------------------------------------------------------
def delta_run(dtype, m, w, qkv, a, b, cache, row, counts):
    from pace_b200.ops import hybrid
    dev = {k: v.float().to(DEV) for k, v in w.items()}
    ring = cache[0]["conv"]

    def run(step, lo, hi):
        x = qkv[lo:hi].to(DEV)
        o = hybrid.delta_rule(step, x, a[lo:hi].to(DEV), b[lo:hi].to(DEV), dev["conv"].t().contiguous(), dev["dt_bias"],
                              -dev["A_log"].double().exp().float(), m["kv_heads"], cache[0]["S"], ring, 1e-6, m["dim"] ** -0.5)
        if not step.decode_only:
            hybrid.conv_store(step, x, ring)
        return o
    return over_portions(cache, row, counts, run)


def delta_plain(dtype, m, w, qkv, a, b):
    n, H, G, d, vd = len(qkv), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    wd = {k: v.double() for k, v in w.items()}
    u = ref.silu(ref.short_conv(qkv.double(), wd["conv"])).to(dtype).double()
    q, k, v = torch.split(u, [G * d, G * d, H * vd], -1)
    q, k = (ref.unit(x.view(n, G, d)).repeat_interleave(H // G, 1) for x in (q, k))
    g = torch.exp(-torch.exp(wd["A_log"])[:, None] * ref.softplus(a.double() + wd["dt_bias"]).view(n, H, d))
    return ref.delta_scan(q * d ** -0.5, k, v.view(n, H, vd), g, ref.sigmoid(b.double())).reshape(n, -1)


def delta_case(dtype, H, G, d, vd, conv, n, decay, seed=0, keys="random", tokens=1024):
    from pace_b200.llm.hybrid_cache import StateSpec
    g = torch.Generator().manual_seed(seed)
    m, ch = lm.cd(H, G, d, vd, conv), 2 * G * d + H * vd
    qkv = torch.randn(n, ch, generator=g)
    if keys == "alike":                      # every key nearly the same: each write corrects all the others
        qkv[:, G * d: 2 * G * d] = qkv[:1, G * d: 2 * G * d] * 2 + qkv[:, G * d: 2 * G * d] * 0.1
    a, b = torch.randn(n, H * d, generator=g).to(dtype), (torch.randn(n, H, generator=g) * 2 + (3 if keys == "alike" else 0)).to(dtype)
    w = {"conv": torch.randn(ch, conv, generator=g) * 0.3 + (torch.arange(conv) == conv - 1) * 0.7,
         "A_log": {"weak": -4.0, "mixed": 0.0, "strong": 2.0}[decay] + torch.randn(H, generator=g),
         "dt_bias": {"weak": -3.0, "mixed": -3.0, "strong": 1.0}[decay] + torch.randn(H * d, generator=g) * (3.0 if decay == "mixed" else 0.5)}
    cache = manager([StateSpec((("S", (H, d, vd)), ("conv", (conv, ch))))], dtype, tokens=tokens)
    return m, w, qkv.to(dtype), a, b, cache


DELTA = [(BF16, 4, 2, 64, 64, 4), (BF16, 6, 2, 24, 40, 3), (BF16, 2, 2, 128, 128, 4), (BF16, 2, 1, 40, 136, 2), (BF16, 3, 3, 13, 21, 1),
         (BF16, 2, 1, 160, 72, 4), (FP32, 6, 2, 24, 40, 3), (FP32, 2, 1, 128, 64, 4), (FP32, 3, 1, 13, 37, 5)]


@pytest.mark.parametrize("dtype,H,G,d,vd,conv", DELTA)
@pytest.mark.parametrize("decay", ["weak", "mixed", "strong"])
@pytest.mark.parametrize("keys", ["random", "alike"])
def test_delta_rule_against_plain(dtype, H, G, d, vd, conv, decay, keys):
    """Decays that differ by channel, from hardly any to the whole row at once; keys that interfere; chunk borders, portions,
    decoding, old slots."""
    n = 330
    m, w, qkv, a, b, cache = delta_case(dtype, H, G, d, vd, conv, n, decay, d + vd, keys)
    want = delta_plain(dtype, m, w, qkv, a, b)
    scale = want.view(n, H, vd).pow(2).mean(-1, keepdim=True).sqrt()
    scale = scale.clamp(min=0.2 * float(scale.mean()))
    for row, counts in ((0, [n]), (1, [129, 1, 1, 2, 3, 64, n - 200]), (0, [n - 40] + [1] * 40), (1, [63, 2, 64, 17, 15, n - 161]),
                        (0, [1] * 30 + [n - 30])):
        got = delta_run(dtype, m, w, qkv, a, b, cache, row, counts)
        err = float(((got - want).view(n, H, vd) / scale).abs().max())
        assert err < (0.04 if dtype == BF16 else 2e-4), (counts, err)
        cache.recycle([row])


@pytest.mark.parametrize("d,vd", [(64, 64), (128, 128), (24, 40)])
def test_delta_rule_keeps_its_state_in_32_bits(d, vd):
    """One key written over and over with beta near 1/256 and no decay: the state creeps to the value in steps that a 16-bit
    state would not take."""
    n = 1500
    m, w, qkv, a, b, cache = delta_case(BF16, 1, 1, d, vd, 1, n, "weak", tokens=2048)
    w["conv"][:], w["A_log"][:], w["dt_bias"][:] = 1.0, -12.0, -12.0
    qkv[:] = 0
    qkv[:, 3], qkv[:, d + 3], qkv[:, 2 * d:] = 4.0, 4.0, 1.0
    a[:] = 0
    b[:] = -5.5
    want = delta_plain(BF16, m, w, qkv, a, b)
    for row, counts in ((0, [n]), (1, [700, n - 700]), (0, [n - 20] + [1] * 20)):
        got = delta_run(BF16, m, w, qkv, a, b, cache, row, counts)
        assert float(((got - want) / want.abs()).abs()[300:].max()) < 5e-3, counts
        cache.recycle([row])


# ---- norms, activations, router, experts --------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("n,part", [(96, 48), (64, 64), (40, 8), (37, 37), (33, 11), (2048, 1024), (4096, 4096), (1200, 600), (256, 1)])
def test_norms_over_parts_with_a_gate(dtype, n, part):
    from pace_b200.ops import hybrid
    T, g = 7, torch.Generator().manual_seed(n + part)
    o, z = torch.randn(T, n, generator=g).to(dtype), torch.randn(T, n + 8, generator=g).to(dtype)[:, 8:]
    w, tol = torch.randn(n, generator=g), dict(rtol=1e-2, atol=1e-2) if dtype == BF16 else dict(rtol=1e-5, atol=1e-5)
    wide = torch.zeros(T, n + 16, dtype=dtype, device=DEV)
    hybrid.part_norm_gate(o.to(DEV), w.to(DEV), z.to(DEV), part, 1e-3, gate_first=True, out=wide[:, 8:-8])
    want = ref.gated_group_norm(o.double(), z.double(), w.double(), n // part, 1e-3)
    torch.testing.assert_close(wide[:, 8:-8].double().cpu(), want, **tol)
    assert float(wide[:, :8].abs().max()) == 0 and float(wide[:, -8:].abs().max()) == 0
    w = w[:part]
    got = hybrid.part_norm_gate(o.to(DEV), w.to(DEV), z.to(DEV), part, 1e-3)
    want = (ref.rms(o.double().view(T, -1, part), 1e-3) * w.double()).view(T, n) * ref.sigmoid(z.double())
    torch.testing.assert_close(got.double().cpu(), want, **tol)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width", [64, 37, 2200])
def test_two_norms_of_one_stream(dtype, width):
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(width)
    step = Step([5], [0], [0], torch.tensor([3, 0, 8, 8, 1]), 9, DEV)
    e, y = torch.randn(9, width, generator=g).to(dtype), torch.randn(5, width, generator=g).to(dtype)
    we, w1, w2, bias = (torch.randn(width, generator=g) for _ in range(4))
    x, eps = torch.empty(5, width, device=DEV), 1e-2
    h1, h2 = hybrid.residual_norm(step, x, embed=e.to(DEV), embed_norm=we.to(DEV), w_next=w1.to(DEV), w_next2=w2.to(DEV), restart=True,
                                  eps=eps, weight_offset=1.0)
    want = ref.rms(e.double()[[3, 0, 8, 8, 1]], eps) * (1 + we.double())
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == BF16 else dict(rtol=1e-5, atol=1e-5)
    for _ in range(2):
        torch.testing.assert_close(x.double().cpu(), want, rtol=2e-6, atol=2e-6)
        torch.testing.assert_close(h1.double().cpu(), ref.rms(want, eps) * (1 + w1.double()), **tol)
        torch.testing.assert_close(h2.double().cpu(), ref.rms(want, eps) * (1 + w2.double()), **tol)
        h1, h2 = hybrid.residual_norm(step, x, y.to(DEV), bias=bias.to(DEV), y_mul=0.3, w_next=w1.to(DEV), w_next2=w2.to(DEV), eps=eps,
                                      weight_offset=1.0)
        want = want + 0.3 * (y.double() + bias.double())


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_ungated_activations_and_caps(dtype):
    from pace_b200 import _C
    from pace_b200.ops import hybrid
    for n in (40, 37):
        x = (torch.randn(6, n, generator=torch.Generator().manual_seed(n)) * 4).to(dtype)
        for act, f in ((_C.ACT_SILU, ref.silu), (_C.ACT_GELU_ERF, ref.gelu_erf)):
            out = torch.zeros(6, n + 16, dtype=dtype, device=DEV)
            hybrid.activate(x.to(DEV), act, out[:, 8:-8])
            torch.testing.assert_close(out[:, 8:-8].double().cpu(), f(x.double()), rtol=1e-2 if dtype == BF16 else 1e-5, atol=2e-6)
            assert float(out[:, :8].abs().max()) == 0 and float(out[:, -8:].abs().max()) == 0
    z = torch.randn(1000, generator=torch.Generator().manual_seed(1)) * 100
    torch.testing.assert_close(hybrid.soft_cap_(z.to(DEV), 30.0).double().cpu(), ref.soft_cap(z.double(), 30.0), rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("T,width,ff,experts,identity,top,shared", [
    (1, 64, 64, 4, 0, 1, 8), (9, 72, 40, 6, 2, 3, 16), (700, 96, 136, 5, 1, 2, 40), (300, 136, 264, 3, 3, 6, 0), (64, 37, 19, 7, 5, 4, 9),
    (33, 512, 256, 64, 0, 8, 0), (2500, 64, 32, 40, 8, 6, 24), (5, 16, 8, 1, 1, 1, 0)])
def test_softmax_router_with_identity_and_shared_experts(dtype, T, width, ff, experts, identity, top, shared):
    """Scores over all outputs, choice with the correction, weights that sum to the scale; identity experts hand their input on;
    the shared expert's rows are added on the way; experts without a token and with all of them."""
    from pace_b200 import _C
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(T)
    n = experts + identity
    h = torch.randn(T, width, generator=g).to(dtype)
    w = {"router": torch.randn(n, width, generator=g) / math.sqrt(width), "correction": torch.randn(n, generator=g) * 0.05}
    if experts > 4:
        w["correction"][1], w["correction"][3] = -5.0, 5.0
    for e in [f"e{i}" for i in range(experts)] + (["shared"] if shared else []):
        f = shared if e == "shared" else ff
        w[e + ".up"], w[e + ".down"] = torch.randn(f, width, generator=g) / math.sqrt(width), torch.randn(width, f, generator=g) / math.sqrt(f)
    w = {k: v.bfloat16() for k, v in w.items()}
    wd = {k: v.double() for k, v in w.items()}
    dev = {k: v.to(DEV, FP32 if k == "correction" else dtype) for k, v in w.items()}
    hd = h.to(DEV)
    routed = hybrid.moe_route(hd, dev["router"], dev["correction"], top, softmax=True, weight_scale=1.6, identity=identity)
    chosen, weight = ref.route(h.double(), wd["router"], wd["correction"], top, 1.6)
    order, mine = chosen.sort(-1), routed.slot_expert.cpu().long().sort(-1)
    assert torch.equal(mine.values, order.values)
    torch.testing.assert_close(routed.slot_weight.cpu().double().gather(1, mine.indices), weight.gather(1, order.indices), rtol=1e-5, atol=1e-6)
    assert torch.equal(routed.count.cpu().long(), torch.bincount(chosen.reshape(-1), minlength=n)[:experts])
    up, down = torch.stack([dev[f"e{e}.up"] for e in range(experts)]), torch.stack([dev[f"e{e}.down"] for e in range(experts)])
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for _ in range(2):                                       # (again over results that are there already)
        hybrid.moe_experts(hd, routed, up, down, _C.ACT_GELU_ERF, status, gated=False)
    y = None
    if shared:
        y = hybrid.activate(hd @ dev["shared.up"].t(), _C.ACT_GELU_ERF) @ dev["shared.down"].t()
    step = Step([T], [0], [0], torch.zeros(T, dtype=torch.long), 1, DEV)
    x = torch.ones(T, width, device=DEV)
    hybrid.residual_norm(step, x, y, routed=routed, y_mul=0.5)
    m = {"router": {"experts": experts, "identity": identity, "top": top, "scale": 1.6}, **({"shared": {"ff": shared}} if shared else {})}
    want = ref.moe_mlp(h.double(), m, wd, "")
    err = float(((x.double().cpu() - 1) / 0.5 - want).abs().max() / want.pow(2).mean().sqrt())
    assert err < (0.06 if dtype == BF16 else 1e-5) and int(status) == 0


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("kind,mixer,mlp", [
    (lm.P, lm.par(lm.left(6, 2, 20, 28, 3, 8), lm.right(4, 2, 24, 16, 4, 2)), None),
    (lm.P, lm.par(lm.left(5, 5, 130, 33, 4, 2), lm.right(3, 1, 9, 21, 2, 7), 0.0, 1.0), None),
    (lm.P, lm.par(lm.left(34, 1, 8, 16, 2, 8, scale=-0.7), lm.right(8, 4, 16, 8, 5, 1), 1.0, 0.0), lm.dense(40)),
    (lm.P, lm.par(lm.left(2, 2, 16, 16, 4, 16, softcap=0.3), lm.right(2, 1, 16, 16, 4, 2)), lm.moe(24, 4, 2, 2, 16)),
    (lm.D, lm.cd(4, 2, 24, 40, 3), None), (lm.D, lm.cd(5, 5, 9, 33, 4), lm.dense(21)), (lm.D, lm.cd(2, 1, 64, 64, 1), lm.moe(24, 6, 2))])
def test_one_layer_models(kind, mixer, mlp, dtype):
    cfg = lm.config([lm.layer(kind, mixer, mlp)], 48)
    model, w = build(cfg, dtype, 5)
    toks = prompt(cfg, 110, 1)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    for sizes in ([110], [2, 3, 64, 5], [70, 1]):
        slot = b.open()
        assert lm.error(feed(b, slot, toks, sizes), want) < TOL[dtype], sizes
        b.close(slot)
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    cfg = lm.CONFIGS[name]
    model, w = build(cfg, dtype)
    toks = prompt(cfg, 220, 2)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    whole = None
    for sizes in ([220], [1], [2], [7, 64, 2, 33], [200, 1], [64], [63, 2, 1], [3, 150, 2]):
        slot = b.open()
        got = feed(b, slot, toks, sizes)
        b.close(slot)
        assert lm.error(got, want) < TOL[dtype], sizes
        whole = got if whole is None else whole
        assert lm.error(got, whole) < TOL[dtype], sizes
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_unequal_requests_in_one_batch(dtype):
    """Prompts, portions and decoded tokens of several requests share steps; slots and pages go round: the pool holds
    fewer tokens than all requests together, rows are freed and taken in another order."""
    cfg = lm.CONFIGS["mixed"]
    model, w = build(cfg, dtype, 7)
    lens = [140, 9, 75, 66, 1, 130, 64, 20, 200]
    toks = [prompt(cfg, n, 20 + i) for i, n in enumerate(lens)]
    want = [ref.run(cfg, w, t) for t in toks]
    b = batcher(model, slots=3, pool_tokens=64 * 8, max_len=64 * 4)
    for s in b.manager.states:
        for x in s.arrays.values():
            x.fill_(float("nan"))
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
        assert lm.error(torch.cat(got[i]), want[i]) < TOL[dtype], i
    bits, free = b.pool.query()
    assert bits == 0 and free == b.pool.n_pages


def test_long_decoding_keeps_its_precision():
    cfg = lm.config([lm.layer(lm.P, lm.par(lm.left(4, 2, 16, 16, 3, 8), lm.right(2, 1, 16, 16, 3, 2)), lm.dense(24)),
                     lm.layer(lm.D, lm.cd(2, 1, 16, 24, 4), lm.moe(16, 4, 2, 1, 8))], 32)
    model, w = build(cfg, FP32, 9)
    toks = prompt(cfg, 700, 3)
    want = ref.run(cfg, w, toks)
    got = feed(batcher(model, slots=1), 0, toks, [5, 1])
    assert lm.error(got[-100:], want[-100:]) < 1e-4


def test_a_step_in_which_nothing_is_wanted():
    model, w = build(lm.CONFIGS["mixed"], BF16, 3)
    b = batcher(model)
    assert b.step({b.open(): prompt(lm.CONFIGS["mixed"], 5, 1)}, {0: []}).shape == (0, 67)


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
    cfg = lm.CONFIGS["mixed"]
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
    # device-resident loop: one recorded step per token, across a page border
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
    cfg = lm.CONFIGS["wide"]
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
    cfg = lm.config([lm.layer(lm.P, lm.par(lm.left(2, 1, 16, 16, 3, 8), lm.right(2, 1, 16, 16, 4, 2)), lm.dense(24)),
                     lm.layer(lm.D, lm.cd(2, 1, 16, 16, 4), lm.moe(16, 4, 2, 1))], 32)
    model, w = build(cfg, FP32, 13)
    p = prompt(cfg, 66, 60)
    got = Generator(model).generate(p[None], SamplingConfig(max_new_tokens=4, num_beams=3)).output_token_ids[0, 66:].tolist()
    beams = [([], 0.0)]
    for _ in range(4):
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
    cfg = lm.CONFIGS["mixed"]
    w = lm.weights(cfg, 15, decided=dtype == BF16)
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
    assert lm.error(out(0), wa[[0, 95]]) < TOL[dtype] and not (tmp_path / "1.f32").exists()
    assert lm.error(out(2), torch.stack([wc[11], wc[5], wa[96]])) < TOL[dtype]
    assert lm.error(out(3), wc[[11]]) < TOL[dtype]
