"""The Gekupel model on the GPU against the plain implementation: every mechanism alone, then whole models, prompts,
portions, decoding, batches, reuse of pages and slots, and generation through the framework's loops."""
import json
import math
import os
import subprocess

import pytest
import torch

import gekupel_models as gk
from oracle import gekupel_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF16, FP32 = torch.bfloat16, torch.float32
TOL = {BF16: 0.06, FP32: 1e-4}
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))


def build(cfg, dtype, seed=0):
    """bf16 models get corrections that settle the choice of experts: rounding then cannot flip one."""
    from pace_b200.llm.registry import build_model
    w = gk.weights(cfg, seed, decided=dtype == BF16)
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


# ---- attention with a span, a distance bias and a sink --------------------------------------------------------------
def span_case(dtype, heads, kv, dim, vdim, n, seed=0, rows=2, tokens=1024):
    from pace_b200.llm.hybrid_cache import HybridCacheManager, KVSpec
    g = torch.Generator().manual_seed(seed)
    qkv = torch.randn(n, heads * dim + kv * (dim + vdim), generator=g).to(dtype)
    return qkv, HybridCacheManager([KVSpec(kv, dim, vdim)], rows, rows * tokens, tokens, dtype, DEV)


def attend(qkv, cache, row, counts, heads, dim, vdim, scale, eps=1e-6, **kw):
    from pace_b200.ops import hybrid
    out, at = [], 0
    kw = {k: v.to(DEV) if isinstance(v, torch.Tensor) else v for k, v in kw.items()}
    for n in counts:
        c = [0] * cache.batch
        c[row] = n
        step = cache.step(c, torch.zeros(n, dtype=torch.long), 1)
        cache.begin_step(step)
        out.append(hybrid.span_attention(step, cache[0], qkv[at: at + n].to(DEV), heads, dim, vdim, scale, eps, **kw).cpu())
        at += n
    cache.pool.check_status()
    return torch.cat(out).double().view(-1, heads, vdim)


def plain_attention(qkv, heads, kv, dim, vdim, scale, eps=1e-6, window=None, chunk=None, slopes=None, sinks=None):
    """From projection rows, with queries and keys rounded as the products take them."""
    n, dt, x = len(qkv), qkv.dtype, qkv.double()
    q = ref.rms_norm(x[:, : heads * dim].view(n, heads, dim), eps).to(dt).double()
    k = ref.rms_norm(x[:, heads * dim: (heads + kv) * dim].view(n, kv, dim), eps).to(dt).double()
    v = x[:, (heads + kv) * dim:].view(n, kv, vdim)
    seen = ref.window_mask(n, window) if window else ref.chunk_mask(n, chunk or n)
    dist = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).double()
    out = []
    for h in range(heads):
        s = q[:, h] @ k[:, h // (heads // kv)].T * scale
        if slopes is not None:
            s = s - float(slopes[h]) * dist
        out.append(ref.masked_softmax(s, seen, None if sinks is None else sinks[h].double()) @ v[:, h // (heads // kv)])
    return torch.stack(out, 1)


SHAPES = [(BF16, 10, 2, 88, 104), (BF16, 8, 4, 33, 64), (BF16, 2, 2, 144, 40), (BF16, 12, 1, 64, 64), (BF16, 40, 2, 128, 128),
          (FP32, 6, 2, 40, 24), (FP32, 3, 3, 128, 128)]


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim", SHAPES)
@pytest.mark.parametrize("rule", ["window", "chunk", "all"])
def test_span_attention_against_plain(dtype, heads, kv, dim, vdim, rule):
    """Every position of a prompt, of portions and of decoding, with bias and sinks, spans below and above a tile."""
    n = 330
    g = torch.Generator().manual_seed(n + heads)
    slopes, sinks = torch.rand(heads, generator=g) * 0.05, torch.randn(heads, generator=g) * 2
    for size in {"window": (1, 40, 64, 200), "chunk": (1, 50, 64, 210), "all": (None,)}[rule]:
        kw = dict(slopes=slopes, sinks=sinks, **({} if size is None else {rule: size}))
        qkv, cache = span_case(dtype, heads, kv, dim, vdim, n, size or 0)
        want = plain_attention(qkv, heads, kv, dim, vdim, 0.3, **kw)
        for row, counts in ((0, [n]), (1, [129, 1, 1, 2, 3, 64, n - 200]), (0, [n - 40] + [1] * 40)):
            got = attend(qkv, cache, row, counts, heads, dim, vdim, 0.3, **kw)
            assert float((got - want).abs().max()) < (0.025 if dtype == BF16 else 2e-5), (size, counts)
            cache.recycle([row])


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim", SHAPES)
def test_one_key_inside_or_outside_a_span(dtype, heads, kv, dim, vdim):
    """One key stands out for one query: inside the span the output is that key's value, one place further out it is not;
    across page borders, in prompts, portions and decoding."""
    n = 300
    cases = [({"window": s}, t, t - s + 1 - d, d == 0) for s in (1, 37, 64, 129) for t in (140, 192, 255) for d in (0, 1)] + \
            [({"chunk": s}, t, t // s * s - d, d == 0) for s in (37, 64, 130) for t in (131, 191, 192, 299) for d in (0, 1)] + \
            [({}, t, j, True) for t, j in ((299, 0), (64, 63), (128, 64), (127, 127))] + [({}, 127, 128, False)]
    for rule, t, j, inside in cases:
        qkv, cache = span_case(dtype, heads, kv, dim, vdim, n, seed=t + j)
        u = torch.randn(dim, generator=torch.Generator().manual_seed(j))
        qkv[t, : heads * dim] = u.repeat(heads).to(dtype)
        qkv[j, heads * dim: (heads + kv) * dim] = u.repeat(kv).to(dtype)
        v = qkv[j, (heads + kv) * dim:].double().view(kv, vdim).repeat_interleave(heads // kv, 0)
        for row, counts in ((0, [n]), (1, [t, 1] + [n - t - 1] * (t < n - 1)), (0, [50, 2, t - 53, 3, n - t - 2] if t < n - 2 else [n - 2, 2])):
            got = attend(qkv, cache, row, counts, heads, dim, vdim, 3.0, **rule)[t]
            gap = float((got - v).abs().max())
            assert (gap < 0.05) == inside, (rule, t, j, counts, gap)
            cache.recycle([row])


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_sink_is_one_term_of_the_denominator(dtype):
    """Equal scores: n visible keys weigh 1 / (n + exp(sink)) each, whatever the scale and the bias of a lone head; a sink
    far above all scores leaves nothing, one far below changes nothing."""
    heads, kv, dim, vdim, n = 4, 2, 16, 16, 200
    qkv, cache = span_case(dtype, heads, kv, dim, vdim, n)
    qkv[:, : heads * dim] = 1
    qkv[:, heads * dim: (heads + kv) * dim] = 0
    qkv[:, heads * dim: (heads + kv) * dim: 2] = 1
    qkv[:, heads * dim + 1: (heads + kv) * dim: 2] = -1         # orthogonal to the query: every score is 0
    qkv[:, (heads + kv) * dim:] = 1
    sinks = torch.tensor([0.0, math.log(50.0), 60.0, -60.0])
    for counts in ([n], [n - 1, 1], [100, 2, 98]):
        got = attend(qkv, cache, 0, counts, heads, dim, vdim, 5.0, sinks=sinks, window=64)[n - 1, :, 0]
        want = torch.tensor([64 / 65, 64 / 114, 0.0, 1.0], dtype=torch.float64)
        assert float((got - want).abs().max()) < (4e-3 if dtype == BF16 else 1e-6)
        cache.recycle([0])


def test_long_contexts_split_over_a_cluster():
    """One decoded token over thousands of keys: the keys of a tile are shared out over the blocks of a cluster."""
    heads, kv, dim, vdim, n = 8, 1, 128, 128, 4000
    qkv, cache = span_case(BF16, heads, kv, dim, vdim, n, tokens=4096, rows=1)
    slopes, sinks = torch.linspace(0.0001, 0.01, heads), torch.linspace(-3, 6, heads)
    for kw in ({}, {"window": 3000}, {"chunk": 1900}):
        want = plain_attention(qkv[-n:], heads, kv, dim, vdim, 0.2, slopes=slopes, sinks=sinks, **kw)[-4:]
        for counts in ([n - 3, 1, 1, 1], [n - 2, 2]):
            got = attend(qkv, cache, 0, counts, heads, dim, vdim, 0.2, slopes=slopes, sinks=sinks, **kw)
            assert float((got[-2:] - want[-2:]).abs().max()) < 0.02, (kw, counts)
            cache.recycle([0])


@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 1, 128, 128), (12, 1, 64, 64), (2, 2, 96, 80)])
def test_softmax_weights_are_not_rounded_to_bf16(heads, kv, dim, vdim):
    """Every key but the first has a weight half way between two bf16 values: rounded, all of them would be off in the
    same direction by 2^-8 of themselves, and half of the outputs would land on another bf16 value."""
    p, n = 0.5 + 2.0 ** -9 * 0.98, 500
    for counts in ([n], [n - 1, 1], [n - 3, 3]):
        qkv, cache = span_case(BF16, heads, kv, dim, vdim, n, 11)
        v = (1.0 + torch.rand(n, kv * vdim, generator=torch.Generator().manual_seed(1))).to(BF16)
        qkv[:, : (heads + kv) * dim] = 0
        qkv[:, : heads * dim: dim] = 1
        qkv[0, heads * dim: (heads + kv) * dim: dim] = 1
        qkv[1:, heads * dim + 1: (heads + kv) * dim: dim] = 1
        qkv[:, (heads + kv) * dim:] = v
        got = attend(qkv, cache, 0, counts, heads, dim, vdim, -math.log(p) / dim, eps=0.0)[n - counts[-1]:]
        w = torch.cat([torch.ones(1, dtype=torch.float64), torch.full((n - 1,), p, dtype=torch.float64)])
        same = []
        for i in range(0, counts[-1], 97):
            t = n - counts[-1] + i
            if t >= 300:
                want = (w[: t + 1] @ v[: t + 1].double()) / w[: t + 1].sum()
                same.append((got[i] == want.view(kv, vdim).repeat_interleave(heads // kv, 0).to(BF16).double()).double().mean())
        assert float(min(same)) > 0.9, (counts, same)


# ---- latent attention ------------------------------------------------------------------------------------------------
LATENTS = [(BF16, 4, 64, 32, 48, 40, 64), (BF16, 6, 128, 64, 128, 96, 256), (BF16, 20, 24, 8, 16, 24, 32), (BF16, 3, 13, 6, 11, 9, 21),
           (BF16, 2, 160, 40, 136, 32, 512), (FP32, 4, 24, 8, 40, 20, 48), (FP32, 3, 13, 6, 11, 9, 21)]


def latent_case(dtype, heads, dim, rot, vdim, q_rank, rank, n, window, scaling, seed=0, rows=2, tokens=512):
    from pace_b200.llm.hybrid_cache import HybridCacheManager, LatentSpec
    g = torch.Generator().manual_seed(seed)
    m = gk.lat(heads, dim, rot, vdim, q_rank, rank, window, 1e4, scaling, scale=0.5 / math.sqrt(dim + rot))
    w = {"dq.norm": 1 + torch.rand(q_rank, generator=g), "dkv.norm": 1 + torch.rand(rank, generator=g),
         "uq": torch.randn(heads * (dim + rot), q_rank, generator=g) / math.sqrt(q_rank),
         "uk": torch.randn(heads * dim, rank, generator=g) / math.sqrt(rank),
         "uv": torch.randn(heads * vdim, rank, generator=g) / math.sqrt(rank),
         "sink": torch.randn(heads, generator=g) * 2}
    w = {k: v.bfloat16() for k, v in w.items()}
    down = torch.randn(n, q_rank + rank + rot, generator=g).to(dtype)
    return m, w, down, HybridCacheManager([LatentSpec(rank, rot)], rows, rows * tokens, tokens, dtype, DEV)


def latents(m, w, down, cache, row, counts, sink, eps):
    from pace_b200.ops import RotaryEmbedding, hybrid
    y = m["rot"].get("scaling")
    kind = {"rope_type": "precise"} if y is None else {"rope_type": "yarn", "factor": y["factor"], "beta_fast": y["fast"],
                                                       "original_max_position_embeddings": y["original"], "beta_slow": y["slow"]}
    tables = RotaryEmbedding(kind, m["rot_dim"], 512, m["rot"]["base"], is_neox_style=False).device_tables(DEV)
    dt, out, at = down.dtype, [], 0
    uq, ukv = w["uq"].to(DEV, dt), torch.cat([w["uk"], w["uv"]]).to(DEV, dt)
    for n in counts:
        c = [0] * cache.batch
        c[row] = n
        step = cache.step(c, torch.zeros(n, dtype=torch.long), 1)
        cache.begin_step(step)
        out.append(hybrid.latent_attention(step, cache[0], down[at: at + n].to(DEV), w["dq.norm"].to(DEV).float(),
                                           w["dkv.norm"].to(DEV).float(), uq, ukv, m["heads"], m["dim"], m["rot_dim"], m["vdim"],
                                           m["scale"], eps, tables, window=m["mask"]["size"],
                                           sinks=w["sink"].to(DEV).float() if sink else None).cpu())
        at += n
    cache.pool.check_status()
    return torch.cat(out).double()


def plain_latents(m, w, down, sink, eps):
    """``ref.latent_attention`` from given down projections: they pass through identities."""
    x = down.double()
    R, r = m["kv_rank"], m["rot_dim"]
    w = {k: v.double() for k, v in w.items()}
    eye = torch.eye(x.shape[1], dtype=torch.float64)
    w.update(dq=eye[: m["q_rank"]], dkv=eye[m["q_rank"]: m["q_rank"] + R + r],
             o=torch.eye(m["heads"] * m["vdim"], dtype=torch.float64))
    return ref.latent_attention(x, m, w, "", eps, sink)


@pytest.mark.parametrize("dtype,heads,dim,rot,vdim,q_rank,rank", LATENTS)
@pytest.mark.parametrize("sink,scaling", [(False, None), (True, gk.yarn(4.0, 300, 16.0, 2.0))])
def test_latent_attention_against_plain(dtype, heads, dim, rot, vdim, q_rank, rank, sink, scaling):
    n = 290
    for window in (1, 50, 64, 170):
        m, w, down, cache = latent_case(dtype, heads, dim, rot, vdim, q_rank, rank, n, window, scaling, seed=window)
        want = plain_latents(m, w, down, sink, 1e-3)
        for row, counts in ((0, [n]), (1, [129, 1, 2, 3, 64, n - 199]), (0, [n - 40] + [1] * 40), (1, [3, 200, 1, 86])):
            got = latents(m, w, down, cache, row, counts, sink, 1e-3)
            err = float((got - want).abs().max() / want.pow(2).mean().sqrt())
            assert err < (0.1 if dtype == BF16 else 1e-4), (window, counts, err)
            cache.recycle([row])


@pytest.mark.parametrize("dtype,heads,dim,rot,vdim,q_rank,rank", [(BF16, 4, 64, 16, 48, 64, 64), (BF16, 2, 32, 8, 24, 32, 32),
                                                                 (FP32, 3, 16, 8, 20, 16, 16)])
def test_one_latent_inside_or_outside_a_window(dtype, heads, dim, rot, vdim, q_rank, rank):
    """Query and key projections are one orthogonal map, so a query sees the key with its own latent: just inside the window
    the output is that key's value, just outside it is not."""
    n = 290
    for window in (1, 37, 64, 130):
        for t in (140, 192, 255):
            for d in (0, 1):
                m, w, down, cache = latent_case(dtype, heads, dim, rot, vdim, q_rank, rank, n, window, None, seed=t)
                m["scale"] = 0.5
                ortho = torch.linalg.qr(torch.randn(dim, rank, generator=torch.Generator().manual_seed(3)).double())[0]
                up = torch.zeros(heads, dim + rot, rank, dtype=torch.float64)
                up[:, :dim] = ortho
                w["uq"], w["uk"] = up.view(-1, rank).bfloat16(), ortho.repeat(heads, 1).bfloat16()
                w["dq.norm"].fill_(2.0)
                j = t - window + 1 - d
                down[j, q_rank: q_rank + rank] = down[t, :q_rank]
                want = plain_latents(m, w, down, False, 1e-6)[t]
                c = ref.rms_norm(down[j, q_rank: q_rank + rank].double(), 1e-6, w["dkv.norm"].double())
                value = w["uv"].double() @ c
                for row, counts in ((0, [n]), (1, [t, 1, n - t - 1]), (0, [50, 2, t - 53, 3, n - t - 2])):
                    got = latents(m, w, down, cache, row, counts, False, 1e-6)[t]
                    scale = float(value.pow(2).mean().sqrt())
                    # (outside, many keys compete: the rounding of sharp scores is amplified)
                    assert float((got - want).abs().max()) / scale < 0.1 or d == 1
                    assert (float((got - value).pow(2).mean().sqrt()) / scale < 0.25) == (d == 0), (window, t, d, counts)
                    cache.recycle([row])


# ---- residual stream, feed-forwards -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("width", [64, 37, 2200])
def test_residual_without_a_norm_in_front(dtype, width):
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(width)
    toks = torch.tensor([3, 0, 8, 8, 1])
    step = Step([5], [0], [0], toks, 9, DEV)
    e, y = torch.randn(9, width, generator=g).to(dtype), torch.randn(5, width, generator=g).to(dtype)
    w = torch.randn(width, generator=g)
    x = torch.empty(5, width, device=DEV)
    h = hybrid.residual_norm(step, x, embed=e.to(DEV), restart=True, embed_scale=3.7, plain=True)
    want = e.double()[toks] * 3.7
    torch.testing.assert_close(x.double().cpu(), want, rtol=1e-6, atol=1e-6)
    assert torch.equal(h.cpu(), x.to(dtype).cpu())
    h = hybrid.residual_norm(step, x, y.to(DEV), w.to(DEV), eps=1e-2, plain=True)
    torch.testing.assert_close(x.double().cpu(), want + ref.rms_norm(y.double(), 1e-2, w.double()), rtol=2e-6, atol=2e-6)
    assert torch.equal(h.cpu(), x.to(dtype).cpu())


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_gated_activations(dtype):
    from pace_b200 import _C
    from pace_b200.ops import hybrid
    for n in (40, 37):
        x = (torch.randn(6, 2 * n, generator=torch.Generator().manual_seed(n)) * 4).to(dtype)
        for act, f in ((_C.ACT_SILU, ref.silu), (_C.ACT_GELU_TANH, ref.gelu_tanh)):
            got = hybrid.glu(x.to(DEV), act).double().cpu()
            torch.testing.assert_close(got, f(x[:, :n].double()) * x[:, n:].double(), rtol=1e-2 if dtype == BF16 else 1e-5, atol=1e-5)


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("T,width,ff,experts,top", [(1, 64, 64, 4, 1), (9, 72, 40, 6, 3), (700, 96, 136, 5, 2), (300, 136, 264, 3, 3),
                                                    (64, 37, 19, 7, 4), (33, 512, 256, 64, 8), (40, 200, 72, 9, 9), (2500, 64, 32, 40, 6)])
def test_mixture_of_experts(dtype, T, width, ff, experts, top):
    """Routing (choice by corrected score, weight without the correction) and experts with any number of tokens, none
    included, against the plain form; the residual takes their weighted sum."""
    from pace_b200 import _C
    from pace_b200.llm.step import Step
    from pace_b200.ops import hybrid
    g = torch.Generator().manual_seed(T)
    h = torch.randn(T, width, generator=g).to(dtype)
    w = {"router": torch.randn(experts, width, generator=g) / math.sqrt(width), "correction": torch.randn(experts, generator=g) * 0.3}
    if experts > 4:
        w["correction"][1] = -5.0                          # an expert without a token
        w["correction"][3] = 5.0                           # one that everybody takes
    for e in range(experts):
        w.update({f"e{e}.gate": torch.randn(ff, width, generator=g) / math.sqrt(width),
                  f"e{e}.up": torch.randn(ff, width, generator=g) / math.sqrt(width),
                  f"e{e}.down": torch.randn(width, ff, generator=g) / math.sqrt(ff)})
    w = {k: v.bfloat16() for k, v in w.items()}
    wd = {k: v.double() for k, v in w.items()}
    dev = {k: v.to(DEV, FP32 if k == "correction" else dtype) for k, v in w.items()}
    routed = hybrid.moe_route(h.to(DEV), dev["router"], dev["correction"], top)
    chosen, weight = ref.route(h.double(), wd["router"], wd["correction"], top)
    order = chosen.sort(-1)
    mine = routed.slot_expert.cpu().long().sort(-1)
    assert torch.equal(mine.values, order.values)
    torch.testing.assert_close(routed.slot_weight.cpu().double().gather(1, mine.indices), weight.gather(1, order.indices), rtol=1e-5, atol=1e-6)
    counts = torch.bincount(chosen.reshape(-1), minlength=experts)
    assert torch.equal(routed.count.cpu().long(), counts)
    gate_up = torch.stack([torch.cat([dev[f"e{e}.gate"], dev[f"e{e}.up"]]) for e in range(experts)])
    down = torch.stack([dev[f"e{e}.down"] for e in range(experts)])
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for _ in range(2):                                       # (again over results that are there already)
        hybrid.moe_experts(h.to(DEV), routed, gate_up, down, _C.ACT_SILU, status)
    step = Step([T], [0], [0], torch.zeros(T, dtype=torch.long), 1, DEV)
    x = torch.zeros(T, width, device=DEV)
    hybrid.residual_norm(step, x, routed=routed)
    want = ref.moe_mlp(h.double(), {"router": {"experts": experts, "top": top}}, wd, "")
    err = float((x.double().cpu() - want).abs().max() / want.pow(2).mean().sqrt())
    assert err < (0.05 if dtype == BF16 else 1e-5) and int(status) == 0
    wn = torch.randn(width, generator=g)
    x.fill_(1.0)
    hybrid.residual_norm(step, x, w_post=wn.to(DEV), eps=1e-2, routed=routed)
    want = 1.0 + ref.rms_norm(want, 1e-2, wn.double())
    assert float((x.double().cpu() - want).abs().max()) < (0.1 if dtype == BF16 else 1e-4)


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("kind,mixer,mlp", [
    (gk.A, gk.att(6, 2, 20, 28, 11), None), (gk.A, gk.att(5, 5, 130, 33, 64), None), (gk.A, gk.att(34, 1, 8, 16, 40, scale=0.7), None),
    (gk.L1, gk.lat(3, 40, 16, 24, 20, 64, 30), None), (gk.L1, gk.lat(7, 8, 2, 8, 8, 16, 70, base=7.0), None),
    (gk.L2, gk.lat(3, 40, 16, 24, 20, 64, 30, scaling=gk.yarn()), None), (gk.L2, gk.lat(2, 24, 32, 40, 30, 32, 64), None),
    (gk.A, gk.att(2, 2, 16, 16, 20), gk.dense(21)), (gk.L1, gk.lat(2, 16, 8, 16, 16, 16, 9), gk.moe(24, 6, 2))])
def test_one_layer_models(kind, mixer, mlp, dtype):
    cfg = gk.config([gk.layer(kind, mixer, mlp)], 48)
    model, w = build(cfg, dtype, 5)
    toks = prompt(cfg, 110, 1)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    for sizes in ([110], [2, 3, 64, 5], [70, 1]):
        slot = b.open()
        assert gk.error(feed(b, slot, toks, sizes), want) < TOL[dtype], sizes
        b.close(slot)
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
@pytest.mark.parametrize("name", list(gk.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype):
    cfg = gk.CONFIGS[name]
    model, w = build(cfg, dtype)
    toks = prompt(cfg, 220, 2)
    want = ref.run(cfg, w, toks)
    b = batcher(model)
    whole = None
    for sizes in ([220], [1], [2], [7, 64, 2, 33], [200, 1], [64], [63, 2, 1], [3, 150, 2]):
        slot = b.open()
        got = feed(b, slot, toks, sizes)
        b.close(slot)
        assert gk.error(got, want) < TOL[dtype], sizes
        whole = got if whole is None else whole
        assert gk.error(got, whole) < TOL[dtype], sizes
    b.pool.check_status()


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_unequal_requests_in_one_batch(dtype):
    """Prompts, portions and decoded tokens of several requests share steps; slots and pages go round: the pool holds
    fewer tokens than all requests together, rows are freed and taken in another order."""
    cfg = gk.CONFIGS["mixed"]
    model, w = build(cfg, dtype, 7)
    lens = [140, 9, 75, 66, 1, 130, 64, 20, 200]
    toks = [prompt(cfg, n, 20 + i) for i, n in enumerate(lens)]
    want = [ref.run(cfg, w, t) for t in toks]
    b = batcher(model, slots=3, pool_tokens=64 * 8, max_len=64 * 4)
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
        assert gk.error(torch.cat(got[i]), want[i]) < TOL[dtype], i
    bits, free = b.pool.query()
    assert bits == 0 and free == b.pool.n_pages


def test_long_decoding_keeps_its_precision():
    cfg = gk.config([gk.layer(gk.A, gk.att(4, 2, 16, 16, 150), gk.dense(24)), gk.layer(gk.L1, gk.lat(2, 16, 8, 16, 16, 24, 90), gk.moe(16, 4, 2)),
                     gk.layer(gk.L2, gk.lat(2, 16, 8, 16, 16, 24, 300, scaling=gk.yarn(2.0, 128)))], 32)
    model, w = build(cfg, FP32, 9)
    toks = prompt(cfg, 700, 3)
    want = ref.run(cfg, w, toks)
    got = feed(batcher(model, slots=1), 0, toks, [5, 1])
    assert gk.error(got[-100:], want[-100:]) < 1e-4


def test_a_layer_with_borrowed_weights_has_its_own_cache():
    """Two runs of one layer's weights: the second run's keys are not the first one's."""
    one = gk.layer(gk.L1, gk.lat(2, 16, 8, 16, 16, 24, 40), gk.dense(24))
    cfg = gk.config([one, {**one, "weights_of": 0}, {**one, "weights_of": 0}], 32)
    model, w = build(cfg, FP32, 3)
    assert sum(p.numel() for p in model.model.layers.parameters()) == sum(p.numel() for p in model.model.layers[0].parameters())
    toks = prompt(cfg, 90, 4)
    assert gk.error(feed(batcher(model), 0, toks, [50, 1]), ref.run(cfg, w, toks)) < 1e-4


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
    cfg = gk.CONFIGS["mixed"]
    model, w = build(cfg, FP32, 11)
    toks = [prompt(cfg, n, 40 + i) for i, n in enumerate((70, 3, 129, 20, 64))]
    want = [greedy(cfg, w, t, 10) for t in toks]
    b = batcher(model, slots=2, pool_tokens=64 * 8, prefill_chunk=48)
    for _ in range(2):                                  # the second run reuses slots and pages
        outs, stats = b.run(toks, 10)
        assert outs == want and stats.output_tokens == 50
    even = torch.stack([prompt(cfg, 30, 50), prompt(cfg, 30, 51)])
    want = [greedy(cfg, w, t, 9) for t in even]
    out = Generator(model).generate(even, SamplingConfig(max_new_tokens=9)).output_token_ids
    assert out[:, 30:].tolist() == want
    # device-resident loop: one recorded step per token, across page, window and chunk borders
    cache = model.new_cache(2, 64 * 8, 200)
    with torch.inference_mode():
        last = model.forward_ragged(even.to(DEV), [30, 30], cache).logits[:, -1].argmax(-1)
        loop = GreedyDeviceLoop(model, cache, last, torch.full((2,), 30, device=DEV), max_new_tokens=80)
        loop.run()
    assert [[int(f)] + r[:8] for f, r in zip(last, loop.tokens.tolist())] == want
    assert loop.tokens[0, :79].tolist() == greedy(cfg, w, even[0], 80)[1:80]


def test_recorded_decoding_in_bf16_follows_the_steps():
    """The recorded step (positions on the device) and steps made on the host give the same tokens."""
    from pace_b200.llm.device_loop import GreedyDeviceLoop
    cfg = gk.CONFIGS["wide"]
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


def test_beam_search_and_rollback_follow_the_caches():
    from pace_b200.llm.configs import SamplingConfig
    from pace_b200.llm.generator import Generator
    cfg = gk.config([gk.layer(gk.A, gk.att(2, 1, 16, 16, 40), gk.dense(24)), gk.layer(gk.L2, gk.lat(2, 16, 8, 16, 16, 24, 30), gk.moe(16, 4, 2))], 32)
    model, w = build(cfg, FP32, 13)
    p = prompt(cfg, 66, 60)
    got = Generator(model).generate(p[None], SamplingConfig(max_new_tokens=5, num_beams=3)).output_token_ids[0, 66:].tolist()
    beams = [([], 0.0)]
    for _ in range(5):
        cand = []
        for seq, s in beams:
            lp = torch.log_softmax(ref.run(cfg, w, p.tolist() + seq)[-1], -1)
            cand += [(seq + [t], s + float(lp[t])) for t in range(cfg["vocab"])]
        beams = sorted(cand, key=lambda c: -c[1])[:3]
    assert got == beams[0][0]
    b = batcher(model, slots=1)
    feed(b, b.open(), prompt(cfg, 10, 9), [10])
    b.manager.remove_cache(7)                           # three tokens stay; attention-only stacks roll back
    toks = torch.cat([prompt(cfg, 10, 9)[:3], prompt(cfg, 40, 61)])
    assert gk.error(feed(b, 0, toks[3:], [20, 1]), ref.run(cfg, w, toks)[3:]) < 1e-4


@pytest.mark.parametrize("dtype", [BF16, FP32])
def test_trace_replay_program(tmp_path, dtype):
    from pace_b200.llm.weights import write_safetensors
    cfg = gk.CONFIGS["mixed"]
    w = gk.weights(cfg, 15, decided=dtype == BF16)
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
    assert gk.error(out(0), wa[[0, 95]]) < TOL[dtype] and not (tmp_path / "1.f32").exists()
    assert gk.error(out(2), torch.stack([wc[11], wc[5], wa[96]])) < TOL[dtype]
    assert gk.error(out(3), wc[[11]]) < TOL[dtype]
