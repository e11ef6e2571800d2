"""Small Kibotar configurations and random weights for the tests (nothing of the product path is used here)."""
import math

import torch

SCALING = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 40}


def att(heads, kv_heads, dim, vdim, window, block, rot, base=1e4, scaling=None, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "pool": block},
            "rot": {"dims": rot, "base": base, "scaling": scaling}, "scale": scale or 1.0 / math.sqrt(dim)}


def gla(heads, dim, vdim, tau=16.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def lat(heads, dim, vdim, kv_rank, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale or 1.0 / math.sqrt(dim)}


A, G, L = "attention", "gla", "latent_attention"


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width, vocab=67, eps=1e-5, scale=3.0, loop=None, bigram=(31, 7, 11)):
    c = {"architecture": "Kibotar", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": scale}}
    if bigram:
        c["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# sizes differ from one another where the design lets them; then sizes that are equal or 1; sizes the vector and tensor-core
# paths do not take; wide heads
CONFIGS = {
    "mixed": config([layer(A, att(6, 2, 40, 24, 37, 5, 24, scaling=SCALING), 56), layer(G, gla(3, 24, 40, 4.0), 40), layer(L, lat(5, 24, 40, 48)),
                     layer(A, att(4, 4, 24, 56, 21, 16, 24, 5e5), 72), layer(G, gla(2, 48, 16))], 88, eps=1e-3, loop=(1, 4, 3)),
    "ones": config([layer(A, att(1, 1, 32, 32, 1, 1, 2), 32), layer(L, lat(1, 32, 32, 32)), layer(G, gla(1, 32, 32, 1.0), 32),
                    layer(A, att(1, 1, 8, 8, 64, 64, 8))], 32, scale=1.0, loop=(0, 4, 1), bigram=(1, 1, 1)),
    "odd": config([layer(G, gla(3, 13, 21, 5.5), 19), layer(L, lat(3, 11, 9, 21), 11), layer(A, att(3, 1, 22, 13, 19, 7, 6, scaling=SCALING), 23),
                   layer(A, att(6, 3, 10, 31, 50, 3, 10), 21)], 37, loop=(2, 4, 2), bigram=(13, 70001, 90001)),
    "wide": config([layer(A, att(16, 4, 128, 128, 70, 8, 64, 1e6), 96), layer(L, lat(4, 128, 64, 160), 64), layer(G, gla(4, 128, 136), 120),
                    layer(A, att(4, 2, 136, 72, 33, 4, 136), 64), layer(A, att(10, 5, 64, 120, 100, 24, 32), 64), layer(G, gla(2, 160, 72))], 160),
}


def weights(cfg, seed=0, rank=10):
    """Random bf16 tensors under the checkpoint's names: unit-gain matrices, norms and biases large enough to matter, decays
    from hardly any to strong, heads mixed about as much as kept."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, generator=g) / math.sqrt(shape[-1])

    def vec(name, *shape, mean=0.0, std=0.3):
        out[name] = torch.randn(*shape, generator=g) * std + mean

    out["embed"] = torch.randn(V, W, generator=g)
    if cfg["embedding"].get("bigram"):
        out["bigram"] = torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, W, generator=g) * 1.5
    if cfg.get("loop"):
        vec("loop.step", cfg["loop"]["times"], W, std=1.0)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        mix, H, d, vd = p + "mix.", m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b"):
            vec(p + n, W, mean=1.0)
        out[p + "shift"] = torch.rand(W, generator=g)
        if lay["type"] == A:
            for n, c in (("q", H * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * vd)):
                mat(mix + n, c, W)
                vec(f"{mix}{n}.b", c)
            out[mix + "q"] *= 2.0                       # scores that differ, so that single keys matter
            out[mix + "talk"] = torch.eye(H) + torch.randn(H, H, generator=g) * 0.5
            mat(mix + "g", H * vd, W)
            vec(mix + "o.b", W)
        elif lay["type"] == G:
            for n, c in (("q", H * d), ("k", H * d), ("v", H * vd), ("g", H * vd)):
                mat(mix + n, c, W)
            mat(mix + "a1", rank, W)
            mat(mix + "a2", H * d, rank)
            vec(mix + "a2.b", H * d, mean=2.0, std=2.0)
            vec(mix + "norm", vd, mean=1.0)
        else:
            mat(mix + "q", H * d, W)
            out[mix + "q"] *= 2.0
            mat(mix + "dkv", m["kv_rank"], W)
            vec(mix + "dkv.norm", m["kv_rank"], mean=1.0)
            mat(mix + "uk", H * d, m["kv_rank"])
            mat(mix + "uv", H * vd, m["kv_rank"])
            mat(mix + "g", H, W)
        mat(mix + "o", W, H * vd)
        if lay["mlp"]:
            for n in ("norm2", "norm2b"):
                vec(p + n, W, mean=1.0)
            mat(p + "mlp.up", lay["mlp"]["ff"], W)
            mat(p + "mlp.down", W, lay["mlp"]["ff"])
    vec("final.norm", W, mean=1.0)
    return {k: v.bfloat16() for k, v in out.items()}


def error(got, want):
    """Largest row error: rms of the mean-free difference over the rms of all wanted logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt()).max() / w.pow(2).mean().sqrt())
