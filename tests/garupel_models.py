"""Small Garupel configurations and random weights for the tests (nothing of the product path is used here)."""
import math

import torch


def att(heads, kv_heads, dim, vdim, scale=None, coef=0.2, every=16):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.0 / math.sqrt(dim),
            "q_temp": {"coef": coef, "every": every}}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def lru(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def lin(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def config(layers, width, vocab=61, loop=None, eps=1e-6):
    c = {"architecture": "Garupel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


# every size differs from every other one where the design lets it; the second and third make sizes equal or 1
CONFIGS = {
    "mixed": config([layer("lightning", lin(3, 20, 36, [0.5, 0.9, 0.995]), 50), layer("attention", att(6, 3, 24, 40)),
                     layer("rglru", lru(60, 3, 3), 44), layer("rglru", lru(36, 2, 5)),
                     layer("attention", att(4, 1, 40, 16, every=5), 28)], 72, loop=(1, 4, 3), eps=1e-4),
    "ones": config([layer("rglru", lru(33, 1, 1), 40), layer("attention", att(1, 1, 96, 96, coef=0.0), 40),
                    layer("lightning", lin(1, 40, 40, [1.0]), 40)], 40),
    "wide": config([layer("attention", att(12, 2, 112, 128), 64), layer("lightning", lin(2, 132, 260, [0.97, 0.2])),
                    layer("rglru", lru(66, 2, 4), 70), layer("attention", att(4, 4, 160, 72), 96)], 136, loop=(0, 1, 2)),
    "big_group": config([layer("attention", att(40, 1, 64, 64, scale=0.3), 32)], 48, loop=(0, 1, 1)),
}


def weights(cfg, seed=0):
    """Random bf16 tensors under the checkpoint's names: unit-gain matrices, norms around one, biases and
    gates large enough to matter."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, generator=g) / math.sqrt(shape[-1])

    def vec(name, *shape, mean=0.0, std=0.3):
        out[name] = torch.randn(*shape, generator=g) * std + mean

    out["embed"] = torch.randn(V, D, generator=g)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        names = ["norm1", "norm1b"] + (["norm2", "norm2b"] if lay["mlp"] else [])
        for n in names:
            vec(p + n, D, mean=1.0)
        mix = p + "mix."
        if lay["type"] == "attention":
            nq, nk, nv, no = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
            for n, r in (("q", nq), ("k", nk), ("v", nv)):
                mat(mix + n, r, D)
                vec(f"{mix}{n}.b", r)
            vec(mix + "q.norm", nq, mean=1.5)
            vec(mix + "k.norm", nk, mean=1.5)
            mat(mix + "g", no, D)
            mat(mix + "o", D, no)
        elif lay["type"] == "rglru":
            W, nb = m["width"], m["blocks"]
            for n in ("y", "x"):
                mat(mix + n, W, D)
                vec(f"{mix}{n}.b", W)
            vec(mix + "conv", W, m["conv"], std=0.5)
            vec(mix + "conv.b", W)
            for n in ("ra", "ri"):
                mat(mix + n, nb, W // nb, W // nb)
                vec(f"{mix}{n}.b", nb, W // nb)
            vec(mix + "lam", W, mean=-4.0, std=1.5)
            mat(mix + "o", D, W)
        else:
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, r in (("q", nk), ("k", nk), ("v", nv), ("g", nv)):
                mat(mix + n, r, D)
            vec(mix + "norm", nv, mean=1.0)
            mat(mix + "o", D, nv)
        if lay["mlp"]:
            mat(p + "mlp.up", lay["mlp"]["ff"], D)
            mat(p + "mlp.down", D, lay["mlp"]["ff"])
    vec("final.norm", D, mean=1.0)
    mat("head", V, D)
    return {k: v.bfloat16() for k, v in out.items()}


def error(got, want):
    """Largest row error: rms of the mean-free difference over the rms of all wanted logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt()).max() / w.pow(2).mean().sqrt())
