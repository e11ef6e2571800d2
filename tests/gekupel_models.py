"""Small Gekupel configurations and random weights for the tests (nothing of the product path is used here)."""
import math

import torch


def att(heads, kv_heads, dim, vdim, chunk, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
            "scale": scale or 1.0 / math.sqrt(dim)}


def lat(heads, dim, rot, vdim, q_rank, kv_rank, window, base=1e4, scaling=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "mask": {"size": window}, "rot": {"dims": rot, "base": base}, "scale": scale or 1.0 / math.sqrt(dim + rot)}
    if scaling:
        m["rot"]["scaling"] = scaling
    return m


def yarn(factor=4.0, original=256, fast=16.0, slow=2.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


A, L1, L2 = "attention", "latent_attention", "latent_attention_2"


def layer(kind, mixer, mlp=None, of=None):
    out = {"type": kind, "mixer": mixer, "mlp": mlp}
    if of is not None:
        out["weights_of"] = of
    return out


def config(layers, width, vocab=59, eps=1e-5, scale=3.5):
    return {"architecture": "Gekupel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": scale}}


_SHARED = layer(A, att(6, 2, 40, 24, 50), moe(24, 5, 2))
_LATENT = layer(L2, lat(3, 32, 8, 40, 56, 48, 21, scaling=yarn()), dense(72))
# sizes differ from one another where the design lets them; then sizes that are equal or 1; sizes the tensor-core kernels
# do not take; wide heads and long windows
CONFIGS = {
    "mixed": config([_LATENT, _SHARED, layer(L1, lat(5, 24, 16, 16, 32, 64, 70, base=5e5)), {**_SHARED, "weights_of": 1},
                     layer(L1, lat(2, 16, 24, 56, 40, 32, 33), moe(40, 7, 3)), {**_LATENT, "weights_of": 0}], 88, eps=1e-3),
    "ones": config([layer(L1, lat(1, 32, 2, 32, 32, 32, 1), dense(32)), layer(A, att(1, 1, 32, 32, 1), moe(32, 1, 1)),
                    layer(L2, lat(1, 8, 8, 8, 8, 8, 4, scaling=yarn(1.0)))], 32, scale=1.0),
    "odd": config([layer(A, att(3, 3, 20, 13, 9), moe(11, 3, 2)), layer(L2, lat(3, 13, 6, 11, 9, 21, 30, scaling=yarn(8.0)), dense(19)),
                   layer(L1, lat(2, 7, 2, 5, 5, 3, 64), moe(20, 9, 9))], 37),
    "wide": config([layer(L2, lat(4, 128, 64, 128, 96, 256, 100, scaling=yarn(2.0, 4096, 32.0, 1.0)), moe(64, 12, 4)),
                    layer(A, att(8, 1, 96, 112, 130), dense(120)), layer(A, att(4, 2, 136, 72, 64)),
                    layer(L1, lat(20, 64, 32, 64, 64, 128, 200), moe(136, 40, 5))], 160),
}


def weights(cfg, seed=0, decided=False):
    """Random bf16 tensors under the checkpoint's names: unit-gain matrices, norms around one, sinks large enough to
    matter.  ``decided``: the corrections settle every choice of experts (no token is a close call)."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, generator=g) / math.sqrt(shape[-1])

    def vec(name, n, mean=0.0, std=0.3):
        out[name] = torch.randn(n, generator=g) * std + mean

    out["embed"] = torch.randn(V, D, generator=g) / cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        if "weights_of" in lay:
            continue
        p, m = f"l{i}.", lay["mixer"]
        mix, mlp = p + "mix.", lay["mlp"]
        vec(p + "norm1", D, mean=1.0)
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        if lay["type"] == A:
            mat(mix + "q", H * d, D)
            mat(mix + "k", m["kv_heads"] * d, D)
            mat(mix + "v", m["kv_heads"] * vd, D)
        else:
            mat(mix + "dq", m["q_rank"], D)
            vec(mix + "dq.norm", m["q_rank"], mean=1.0)
            mat(mix + "uq", H * (d + m["rot_dim"]), m["q_rank"])
            mat(mix + "dkv", m["kv_rank"] + m["rot_dim"], D)
            vec(mix + "dkv.norm", m["kv_rank"], mean=1.0)
            mat(mix + "uk", H * d, m["kv_rank"])
            mat(mix + "uv", H * vd, m["kv_rank"])
        if lay["type"] != L1:
            vec(mix + "sink", H, mean=1.0, std=1.0)
        mat(mix + "o", D, H * vd)
        if mlp:
            vec(p + "norm2", D, mean=1.0)
            q = p + "mlp."
            parts = [(q, mlp["ff"])] if mlp["kind"] == "dense" else \
                [(f"{q}e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            for pre, ff in parts:
                mat(pre + "gate", ff, D)
                mat(pre + "up", ff, D)
                mat(pre + "down", D, ff)
            if mlp["kind"] == "moe":
                E = mlp["router"]["experts"]
                mat(q + "router", E, D)
                vec(q + "correction", E, std=0.2)
                if decided:
                    out[q + "correction"] = (torch.randperm(E, generator=g) < mlp["router"]["top"]).float() * 2
    vec("final.norm", D, mean=1.0)
    mat("head", V, D)
    return {k: v.bfloat16() for k, v in out.items()}


def error(got, want):
    """Largest row error: rms of the mean-free difference over the rms of all wanted logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt()).max() / w.pow(2).mean().sqrt())
