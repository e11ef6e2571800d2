"""Small Lesosun configurations and random weights for the tests (nothing of the product path is used here)."""
import math

import torch


def left(heads, kv_heads, dim, vdim, conv, rot, base=1e4, scale=None, softcap=5.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rot": {"dims": rot, "base": base},
            "scale": scale or 1.0 / math.sqrt(dim), "softcap": softcap}


def right(heads, groups, state, vdim, conv, norm_groups):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}


def par(a, r, left_scale=1.3, right_scale=0.6):
    return {"left": a, "right": r, "left_scale": left_scale, "right_scale": right_scale}


def cd(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity=0, shared=None, scale=1.7):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


P, D = "parallel", "channel_delta"


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width, vocab=67, eps=1e-5, mult=0.7, cap=9.0):
    return {"architecture": "Lesosun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "residual_mult": mult, "logit_softcap": cap}


# sizes differ from one another where the design lets them; then sizes that are equal or 1; sizes the vector and tensor-core
# paths do not take; wide heads
CONFIGS = {
    "mixed": config([layer(P, par(left(6, 2, 40, 24, 3, 16), right(6, 3, 24, 16, 4, 2)), moe(24, 5, 3, 2, 40)),
                     layer(D, cd(6, 2, 24, 40, 3), dense(56)), layer(D, cd(3, 3, 48, 16, 5)),
                     layer(P, par(left(4, 4, 32, 48, 2, 32, 5e5, softcap=2.0), right(4, 1, 40, 32, 2, 4), 0.8, -1.1), dense(72)),
                     layer(D, cd(4, 1, 64, 72, 4), moe(40, 6, 2, 1))], 88, eps=1e-3),
    "ones": config([layer(P, par(left(1, 1, 32, 32, 1, 2), right(1, 1, 32, 32, 1, 1), 1.0, 1.0), moe(32, 1, 1)),
                    layer(D, cd(1, 1, 32, 32, 1), moe(32, 1, 1, 1, 32, 1.0)), layer(P, par(left(1, 1, 8, 8, 4, 8), right(1, 1, 8, 8, 4, 1)))],
                   32, mult=1.0),
    "odd": config([layer(P, par(left(3, 1, 22, 13, 5, 6), right(6, 2, 11, 7, 3, 3)), moe(11, 3, 2, 1, 9)),
                   layer(D, cd(3, 3, 13, 21, 2), dense(19)), layer(P, par(left(2, 2, 10, 31, 3, 10), right(5, 1, 3, 1, 6, 1)), moe(20, 4, 6, 3))],
                  37),
    "wide": config([layer(P, par(left(8, 2, 128, 128, 4, 64, 1e6), right(8, 2, 128, 64, 4, 2)), moe(64, 12, 4, 2, 96)),
                    layer(D, cd(4, 2, 128, 128, 4), moe(136, 40, 5, 8, 64)),
                    layer(P, par(left(4, 1, 136, 72, 4, 136), right(2, 1, 144, 136, 4, 1)), dense(120)), layer(D, cd(2, 1, 160, 136, 4))], 160),
}


def weights(cfg, seed=0, decided=False, ranks=(10, 19)):
    """Random bf16 tensors under the checkpoint's names: unit-gain matrices, norms and biases large enough to matter, decays
    from hardly any to strong.  ``decided``: the corrections settle every choice of experts (no token is a close call)."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, *shape):
        out[name] = torch.randn(*shape, generator=g) / math.sqrt(shape[-1])

    def vec(name, *shape, mean=0.0, std=0.3):
        out[name] = torch.randn(*shape, generator=g) * std + mean

    out["embed"] = torch.randn(V, W, generator=g)
    vec("embed.norm", W)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        mix, mlp = p + "mix.", lay["mlp"]
        vec(p + "norm1", W)
        if lay["type"] == P:
            a, r, pre = m["left"], m["right"], mix + "left."
            for n, c in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                mat(pre + n, c, W)
                vec(f"{pre}{n}.b", c)
                vec(f"{pre}{n}.conv", c, a["conv"], std=0.6)
            vec(pre + "q.norm", a["dim"], mean=1.5)
            vec(pre + "k.norm", a["dim"], mean=1.5)
            mat(pre + "o", W, a["heads"] * a["vdim"])
            vec(pre + "o.b", W)
            pre, inner, H = mix + "right.", r["heads"] * r["vdim"], r["heads"]
            ch = inner + 2 * r["groups"] * r["state"]
            mat(pre + "in", inner + ch + H, W)
            vec(pre + "conv", ch, r["conv"], std=0.6)
            vec(pre + "conv.b", ch)
            vec(pre + "dt_bias", H, mean=-1.5, std=1.0)
            vec(pre + "A_log", H, mean=0.0, std=1.0)
            vec(pre + "D", H, mean=1.0)
            vec(pre + "norm", inner, mean=1.0)
            mat(pre + "o", W, inner)
        else:
            H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * vd)):
                mat(mix + n, c, W)
                vec(f"{mix}{n}.conv", c, m["conv"], std=0.6)
            mat(mix + "b", H, W)
            mat(mix + "a1", ranks[0], W)
            mat(mix + "a2", H * d, ranks[0])
            mat(mix + "g1", ranks[1], W)
            mat(mix + "g2", H * vd, ranks[1])
            vec(mix + "dt_bias", H * d, mean=-2.0, std=2.0)
            vec(mix + "A_log", H, mean=0.0, std=1.0)
            vec(mix + "norm", vd, mean=1.0)
            mat(mix + "o", W, H * vd)
        if mlp:
            vec(p + "norm2", W)
            q = p + "mlp."
            if mlp["kind"] == "dense":
                mat(q + "gate", mlp["ff"], W)
                mat(q + "up", mlp["ff"], W)
                mat(q + "down", W, mlp["ff"])
                continue
            r = mlp["router"]
            parts = [(f"{q}e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
            if mlp.get("shared"):
                parts.append((q + "shared.", mlp["shared"]["ff"]))
            for pre, ff in parts:
                mat(pre + "up", ff, W)
                mat(pre + "down", W, ff)
            n = r["experts"] + r["identity"]
            mat(q + "router", n, W)
            vec(q + "correction", n, std=0.1)
            if decided:
                out[q + "correction"] = (torch.randperm(n, generator=g) < r["top"]).float() * 2
    vec("final.norm", W)
    return {k: v.bfloat16() for k, v in out.items()}


def error(got, want):
    """Largest row error: rms of the mean-free difference over the rms of all wanted logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt()).max() / w.pow(2).mean().sqrt())
