"""Plain, slow restatement of the Gekupel decoder, one function per mechanism (torch on the CPU, float64 unless the
caller's tensors say otherwise).  Test infrastructure: nothing here is used by the product path and nothing of the
product path is used here.

A sequence is processed as a whole: row i of every matrix is position i, and what a position may see is one boolean
matrix ``[n, n]``.  There is no cache, no portion and no batch, so a fault of any of them cannot be here as well.
``w`` maps tensor names to tensors.
"""
import math

import torch


def rms_norm(x, eps, weight=None):
    """x / sqrt(mean(x^2) + eps) (* weight) over the last axis."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ---- what a position sees -------------------------------------------------------------------------------------
def window_mask(n, size):
    """[i, j]: j is i or one of the size - 1 positions in front of it."""
    d = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (d >= 0) & (d < size)


def chunk_mask(n, size):
    """[i, j]: j is not behind i and lies in the same stretch of ``size`` positions counted from 0."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


# ---- positions --------------------------------------------------------------------------------------------------
def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def rotation_frequencies(dims, base, scaling=None):
    """(frequency per pair, factor of cos and sin).  With scaling (YaRN): pairs that turn often within the original
    length keep their frequency, pairs that turn seldom are slowed down by the factor, a linear ramp in between."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def pair_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, dims, freq, mult):
    """x ``[n, heads, d]``: neighbours (2i, 2i + 1) of the first ``dims`` elements turn by position * freq[i]."""
    n = x.shape[0]
    a = torch.arange(n, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None, :]
    c, s = (torch.cos(a) * mult).to(x.dtype)[:, None, :], (torch.sin(a) * mult).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


# ---- attention ----------------------------------------------------------------------------------------------------
def masked_softmax(scores, seen, sink=None):
    """Weights over the last axis where ``seen``; ``sink`` (a number) only adds exp(sink) to the denominator."""
    s = scores.masked_fill(~seen, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    p = torch.exp(s - top)
    den = p.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return p / den


def attention(h, m, w, pre, eps):
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[pre + "q"].T).view(n, H, d), eps)
    k = rms_norm((h @ w[pre + "k"].T).view(n, G, d), eps)
    v = (h @ w[pre + "v"].T).view(n, G, vd)
    seen = chunk_mask(n, m["mask"]["size"])
    dist = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).to(h.dtype)
    out = []
    for i, slope in enumerate(distance_slopes(H)):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].T) * m["scale"] - slope * dist
        out.append(masked_softmax(s, seen, w[pre + "sink"][i]) @ v[:, g])
    return torch.cat(out, -1) @ w[pre + "o"].T


def latent_attention(h, m, w, pre, eps, sink):
    n, H, d, r, vd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[pre + "dq"].T, eps, w[pre + "dq.norm"])
    q = (cq @ w[pre + "uq"].T).view(n, H, d + r)
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :R], eps, w[pre + "dkv.norm"])
    freq, mult = rotation_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    kr = rotate_pairs(down[:, None, R:], m["rot"]["dims"], freq, mult)[:, 0]
    qr = rotate_pairs(q[..., d:], m["rot"]["dims"], freq, mult)
    k = (c @ w[pre + "uk"].T).view(n, H, d)
    v = (c @ w[pre + "uv"].T).view(n, H, vd)
    seen = window_mask(n, m["mask"]["size"])
    out = []
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        out.append(masked_softmax(s, seen, w[pre + "sink"][i] if sink else None) @ v[:, i])
    return torch.cat(out, -1) @ w[pre + "o"].T


MIXERS = {"attention": attention,
          "latent_attention": lambda *a: latent_attention(*a, sink=False),
          "latent_attention_2": lambda *a: latent_attention(*a, sink=True)}


# ---- feed-forward -------------------------------------------------------------------------------------------------
def dense_mlp(h, w, pre):
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(h, router, correction, top):
    """(chosen experts ``[n, top]``, their weights): the choice looks at score + correction, the weights do not."""
    s = 1.0 / (1.0 + torch.exp(-(h @ router.T)))
    chosen = torch.argsort(s + correction, dim=-1, descending=True)[:, :top]
    return chosen, s.gather(-1, chosen)


def expert_mlp(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def moe_mlp(h, m, w, pre):
    chosen, weight = route(h, w[pre + "router"], w[pre + "correction"], m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        tok, place = (chosen == e).nonzero(as_tuple=True)
        if len(tok):
            out[tok] += weight[tok, place][:, None] * expert_mlp(h[tok], w, f"{pre}e{e}.")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def run(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits ``[n, vocab]`` of a sequence (and the residual stream behind every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    seen = []
    for i, lay in enumerate(cfg["layers"]):
        pre = f"l{lay.get('weights_of', i)}."
        x = x + rms_norm(MIXERS[lay["type"]](x, lay["mixer"], w, pre + "mix.", eps), eps, w[pre + "norm1"])
        mlp = lay.get("mlp")
        if mlp is not None:
            y = dense_mlp(x, w, pre + "mlp.") if mlp["kind"] == "dense" else moe_mlp(x, mlp, w, pre + "mlp.")
            x = x + rms_norm(y, eps, w[pre + "norm2"])
        seen.append(x)
    logits = rms_norm(x, eps, w["final.norm"]) @ w["head"].T
    return (logits, torch.stack(seen)) if want_layers else logits
