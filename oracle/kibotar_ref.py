"""Plain, slow restatement of the Kibotar decoder, one function per mechanism (torch on the CPU, float64 unless the caller's
tensors say otherwise).  Test infrastructure: nothing here is used by the product path and nothing of the product path is used
here.

A sequence is processed as a whole: row i of every matrix is position i.  Recurrences walk over the positions one by one from a
zero state, attention is a matrix of weights over all tokens and blocks with boolean masks.  There is no cache, no portion and
no batch, so a fault of any of them cannot be here as well.  ``w`` maps tensor names to tensors.
"""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- what comes before the layers -----------------------------------------------------------------------------------
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table per position; the first token takes the row behind the last bucket."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embed(tokens, cfg, w):
    e = cfg["embedding"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * e["scale"]
    b = e.get("bigram")
    if b:
        x = x + w["bigram"][torch.tensor(bigram_rows(list(map(int, tokens)), b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


def token_shift(h, mix):
    """Every element between the token's own (mix 0) and the one of the token before (mix 1; zeros in front of the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


# ---- attention over a window and pooled blocks ---------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / f
            n, low, high = scaling["original"], scaling["low"], scaling["high"]
            if length > n / low:
                f = f / scaling["factor"]
            elif length >= n / high:
                s = (n / length - low) / (high - low)
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_half(x, dims, base, scaling=None):
    """x ``[n, heads, d]``: elements i and i + dims / 2 of the first ``dims`` turn by position * frequency i."""
    n, half = x.shape[0], dims // 2
    a = torch.arange(n, dtype=torch.float64)[:, None] * frequencies(dims, base, scaling)[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def block_means(x, size):
    """Means of the whole blocks of ``size`` rows."""
    b = x.shape[0] // size
    return x[: b * size].reshape(b, size, *x.shape[1:]).mean(1)


def pooled_mask(n, window, size):
    """Boolean ``[n, n + blocks]``: the tokens, then the blocks, that a position sees."""
    i = torch.arange(n)[:, None]
    d = i - torch.arange(n)[None, :]
    last = torch.arange(n // size)[None, :] * size + size - 1
    return torch.cat([(d >= 0) & (d < window), last <= i - window], 1)


def softmax_plus_one(s):
    """exp(s) / (1 + sum exp(s))."""
    m = torch.clamp(s.amax(-1, keepdim=True), min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def pooled_weights(q, k, scale, window, size):
    """Softmax weights ``[heads, n, n + blocks]``; q ``[n, heads, d]``, k ``[n, kv_heads, d]``."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    keys = torch.cat([k, block_means(k, size)])
    unseen = ~pooled_mask(n, window, size)
    return torch.stack([softmax_plus_one(((q[:, h] @ keys[:, h // (H // G)].T) * scale).masked_fill(unseen, -math.inf))
                        for h in range(H)])


def mixed_heads(p, v, talk, size):
    """Weights mixed over the heads, then the values of every head's own key/value head: ``[n, heads, vdim]``."""
    H, G = p.shape[0], v.shape[1]
    values = torch.cat([v, block_means(v, size)])
    mixed = torch.einsum("hg,gij->hij", talk, p)
    return torch.stack([mixed[h] @ values[:, h // (H // G)] for h in range(H)], 1)


def attention(h, m, w, pre, eps):
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[pre + x].T + w[f"{pre}{x}.b"]).view(n, c, e) for x, c, e in (("q", H, d), ("k", G, d), ("v", G, vd)))
    r = m["rot"]
    q, k = (rotate_half(x, r["dims"], r["base"], r.get("scaling")) for x in (q, k))
    size, window = m["mask"]["pool"], m["mask"]["size"]
    o = mixed_heads(pooled_weights(q, k, m["scale"], window, size), v, w[pre + "talk"], size).reshape(n, H * vd)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T + w[pre + "o.b"]


# ---- gated linear attention ----------------------------------------------------------------------------------------
def gla_scan(q, k, v, alpha):
    """q, k, alpha ``[n, heads, dim]``, v ``[n, heads, vdim]``: S = diag(alpha) S + k v^T, o = S^T q."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gla(h, m, w, pre, eps):
    n, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[pre + x].T).view(n, H, d) for x in "qk")
    z = ((h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]).view(n, H, d)
    o = gla_scan(q * d ** -0.5, k, (h @ w[pre + "v"].T).view(n, H, vd), sigmoid(z) ** (1.0 / m["tau"]))
    return ((rms(o, eps) * w[pre + "norm"]).reshape(n, H * vd) * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- latent attention ----------------------------------------------------------------------------------------------
def causal_softmax(q, k, v, scale):
    """q, k ``[n, heads, d]``, v ``[n, heads, vdim]``."""
    unseen = torch.ones(q.shape[0], q.shape[0], dtype=torch.bool).triu(1)
    return torch.stack([torch.softmax(((q[:, h] @ k[:, h].T) * scale).masked_fill(unseen, -math.inf), -1) @ v[:, h]
                        for h in range(q.shape[1])], 1)


def latent_attention(h, m, w, pre, eps):
    n, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c = rms(h @ w[pre + "dkv"].T, eps) * w[pre + "dkv.norm"]
    q, k, v = ((x @ w[pre + y].T).view(n, H, -1) for x, y in ((h, "q"), (c, "uk"), (c, "uv")))
    o = causal_softmax(q, k, v, m["scale"]) * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(n, H * vd) @ w[pre + "o"].T


MIXERS = {"attention": attention, "gla": gla, "latent_attention": latent_attention}


# ---- the model -----------------------------------------------------------------------------------------------------
def dense_mlp(h, w, pre):
    return torch.clamp(h @ w[pre + "up"].T, min=0) ** 2 @ w[pre + "down"].T


def runs(cfg):
    """(layer, number of the pass it opens or None) in execution order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return out + [(i, None) for i in range(lp["stop"], n)]


def run(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits ``[n, vocab]`` of a sequence (and the residual stream behind every layer run)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return rms(x, eps) * w[name]

    x, seen = embed(tokens, cfg, w), []
    for i, t in runs(cfg):
        lay, pre = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        h = token_shift(norm(x, pre + "norm1"), w[pre + "shift"])
        x = x + norm(MIXERS[lay["type"]](h, lay["mixer"], w, pre + "mix.", eps), pre + "norm1b")
        if lay.get("mlp"):
            x = x + norm(dense_mlp(norm(x, pre + "norm2"), w, pre + "mlp."), pre + "norm2b")
        seen.append(x)
    logits = norm(x, "final.norm") @ w["embed"].T
    return (logits, torch.stack(seen)) if want_layers else logits
