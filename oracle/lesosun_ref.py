"""Plain, slow restatement of the Lesosun decoder, one function per mechanism (torch on the CPU, float64 unless the
caller's tensors say otherwise).  Test infrastructure: nothing here is used by the product path and nothing of the
product path is used here.

A sequence is processed as a whole: row i of every matrix is position i.  Recurrences walk over the positions one by one
from a zero state.  There is no cache, no portion and no batch, so a fault of any of them cannot be here as well.
``w`` maps tensor names to tensors.
"""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def short_conv(u, taps, bias=None):
    """u ``[n, channels]``, taps ``[channels, k]``: the last tap weighs the current position, zeros in front."""
    n, k = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, u.shape[1], dtype=u.dtype), u])
    out = torch.zeros_like(u) if bias is None else bias.expand_as(u).clone()
    for j in range(k):
        out = out + taps[:, j] * padded[j: j + n]
    return out


def rotate_pairs(x, dims, base):
    """x ``[n, heads, d]``: neighbours (2i, 2i + 1) of the first ``dims`` elements turn by position * base^(-2i / dims)."""
    n = x.shape[0]
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(n, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


# ---- mixers -------------------------------------------------------------------------------------------------------
def capped_attention(h, m, w, pre, eps):
    """Causal softmax attention behind short convolutions of q, k and v; normalised and rotated q and k; capped scores."""
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    p = {x: short_conv(h @ w[pre + x].T + w[f"{pre}{x}.b"], w[f"{pre}{x}.conv"]) for x in "qkv"}
    rot = m["rot"]
    q = rotate_pairs(rms(p["q"].view(n, H, d), eps) * w[pre + "q.norm"], rot["dims"], rot["base"])
    k = rotate_pairs(rms(p["k"].view(n, G, d), eps) * w[pre + "k.norm"], rot["dims"], rot["base"])
    v = p["v"].view(n, G, vd)
    unseen = torch.ones(n, n, dtype=torch.bool).triu(1)
    out = []
    for i in range(H):
        g = i // (H // G)
        s = soft_cap((q[:, i] @ k[:, g].T) * m["scale"], m["softcap"]).masked_fill(unseen, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.cat(out, -1) @ w[pre + "o"].T + w[pre + "o.b"]


def ssd_scan(x, b, c, dt, a_log, d_skip):
    """x ``[n, heads, vdim]``, b and c ``[n, heads, N]``, dt ``[n, heads]``: S = exp(-exp(a_log) dt) S + dt b x^T,
    y = S^T c + d_skip x."""
    n, H, P = x.shape
    S = torch.zeros(H, b.shape[2], P, dtype=x.dtype)
    out = []
    for t in range(n):
        S = torch.exp(-torch.exp(a_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, c[t]) + d_skip[:, None] * x[t])
    return torch.stack(out)


def gated_group_norm(y, z, weight, groups, eps):
    """Gate first, then every one of ``groups`` equal parts by its own root mean square."""
    y = y * silu(z)
    return rms(y.view(y.shape[0], groups, -1), eps).reshape(y.shape) * weight


def state_space(h, m, w, pre, eps):
    n, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w[pre + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, b, c = torch.split(xbc, [inner, G * N, G * N], -1)
    b, c = (t.view(n, G, N).repeat_interleave(H // G, 1) for t in (b, c))
    y = ssd_scan(x.view(n, H, P), b, c, softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], w[pre + "D"])
    return gated_group_norm(y.reshape(n, inner), z, w[pre + "norm"], m["norm_groups"], eps) @ w[pre + "o"].T


def parallel(h, m, w, pre, eps):
    return (m["left_scale"] * capped_attention(h, m["left"], w, pre + "left.", eps)
            + m["right_scale"] * state_space(h, m["right"], w, pre + "right.", eps))


def delta_scan(q, k, v, g, beta):
    """q, k, g ``[n, heads, dim]``, v ``[n, heads, vdim]``, beta ``[n, heads]``: S = g S; u = beta (v - S^T k); S += k u^T;
    o = S^T q."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta(h, m, w, pre, eps):
    n, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    p = {x: silu(short_conv(h @ w[pre + x].T, w[f"{pre}{x}.conv"])) for x in "qkv"}
    q, k = (unit(p[x].view(n, G, d)).repeat_interleave(H // G, 1) for x in "qk")
    beta = sigmoid(h @ w[pre + "b"].T)
    a = softplus((h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]).view(n, H, d)
    g = torch.exp(-torch.exp(w[pre + "A_log"])[:, None] * a)
    o = delta_scan(q * d ** -0.5, k, p["v"].view(n, H, vd), g, beta)
    gate = sigmoid((h @ w[pre + "g1"].T) @ w[pre + "g2"].T)
    return ((rms(o, eps) * w[pre + "norm"]).reshape(n, H * vd) * gate) @ w[pre + "o"].T


MIXERS = {"parallel": parallel, "channel_delta": channel_delta}


# ---- feed-forward -------------------------------------------------------------------------------------------------
def dense_mlp(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def expert_mlp(h, w, pre):
    return gelu_erf(h @ w[pre + "up"].T) @ w[pre + "down"].T


def route(h, router, correction, top, scale):
    """(chosen outputs ``[n, top]``, their weights): softmax scores; the choice looks at score + correction, the weights are
    the chosen scores, made to sum to ``scale``."""
    s = torch.softmax(h @ router.T, -1)
    chosen = torch.argsort(s + correction, dim=-1, descending=True, stable=True)[:, :top]
    picked = s.gather(-1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20) * scale


def moe_mlp(h, m, w, pre):
    r = m["router"]
    chosen, weight = route(h, w[pre + "router"], w[pre + "correction"], r["top"], r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        tok, place = (chosen == e).nonzero(as_tuple=True)
        if len(tok):
            y = expert_mlp(h[tok], w, f"{pre}e{e}.") if e < r["experts"] else h[tok]
            out[tok] += weight[tok, place][:, None] * y
    if m.get("shared"):
        out = out + expert_mlp(h, w, pre + "shared.")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def run(cfg, weights, tokens, dtype=torch.float64, want_layers=False):
    """Logits ``[n, vocab]`` of a sequence (and the residual stream behind every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return rms(x, eps) * (1.0 + w[name])

    x = norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], "embed.norm")
    seen = []
    for i, lay in enumerate(cfg["layers"]):
        pre = f"l{i}."
        y = MIXERS[lay["type"]](norm(x, pre + "norm1"), lay["mixer"], w, pre + "mix.", eps)
        mlp = lay.get("mlp")
        if mlp is not None:
            h = norm(x, pre + "norm2")
            y = y + (dense_mlp(h, w, pre + "mlp.") if mlp["kind"] == "dense" else moe_mlp(h, mlp, w, pre + "mlp."))
        x = x + cfg["residual_mult"] * y
        seen.append(x)
    logits = soft_cap(norm(x, "final.norm") @ w["embed"].T, cfg["logit_softcap"])
    return (logits, torch.stack(seen)) if want_layers else logits
