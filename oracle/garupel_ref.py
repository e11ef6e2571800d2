"""Plain, slow restatement of the Garupel decoder, one function per mechanism (torch on the CPU, float64
unless the caller's tensors say otherwise).  Test infrastructure: nothing here is used by the product path
and nothing of the product path is used here.

A sequence is processed token by token; a layer's memory is whatever its function keeps in ``cache`` (a dict
that starts empty), so prompts, portions and decoding are the same code.  ``w`` maps tensor names to tensors.
"""
import math

import torch


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def query_temperature(pos, coef, every):
    """Factor of the query at position ``pos``: grows with the log of the number of blocks of ``every`` tokens."""
    return 1.0 + coef * math.log((pos + 1) // every + 1)


def softmax_read(q, keys, values, scale):
    """One query ``[dim]`` over keys ``[n, dim]`` and values ``[n, vdim]``."""
    s = (keys @ q) * scale
    p = torch.exp(s - s.max())
    return (p / p.sum()) @ values


def attention_token(h, pos, m, w, pre, cache, eps):
    """Causal grouped-query attention of one token: whole-projection norms, no rotation, query temperature,
    sigmoid output gate."""
    H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = w[pre + "q"] @ h + w[pre + "q.b"]
    k = w[pre + "k"] @ h + w[pre + "k.b"]
    v = w[pre + "v"] @ h + w[pre + "v.b"]
    q = rms_norm(q, w[pre + "q.norm"], eps).view(H, d) * query_temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])
    k = rms_norm(k, w[pre + "k.norm"], eps).view(G, d)
    cache.setdefault("k", []).append(k)
    cache.setdefault("v", []).append(v.view(G, vd))
    ks, vs = torch.stack(cache["k"]), torch.stack(cache["v"])
    out = [softmax_read(q[i], ks[:, i // (H // G)], vs[:, i // (H // G)], m["scale"]) for i in range(H)]
    o = torch.cat(out) * torch.sigmoid(w[pre + "g"] @ h)
    return w[pre + "o"] @ o


def causal_conv_token(x, taps, bias, past):
    """``taps`` [channels, n]: the last column weighs the current token; ``past``: inputs so far, oldest first
    (changed in place)."""
    past.append(x)
    n = taps.shape[1]
    out = bias.clone()
    for j in range(n):
        at = len(past) - n + j
        if at >= 0:
            out = out + taps[:, j] * past[at]
    return out


def rglru_gates(u, ra, ra_b, ri, ri_b):
    """Block-diagonal gates of the recurrence: (r, i)."""
    ub = u.view(ra.shape[0], -1)
    r = torch.sigmoid(torch.einsum("boi,bi->bo", ra, ub) + ra_b)
    i = torch.sigmoid(torch.einsum("boi,bi->bo", ri, ub) + ri_b)
    return r.reshape(-1), i.reshape(-1)


def rglru_step(state, u, r, i, lam):
    log_a = -8.0 * r * torch.nn.functional.softplus(lam)
    return torch.exp(log_a) * state + torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u


def rglru_token(h, m, w, pre, cache):
    y = gelu_tanh(w[pre + "y"] @ h + w[pre + "y.b"])
    u = causal_conv_token(w[pre + "x"] @ h + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"],
                          cache.setdefault("inputs", []))
    r, i = rglru_gates(u, w[pre + "ra"], w[pre + "ra.b"], w[pre + "ri"], w[pre + "ri.b"])
    cache["S"] = rglru_step(cache.get("S", torch.zeros_like(u)), u, r, i, w[pre + "lam"])
    return w[pre + "o"] @ (cache["S"] * y)


def lightning_step(state, q, k, v, decay):
    """state [heads, dim, vdim], q/k [heads, dim], v [heads, vdim], decay [heads] -> (state, out [heads, vdim])."""
    state = decay[:, None, None] * state + k[:, :, None] * v[:, None, :]
    return state, torch.einsum("hdv,hd->hv", state, q)


def lightning_token(h, m, w, pre, cache, eps):
    n, d, vd = m["heads"], m["dim"], m["vdim"]
    silu = torch.nn.functional.silu
    q, k = silu(w[pre + "q"] @ h).view(n, d), silu(w[pre + "k"] @ h).view(n, d)
    v = silu(w[pre + "v"] @ h).view(n, vd)
    S = cache.get("S", torch.zeros(n, d, vd, dtype=h.dtype))
    cache["S"], o = lightning_step(S, q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    o = rms_norm(o.reshape(-1), w[pre + "norm"], eps) * torch.sigmoid(w[pre + "g"] @ h)
    return w[pre + "o"] @ o


def mlp_token(h, w, pre):
    return w[pre + "down"] @ torch.relu(w[pre + "up"] @ h) ** 2


def layer_runs(cfg):
    """(layer, opens a repeated pass) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    runs = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


class Sequence:
    """One sequence through the whole model, a token at a time."""

    def __init__(self, cfg, weights, dtype=torch.float64):
        self.cfg, self.w = cfg, {k: v.to(dtype) for k, v in weights.items()}
        self.runs = layer_runs(cfg)
        self.caches = [{} for _ in self.runs]
        self.pos = 0

    def token(self, tok, want_layers=False):
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        emb = w["embed"][tok]
        x, seen = emb, []
        for (i, opens), cache in zip(self.runs, self.caches):
            if opens:
                x = x + emb
            lay, pre = cfg["layers"][i], f"l{i}."
            h = rms_norm(x, w[pre + "norm1"], eps)
            m, mix = lay["mixer"], pre + "mix."
            if lay["type"] == "attention":
                y = attention_token(h, self.pos, m, w, mix, cache, eps)
            elif lay["type"] == "rglru":
                y = rglru_token(h, m, w, mix, cache)
            else:
                y = lightning_token(h, m, w, mix, cache, eps)
            x = x + rms_norm(y, w[pre + "norm1b"], eps)
            if lay["mlp"] is not None:
                y = mlp_token(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.")
                x = x + rms_norm(y, w[pre + "norm2b"], eps)
            seen.append(x)
        self.pos += 1
        logits = w["head"] @ rms_norm(x, w["final.norm"], eps)
        return (logits, torch.stack(seen)) if want_layers else logits

    def run(self, tokens):
        return torch.stack([self.token(int(t)) for t in tokens])
