"""Garupel: a decoder whose layers mix softmax attention, a real-gated linear recurrence (RG-LRU) and decayed
linear attention, with norms on both sides of every sublayer and a stretch of layers that runs several times.

Everything runs on a packed ``Step`` of tokens.  Between two sublayers one kernel adds the normalised output of
the first to the fp32 residual stream and normalises it for the second (at a pass boundary of the loop it also
adds the embedding rows again); per mixer the launches are

    attention  one projection (q, k, v, gate) -> norms + temperature + append -> attention -> output gate -> W_o
    rglru      one projection (y, x) -> convolution, gate products, scan (decode: one launch) -> W_o
    lightning  one projection (q, k, v, gate) -> silu + recurrence -> norm + gate -> W_o

A layer run (layer i in pass p) has its own K/V rows or state; the weights of a layer are shared by its runs.
"""
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple, Union

import torch
import torch.nn.functional as F
from torch import nn

from pace_b200.llm.cache import KVCacheType
from pace_b200.llm.hybrid_cache import HybridCacheManager, KVSpec, StateSpec
from pace_b200.llm.outputs import ModelOutput
from pace_b200.llm.registry import model_registry
from pace_b200.llm.step import Step
from pace_b200.ops import hybrid
from pace_b200.ops.linear import linear


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float
    temp_every: float


@dataclass(frozen=True)
class RglruConfig:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[AttentionConfig, RglruConfig, LightningConfig]
    ff: Optional[int]         # None: the layer has no feed-forward


def _mixer_config(kind: str, m: dict):
    if kind == "attention":
        t = m["q_temp"]
        c = AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(t["coef"]),
                            float(t["every"]))
        if c.heads % c.kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        return c
    if kind == "rglru":
        c = RglruConfig(m["width"], m["blocks"], m["conv"])
        if c.width % c.blocks:
            raise ValueError("the recurrence's width must be a multiple of its blocks")
        return c
    if kind == "lightning":
        decay = m["decay"] if isinstance(m["decay"], (list, tuple)) else [m["decay"]] * m["heads"]
        if len(decay) != m["heads"]:
            raise ValueError("one decay per head is needed")
        return LightningConfig(m["heads"], m["dim"], m["vdim"], tuple(float(d) for d in decay))
    raise ValueError(f"unknown mixer type {kind!r}")


@dataclass(frozen=True)
class GarupelConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerConfig, ...]
    eps: float
    loop: Tuple[int, int, int] = (0, 0, 1)    # layers start .. stop - 1 run `times` times in a row

    @staticmethod
    def from_dict(c: dict) -> "GarupelConfig":
        layers = []
        for lay in c["layers"]:
            mlp = lay.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerConfig(_mixer_config(lay["type"], lay["mixer"]), mlp["ff"] if mlp is not None else None))
        lp = c.get("loop")
        loop = (lp["start"], lp["stop"], lp["times"]) if lp else (0, 0, 1)
        if not 0 <= loop[0] <= loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError("loop must name a range of layers and a positive count")
        return GarupelConfig(c["vocab"], c["width"], tuple(layers), float(c["norm"]["eps"]), loop)

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, starts a pass after the first) in execution order."""
        start, stop, times = self.loop
        out = [(i, False) for i in range(start)]
        for t in range(times):
            out += [(i, t > 0 and i == start) for i in range(start, stop)]
        return out + [(i, False) for i in range(stop, len(self.layers))]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs())


def _vec(n: int, value: float = 0.0) -> nn.Parameter:
    """A small constant of a layer (norm weight, bias, taps): fp32 whatever the activations are."""
    return nn.Parameter(torch.full((n,) if isinstance(n, int) else n, value, dtype=torch.float32), requires_grad=False)


def _mat(rows: int, cols: int, dtype: torch.dtype) -> nn.Parameter:
    return nn.Parameter(torch.empty(rows, cols, dtype=dtype), requires_grad=False)


class _Tensors:
    """A checkpoint's tensors, handed out by name with their shapes checked; knows which were never asked for."""

    def __init__(self, tensors: Dict[str, torch.Tensor]):
        self.tensors, self.used = tensors, set()

    def take(self, name: str, *shape: int) -> torch.Tensor:
        if name not in self.tensors:
            raise KeyError(f"checkpoint has no tensor {name}")
        t = self.tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, the configuration wants {shape}")
        self.used.add(name)
        return t

    def unused(self) -> List[str]:
        return sorted(set(self.tensors) - self.used)


class AttentionMixer(nn.Module):
    def __init__(self, c: AttentionConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.nq, self.nk, self.nv = c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim
        self.n_out = c.heads * c.vdim
        self.qkvg = _mat(self.nq + self.nk + self.nv + self.n_out, width, dtype)
        self.bias = nn.Parameter(torch.zeros(self.qkvg.shape[0], dtype=dtype), requires_grad=False)   # zero under the gate
        self.q_norm, self.k_norm = _vec(self.nq, 1.0), _vec(self.nk, 1.0)
        self.o = _mat(width, self.n_out, dtype)

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.c.kv_heads, self.c.dim, self.c.vdim)

    def load(self, t: _Tensors, pre: str) -> None:
        W, off = self.qkvg.shape[1], 0
        for name, n in (("q", self.nq), ("k", self.nk), ("v", self.nv), ("g", self.n_out)):
            self.qkvg[off: off + n].copy_(t.take(pre + name, n, W))
            if name != "g":
                self.bias[off: off + n].copy_(t.take(f"{pre}{name}.b", n))
            off += n
        self.q_norm.copy_(t.take(pre + "q.norm", self.nq))
        self.k_norm.copy_(t.take(pre + "k.norm", self.nk))
        self.o.copy_(t.take(pre + "o", W, self.n_out))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c = self.c
        qkvg = linear(h, self.qkvg, self.bias)
        heads = hybrid.step_attention(step, cache, qkvg, c.heads, c.dim, c.vdim, c.scale, self.q_norm, self.k_norm, self.eps,
                                      c.temp_coef, c.temp_every)
        gated = hybrid.gate_heads(step, heads, qkvg[:, self.nq + self.nk + self.nv:], c.vdim)
        return linear(gated, self.o)


class RglruMixer(nn.Module):
    def __init__(self, c: RglruConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c = c
        n, W = c.width // c.blocks, c.width
        self.yx = _mat(2 * W, width, dtype)
        self.bias = nn.Parameter(torch.zeros(2 * W, dtype=dtype), requires_grad=False)
        self.taps, self.conv_bias = _vec((c.conv, W)), _vec(W)
        self.gate_w = nn.Parameter(torch.empty(c.blocks, 2, n, n, dtype=dtype), requires_grad=False)
        self.ra_bias, self.ri_bias = _vec(W), _vec(W)
        self.decay_base = _vec(W, -8.0)        # -8 softplus(lam): log a at r = 1
        self.o = _mat(width, W, dtype)

    def cache_spec(self) -> StateSpec:
        # the newest inputs of the convolution, row = position % taps
        return StateSpec((("S", (self.c.width,)), ("conv", (self.c.conv, self.c.width))))

    def load(self, t: _Tensors, pre: str) -> None:
        c, W, n, D = self.c, self.c.width, self.c.width // self.c.blocks, self.o.shape[0]
        for off, name in ((0, "y"), (W, "x")):
            self.yx[off: off + W].copy_(t.take(pre + name, W, D))
            self.bias[off: off + W].copy_(t.take(f"{pre}{name}.b", W))
        self.taps.copy_(t.take(pre + "conv", W, c.conv).t())
        self.conv_bias.copy_(t.take(pre + "conv.b", W))
        for j, (name, bias) in enumerate((("ra", self.ra_bias), ("ri", self.ri_bias))):
            self.gate_w[:, j].copy_(t.take(pre + name, c.blocks, n, n))
            bias.copy_(t.take(f"{pre}{name}.b", c.blocks, n).reshape(-1))
        self.decay_base.copy_(-8.0 * F.softplus(t.take(pre + "lam", W).double()))
        self.o.copy_(t.take(pre + "o", D, W))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        yx = linear(h, self.yx, self.bias)
        s = hybrid.rglru(step, yx, self.gate_w, self.taps, self.conv_bias, self.ra_bias, self.ri_bias, self.decay_base,
                         cache["S"], cache["conv"])
        return linear(s, self.o)


class LightningMixer(nn.Module):
    def __init__(self, c: LightningConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.nk, self.nv = c.heads * c.dim, c.heads * c.vdim
        self.qkvg = _mat(2 * self.nk + 2 * self.nv, width, dtype)
        self.decay = nn.Parameter(torch.tensor(c.decay, dtype=torch.float32), requires_grad=False)
        self.norm = _vec(self.nv, 1.0)
        self.o = _mat(width, self.nv, dtype)

    def cache_spec(self) -> StateSpec:
        return StateSpec((("S", (self.c.heads, self.c.dim, self.c.vdim)),))

    def load(self, t: _Tensors, pre: str) -> None:
        W, off = self.qkvg.shape[1], 0
        for name, n in (("q", self.nk), ("k", self.nk), ("v", self.nv), ("g", self.nv)):
            self.qkvg[off: off + n].copy_(t.take(pre + name, n, W))
            off += n
        self.norm.copy_(t.take(pre + "norm", self.nv))
        self.o.copy_(t.take(pre + "o", W, self.nv))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        qkvg = linear(h, self.qkvg)
        o = hybrid.lightning(step, qkvg, self.decay, cache["S"])
        return linear(hybrid.norm_gate(o, self.norm, qkvg[:, 2 * self.nk + self.nv:], self.eps), self.o)


_MIXERS = {AttentionConfig: AttentionMixer, RglruConfig: RglruMixer, LightningConfig: LightningMixer}


class GarupelLayer(nn.Module):
    """The weights of a layer; the residual stream and the norms around its sublayers are the model's business."""

    def __init__(self, c: LayerConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.mix = _MIXERS[type(c.mixer)](c.mixer, width, eps, dtype)
        self.norm1, self.norm1b = _vec(width, 1.0), _vec(width, 1.0)
        self.ff = c.ff
        if c.ff is not None:
            self.norm2, self.norm2b = _vec(width, 1.0), _vec(width, 1.0)
            self.up, self.down = _mat(c.ff, width, dtype), _mat(width, c.ff, dtype)

    def load(self, t: _Tensors, pre: str) -> None:
        W = self.norm1.shape[0]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if self.ff is not None else ()):
            getattr(self, n).copy_(t.take(pre + n, W))
        self.mix.load(t, pre + "mix.")
        if self.ff is not None:
            self.up.copy_(t.take(pre + "mlp.up", self.ff, W))
            self.down.copy_(t.take(pre + "mlp.down", W, self.ff))

    def mlp(self, h: torch.Tensor) -> torch.Tensor:
        return linear(hybrid.relu_squared_(linear(h, self.up)), self.down)


class GarupelModel(nn.Module):
    def __init__(self, config: GarupelConfig, dtype: torch.dtype):
        super().__init__()
        self.config, self.dtype = config, dtype
        self.embed = _mat(config.vocab_size, config.hidden_size, dtype)
        self.layers = nn.ModuleList([GarupelLayer(c, config.hidden_size, config.eps, dtype) for c in config.layers])
        self.norm = _vec(config.hidden_size, 1.0)
        self.runs = config.runs()

    def forward_step(self, step: Step, cache: HybridCacheManager) -> torch.Tensor:
        """Hidden rows behind the last norm, ``[n_tokens, width]`` in the step's token order."""
        eps = self.config.eps
        cache.begin_step(step)
        x = torch.empty(step.n_tokens, self.config.hidden_size, dtype=torch.float32, device=self.embed.device)
        first = self.layers[self.runs[0][0]] if self.runs else None
        h = hybrid.residual_norm(step, x, embed=self.embed, w_next=first.norm1 if first is not None else self.norm, eps=eps,
                                 restart=True)
        for r, (i, _) in enumerate(self.runs):
            lay = self.layers[i]
            y, post = lay.mix(h, step, cache[r]), lay.norm1b
            if lay.ff is not None:
                h = hybrid.residual_norm(step, x, y, post, w_next=lay.norm2, eps=eps)
                y, post = lay.mlp(h), lay.norm2b
            last = r + 1 == len(self.runs)
            again = not last and self.runs[r + 1][1]          # the next run opens another pass of the loop
            h = hybrid.residual_norm(step, x, y, post, embed=self.embed if again else None,
                                     w_next=self.norm if last else self.layers[self.runs[r + 1][0]].norm1, eps=eps)
        return h

    def forward_tokens(self, new_ids: torch.Tensor, kv_cache: HybridCacheManager, position_ids: torch.Tensor,
                       kv_start: Optional[torch.Tensor] = None, n_new: Optional[Sequence[int]] = None) -> torch.Tensor:
        """The padded form the generation loops call: ``new_ids`` [B, n] with ``n_new[b]`` (default n) tokens per
        row, positions as cached.  One token per row takes its position from ``position_ids`` on the device."""
        if kv_start is not None:
            raise NotImplementedError("left padding is not part of hybrid decoders: use ragged counts")
        B, n = new_ids.shape
        if n == 1 and n_new is None and new_ids.is_cuda and B == kv_cache.batch:
            step = kv_cache.decode_step()
            step.set_decode(new_ids.reshape(-1), position_ids.reshape(-1))
            return self.forward_step(step, kv_cache).view(B, 1, -1)
        counts = [n] * B if n_new is None else [int(c) for c in n_new]
        step = kv_cache.step(counts, new_ids, self.config.vocab_size, base=[b * n for b in range(B)])
        hidden = self.forward_step(step, kv_cache)
        out = torch.zeros(B, n, hidden.shape[1], dtype=hidden.dtype, device=hidden.device)
        entry = step.tok_entry.long()
        rows = torch.tensor(step.rows, device=hidden.device)[entry]
        out[rows, (step.tok_pos - step.start[entry]).long()] = hidden
        return out


class _Head(nn.Module):
    def __init__(self, vocab: int, width: int, dtype: torch.dtype):
        super().__init__()
        self.weight = _mat(vocab, width, dtype)


class GarupelForCausalLM(nn.Module):
    def __init__(self, config: GarupelConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__()
        # bf16 products accumulate in fp32 to the end; fp32 products stay out of the reduced-precision modes
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.config, self.dtype, self.vocab_size = config, dtype, config.vocab_size
        self.model = GarupelModel(config, dtype)
        self.lm_head = _Head(config.vocab_size, config.hidden_size, dtype)

    # -- weights and caches --------------------------------------------------------------------------
    @torch.no_grad()
    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        t, V, W = _Tensors(tensors), self.config.vocab_size, self.config.hidden_size
        self.model.embed.copy_(t.take("embed", V, W))
        for i, lay in enumerate(self.model.layers):
            lay.load(t, f"l{i}.")
        self.model.norm.copy_(t.take("final.norm", W))
        self.lm_head.weight.copy_(t.take("head", V, W))
        if t.unused():
            raise ValueError(f"checkpoint tensors without a place in the model: {t.unused()[:8]}")

    @torch.no_grad()
    def random_init_(self, seed: int, std: float = 0.02) -> "GarupelForCausalLM":
        """Synthetic weights: N(0, std) matrices, unit norms, a few taps and decays of ordinary size."""
        g = torch.Generator(device=self.lm_head.weight.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if p.dim() >= 2 or name.endswith("taps"):
                p.copy_(torch.randn(p.shape, generator=g, device=p.device) * (0.3 if name.endswith("taps") else std))
            elif name.endswith("decay_base"):
                p.copy_(-8.0 * F.softplus(torch.rand(p.shape, generator=g, device=p.device) * 4.0 - 6.0))
        return self

    def new_cache(self, batch: int, pool_tokens: int, max_seq_len: int,
                  cache_type: KVCacheType = KVCacheType.DYNAMIC) -> HybridCacheManager:
        """Pools and states for ``batch`` rows; called by the schedulers and generation loops."""
        specs = [self.model.layers[i].mix.cache_spec() for i, _ in self.model.runs]
        return HybridCacheManager(specs, batch, pool_tokens, max_seq_len, self.dtype, self.lm_head.weight.device, cache_type)

    # -- forward forms ---------------------------------------------------------------------------------
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits of hidden rows ``[n, width]``."""
        return hybrid.linear_f32(hidden, self.lm_head.weight)

    def forward_packed(self, tokens: torch.Tensor, counts: Sequence[int], kv_cache: HybridCacheManager,
                       rows: Optional[Sequence[int]] = None) -> ModelOutput:
        """``tokens`` [T]: the new tokens of every batch row back to back, ``counts[b]`` of them for row b.
        Returns the last new token's logits per row, ``[B, vocab]`` (zero for rows that sit out), or with ``rows``
        (places in ``tokens``) the logits of those."""
        step = kv_cache.step(counts, tokens, self.config.vocab_size)
        hidden = self.model.forward_step(step, kv_cache)
        dev = hidden.device
        if rows is not None:
            at, off = {}, 0                 # place in `tokens` -> row of the step (entries are ordered decode first)
            for b, c in enumerate(counts):
                if c:
                    at.update((off + j, step.first_row[b] + j) for j in range(c))
                off += c
            picked = torch.tensor([at[int(r)] for r in rows], dtype=torch.long, device=dev)
            return ModelOutput(logits=self.logits(hidden.index_select(0, picked)))
        live = self.logits(hidden.index_select(0, torch.tensor(step.last_rows, device=dev)))
        out = torch.zeros(len(counts), self.vocab_size, dtype=torch.float32, device=dev)
        out[torch.tensor(step.rows, device=dev)] = live
        return ModelOutput(logits=out)

    def forward_ragged(self, new_ids: torch.Tensor, n_new: Sequence[int], kv_cache: HybridCacheManager) -> ModelOutput:
        """``new_ids`` [B, n_max], left-aligned, ``n_new[b]`` tokens of row b; logits ``[B, n_max, vocab]``."""
        hidden = self.model.forward_tokens(new_ids, kv_cache, None, None, n_new)
        return ModelOutput(logits=self.logits(hidden.flatten(0, 1)).view(*new_ids.shape, -1))

    def forward(self, input_ids: torch.Tensor, kv_cache: HybridCacheManager, attention_mask: Optional[torch.Tensor] = None,
                inputs_embeds=None) -> ModelOutput:
        """The whole history; what the cache holds is sliced off.  Rows of one length, no padding."""
        if inputs_embeds is not None or (attention_mask is not None and bool((attention_mask == 0).any())):
            raise NotImplementedError("inputs_embeds and padded batches are not supported")
        new = input_ids[:, len(kv_cache):]
        return self.forward_ragged(new, [new.shape[1]] * new.shape[0], kv_cache)


model_registry.register("Garupel", lambda config, dtype: GarupelForCausalLM(GarupelConfig.from_dict(config), dtype),
                        dtypes=(torch.bfloat16, torch.float32))
