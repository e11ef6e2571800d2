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
from typing import List, Optional, Tuple, Union

import torch
import torch.nn.functional as F
from torch import nn

from pace_b200.llm.hybrid_cache import HybridCacheManager, KVSpec, StateSpec
from pace_b200.llm.models.step_decoder import CheckpointTensors, StepCausalLM, StepModel, mat, vec
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


class AttentionMixer(nn.Module):
    def __init__(self, c: AttentionConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.nq, self.nk, self.nv = c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim
        self.n_out = c.heads * c.vdim
        self.qkvg = mat(self.nq + self.nk + self.nv + self.n_out, width, dtype=dtype)
        self.bias = nn.Parameter(torch.zeros(self.qkvg.shape[0], dtype=dtype), requires_grad=False)   # zero under the gate
        self.q_norm, self.k_norm = vec(self.nq, 1.0), vec(self.nk, 1.0)
        self.o = mat(width, self.n_out, dtype=dtype)

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.c.kv_heads, self.c.dim, self.c.vdim)

    def load(self, t: CheckpointTensors, pre: str) -> None:
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
        self.yx = mat(2 * W, width, dtype=dtype)
        self.bias = nn.Parameter(torch.zeros(2 * W, dtype=dtype), requires_grad=False)
        self.taps, self.conv_bias = vec((c.conv, W)), vec(W)
        self.gate_w = nn.Parameter(torch.empty(c.blocks, 2, n, n, dtype=dtype), requires_grad=False)
        self.ra_bias, self.ri_bias = vec(W), vec(W)
        self.decay_base = vec(W, -8.0)        # -8 softplus(lam): log a at r = 1
        self.o = mat(width, W, dtype=dtype)

    def cache_spec(self) -> StateSpec:
        # the newest inputs of the convolution, row = position % taps
        return StateSpec((("S", (self.c.width,)), ("conv", (self.c.conv, self.c.width))))

    def load(self, t: CheckpointTensors, pre: str) -> None:
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
        self.qkvg = mat(2 * self.nk + 2 * self.nv, width, dtype=dtype)
        self.decay = nn.Parameter(torch.tensor(c.decay, dtype=torch.float32), requires_grad=False)
        self.norm = vec(self.nv, 1.0)
        self.o = mat(width, self.nv, dtype=dtype)

    def cache_spec(self) -> StateSpec:
        return StateSpec((("S", (self.c.heads, self.c.dim, self.c.vdim)),))

    def load(self, t: CheckpointTensors, pre: str) -> None:
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
        self.norm1, self.norm1b = vec(width, 1.0), vec(width, 1.0)
        self.ff = c.ff
        if c.ff is not None:
            self.norm2, self.norm2b = vec(width, 1.0), vec(width, 1.0)
            self.up, self.down = mat(c.ff, width, dtype=dtype), mat(width, c.ff, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        W = self.norm1.shape[0]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if self.ff is not None else ()):
            getattr(self, n).copy_(t.take(pre + n, W))
        self.mix.load(t, pre + "mix.")
        if self.ff is not None:
            self.up.copy_(t.take(pre + "mlp.up", self.ff, W))
            self.down.copy_(t.take(pre + "mlp.down", W, self.ff))

    def mlp(self, h: torch.Tensor) -> torch.Tensor:
        return linear(hybrid.relu_squared_(linear(h, self.up)), self.down)


class GarupelModel(StepModel):
    def __init__(self, config: GarupelConfig, dtype: torch.dtype):
        super().__init__()
        self.config, self.dtype = config, dtype
        self.embed = mat(config.vocab_size, config.hidden_size, dtype=dtype)
        self.layers = nn.ModuleList([GarupelLayer(c, config.hidden_size, config.eps, dtype) for c in config.layers])
        self.norm = vec(config.hidden_size, 1.0)
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

    def cache_specs(self) -> list:
        return [self.layers[i].mix.cache_spec() for i, _ in self.runs]


class GarupelForCausalLM(StepCausalLM):
    def __init__(self, config: GarupelConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, GarupelModel(config, dtype), dtype)

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


model_registry.register("Garupel", lambda config, dtype: GarupelForCausalLM(GarupelConfig.from_dict(config), dtype),
                        dtypes=(torch.bfloat16, torch.float32))
