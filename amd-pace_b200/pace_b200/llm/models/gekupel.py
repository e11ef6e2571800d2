"""Gekupel: a decoder whose layers mix attention over chunks of the sequence (keys and queries normalised per head, a
distance bias, a sink) with two kinds of latent attention over a sliding window (with and without YaRN and a sink), dense
or mixture-of-experts feed-forwards, and norms behind the sublayers only.

Everything runs on a packed ``Step`` of tokens.  Sublayers read the fp32 residual stream itself (rounded to the activations'
type); behind a sublayer one kernel normalises its output - for a mixture it first sums the chosen experts' rows - and
adds it.  Per mixer the launches are

    attention         one projection (q, k, v) -> norms + append -> attention -> W_o
    latent attention  one down projection (query latent, key/value latent, rotated key) -> norms + rotation + append ->
                      query up projection -> absorbed or expanded attention (``ops.hybrid.latent_attention``) -> W_o

A layer that uses another one's weights is the same module, with a cache of its own.
"""
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch
from torch import nn

from pace_b200 import _C
from pace_b200.llm.hybrid_cache import HybridCacheManager, KVSpec, LatentSpec
from pace_b200.llm.models.step_decoder import CheckpointTensors, StepCausalLM, StepModel, mat, vec
from pace_b200.llm.registry import model_registry
from pace_b200.llm.step import Step
from pace_b200.ops import hybrid
from pace_b200.ops.linear import linear
from pace_b200.ops.rotary_embedding import RotaryEmbedding


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]


@dataclass(frozen=True)
class YarnConfig:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: Optional[int]
    rot_dims: int              # rotated dimensions of the rot_dim part
    rot_base: float
    yarn: Optional[YarnConfig]
    sink: bool


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[AttentionConfig, LatentConfig]
    mlp: Union[DenseConfig, MoeConfig, None]
    weights_of: Optional[int] = None      # the layer whose weights this one uses


def _size(m: dict) -> Optional[int]:
    size = (m.get("mask") or {}).get("size")
    if size is not None and size < 1:
        raise ValueError("a mask needs a positive size")
    return size


def _mixer_config(kind: str, m: dict):
    if kind == "attention":
        c = AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), _size(m))
        if c.heads % c.kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        return c
    if kind in ("latent_attention", "latent_attention_2"):
        rot, second = m["rot"], kind == "latent_attention_2"
        y = rot.get("scaling")
        yarn = YarnConfig(float(y["factor"]), float(y["original"]), float(y["fast"]), float(y["slow"])) if y else None
        c = LatentConfig(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), _size(m),
                         rot["dims"], float(rot["base"]), yarn, second)
        if c.rot_dims % 2 or c.rot_dims > c.rot_dim:
            raise ValueError("rotated dimensions come in pairs within rot_dim")
        return c
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp_config(m: Optional[dict]):
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseConfig(m["ff"])
    if m["kind"] == "moe":
        c = MoeConfig(m["expert"]["ff"], m["router"]["experts"], m["router"]["top"])
        if not 1 <= c.top <= c.experts:
            raise ValueError("a router chooses between one and all of its experts")
        return c
    raise ValueError(f"unknown feed-forward kind {m['kind']!r}")


@dataclass(frozen=True)
class GekupelConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerConfig, ...]
    eps: float
    embedding_scale: float

    @staticmethod
    def from_dict(c: dict) -> "GekupelConfig":
        layers = []
        for i, lay in enumerate(c["layers"]):
            of = lay.get("weights_of")
            layers.append(LayerConfig(_mixer_config(lay["type"], lay["mixer"]), _mlp_config(lay.get("mlp")), of))
            if of is not None:
                seen = set()
                while of != i and of is not None and 0 <= of < len(c["layers"]) and of not in seen:
                    seen.add(of)
                    last, of = of, c["layers"][of].get("weights_of")
                if of is not None:
                    raise ValueError(f"layer {i}: weights_of does not lead to a layer with weights")
                layers[-1] = LayerConfig(layers[-1].mixer, layers[-1].mlp, last)
        for i, lay in enumerate(layers):
            if lay.weights_of is not None and (lay.mixer, lay.mlp) != (layers[lay.weights_of].mixer, layers[lay.weights_of].mlp):
                raise ValueError(f"layer {i} differs from layer {lay.weights_of}, whose weights it uses")
        return GekupelConfig(c["vocab"], c["width"], tuple(layers), float(c["norm"]["eps"]), float(c["embedding"]["scale"]))

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


class AttentionMixer(nn.Module):
    def __init__(self, c: AttentionConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.parts = (("q", c.heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.kv_heads * c.vdim))
        self.qkv = mat(sum(n for _, n in self.parts), width, dtype=dtype)
        self.sink = vec(c.heads)
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / c.heads) for h in range(c.heads)], dtype=torch.float64)
        self.slopes = nn.Parameter(slopes.float(), requires_grad=False)
        self.o = mat(width, c.heads * c.vdim, dtype=dtype)

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.c.kv_heads, self.c.dim, self.c.vdim)

    def prepare(self, max_seq_len: int) -> None:
        pass

    def load(self, t: CheckpointTensors, pre: str) -> None:
        W, off = self.qkv.shape[1], 0
        for name, n in self.parts:
            self.qkv[off: off + n].copy_(t.take(pre + name, n, W))
            off += n
        self.sink.copy_(t.take(pre + "sink", self.c.heads))
        self.o.copy_(t.take(pre + "o", *self.o.shape))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c = self.c
        heads = hybrid.span_attention(step, cache, linear(h, self.qkv), c.heads, c.dim, c.vdim, c.scale, self.eps, chunk=c.chunk,
                                      slopes=self.slopes, sinks=self.sink)
        return linear(heads, self.o)


class LatentMixer(nn.Module):
    def __init__(self, c: LatentConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.down = mat(c.q_rank + c.kv_rank + c.rot_dim, width, dtype=dtype)
        self.q_norm, self.kv_norm = vec(c.q_rank, 1.0), vec(c.kv_rank, 1.0)
        self.uq = mat(c.heads * (c.dim + c.rot_dim), c.q_rank, dtype=dtype)
        self.ukv = mat(c.heads * (c.dim + c.vdim), c.kv_rank, dtype=dtype)      # keys of all heads, then values
        if c.sink:
            self.sink = vec(c.heads)
        self.o = mat(width, c.heads * c.vdim, dtype=dtype)
        self.tables = None

    def cache_spec(self) -> LatentSpec:
        return LatentSpec(self.c.kv_rank, self.c.rot_dim)

    def prepare(self, max_seq_len: int) -> None:
        """Rotation tables for every position of the longest sequence."""
        if self.tables is not None and self.tables[0].shape[0] >= max_seq_len:
            return
        y = self.c.yarn
        kind = {"rope_type": "precise"} if y is None else {
            "rope_type": "yarn", "factor": y.factor, "original_max_position_embeddings": y.original, "beta_fast": y.fast,
            "beta_slow": y.slow}
        rope = RotaryEmbedding(kind, self.c.rot_dims, max_seq_len, self.c.rot_base, is_neox_style=False)
        self.tables = rope.device_tables(self.down.device)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        c, W = self.c, self.down.shape[1]
        self.down[: c.q_rank].copy_(t.take(pre + "dq", c.q_rank, W))
        self.down[c.q_rank:].copy_(t.take(pre + "dkv", c.kv_rank + c.rot_dim, W))
        self.q_norm.copy_(t.take(pre + "dq.norm", c.q_rank))
        self.kv_norm.copy_(t.take(pre + "dkv.norm", c.kv_rank))
        self.uq.copy_(t.take(pre + "uq", *self.uq.shape))
        n = c.heads * c.dim
        self.ukv[:n].copy_(t.take(pre + "uk", n, c.kv_rank))
        self.ukv[n:].copy_(t.take(pre + "uv", c.heads * c.vdim, c.kv_rank))
        if c.sink:
            self.sink.copy_(t.take(pre + "sink", c.heads))
        self.o.copy_(t.take(pre + "o", *self.o.shape))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c = self.c
        heads = hybrid.latent_attention(step, cache, linear(h, self.down), self.q_norm, self.kv_norm, self.uq, self.ukv, c.heads,
                                        c.dim, c.rot_dim, c.vdim, c.scale, self.eps, self.tables, window=c.window,
                                        sinks=self.sink if c.sink else None)
        return linear(heads, self.o)


class DenseMlp(nn.Module):
    def __init__(self, c: DenseConfig, width: int, dtype: torch.dtype):
        super().__init__()
        self.ff = c.ff
        self.gate_up, self.down = mat(2 * c.ff, width, dtype=dtype), mat(width, c.ff, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        W = self.down.shape[0]
        self.gate_up[: self.ff].copy_(t.take(pre + "gate", self.ff, W))
        self.gate_up[self.ff:].copy_(t.take(pre + "up", self.ff, W))
        self.down.copy_(t.take(pre + "down", W, self.ff))

    def forward(self, h: torch.Tensor, cache):
        return linear(hybrid.glu(linear(h, self.gate_up), _C.ACT_GELU_TANH), self.down), None


class MoeMlp(nn.Module):
    def __init__(self, c: MoeConfig, width: int, dtype: torch.dtype):
        super().__init__()
        self.c = c
        self.router, self.correction = mat(c.experts, width, dtype=dtype), vec(c.experts)
        self.gate_up = mat(c.experts, 2 * c.ff, width, dtype=dtype)
        self.down = mat(c.experts, width, c.ff, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        c, W = self.c, self.router.shape[1]
        self.router.copy_(t.take(pre + "router", c.experts, W))
        self.correction.copy_(t.take(pre + "correction", c.experts))
        for e in range(c.experts):
            self.gate_up[e, : c.ff].copy_(t.take(f"{pre}e{e}.gate", c.ff, W))
            self.gate_up[e, c.ff:].copy_(t.take(f"{pre}e{e}.up", c.ff, W))
            self.down[e].copy_(t.take(f"{pre}e{e}.down", W, c.ff))

    def forward(self, h: torch.Tensor, cache):
        """Returns the router's choice with the experts' rows; the kernel behind sums them up."""
        routed = hybrid.moe_route(h, self.router, self.correction, self.c.top)
        return None, hybrid.moe_experts(h, routed, self.gate_up, self.down, _C.ACT_SILU, cache.pool.status_word())


_MIXERS = {AttentionConfig: AttentionMixer, LatentConfig: LatentMixer}
_MLPS = {DenseConfig: DenseMlp, MoeConfig: MoeMlp}


class GekupelLayer(nn.Module):
    """The weights of a layer; the residual stream and the norms behind its sublayers are the model's business."""

    def __init__(self, c: LayerConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.mix = _MIXERS[type(c.mixer)](c.mixer, width, eps, dtype)
        self.norm1 = vec(width, 1.0)
        self.mlp = None
        if c.mlp is not None:
            self.mlp, self.norm2 = _MLPS[type(c.mlp)](c.mlp, width, dtype), vec(width, 1.0)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        self.norm1.copy_(t.take(pre + "norm1", self.norm1.shape[0]))
        self.mix.load(t, pre + "mix.")
        if self.mlp is not None:
            self.norm2.copy_(t.take(pre + "norm2", self.norm2.shape[0]))
            self.mlp.load(t, pre + "mlp.")


class GekupelModel(StepModel):
    def __init__(self, config: GekupelConfig, dtype: torch.dtype):
        super().__init__()
        self.config, self.dtype = config, dtype
        self.embed = mat(config.vocab_size, config.hidden_size, dtype=dtype)
        layers = [GekupelLayer(c, config.hidden_size, config.eps, dtype) if c.weights_of is None else None for c in config.layers]
        self.layers = nn.ModuleList([lay if lay is not None else layers[c.weights_of] for lay, c in zip(layers, config.layers)])
        self.norm = vec(config.hidden_size, 1.0)

    def cache_specs(self) -> list:
        return [lay.mix.cache_spec() for lay in self.layers]

    def prepare(self, max_seq_len: int) -> None:
        for lay in self.layers:
            lay.mix.prepare(max_seq_len)

    def forward_step(self, step: Step, cache: HybridCacheManager) -> torch.Tensor:
        eps, n = self.config.eps, len(self.layers)
        cache.begin_step(step)
        x = torch.empty(step.n_tokens, self.config.hidden_size, dtype=torch.float32, device=self.embed.device)
        h = hybrid.residual_norm(step, x, embed=self.embed, embed_scale=self.config.embedding_scale, restart=True, eps=eps,
                                 plain=n > 0, w_next=None if n else self.norm)
        for i, lay in enumerate(self.layers):
            last = i + 1 == n
            y = lay.mix(h, step, cache[i])
            final = last and lay.mlp is None
            h = hybrid.residual_norm(step, x, y, lay.norm1, w_next=self.norm if final else None, eps=eps, plain=not final)
            if lay.mlp is not None:
                y, routed = lay.mlp(h, cache[i])
                h = hybrid.residual_norm(step, x, y, lay.norm2, w_next=self.norm if last else None, eps=eps, plain=not last,
                                         routed=routed)
        return h


class GekupelForCausalLM(StepCausalLM):
    def __init__(self, config: GekupelConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, GekupelModel(config, dtype), dtype)

    @torch.no_grad()
    def random_init_(self, seed: int, std: float = 0.02) -> "GekupelForCausalLM":
        """Synthetic weights: N(0, std) matrices, unit norms, small sinks and corrections."""
        g = torch.Generator(device=self.lm_head.weight.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if p.dim() >= 2 or name.endswith(("sink", "correction")):
                p.copy_(torch.randn(p.shape, generator=g, device=p.device) * std)
        return self


model_registry.register("Gekupel", lambda config, dtype: GekupelForCausalLM(GekupelConfig.from_dict(config), dtype),
                        dtypes=(torch.bfloat16, torch.float32))
