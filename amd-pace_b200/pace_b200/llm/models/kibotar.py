"""Kibotar: a decoder whose layers mix softmax attention over a window and pooled blocks (weights mixed over the heads), gated linear
attention and latent attention without positions; mixers read inputs shifted towards the previous token's, norms stand on both sides of
every sublayer, a stretch of layers runs several times, and a table of token pairs is added to the embeddings.

Everything runs on a packed ``Step`` of tokens.  Between two layers one kernel takes up the sublayer's output (normalised) and the
vector of a loop pass, normalises the stream and shifts the norm; between a mixer and its feed-forward the same without shift.  Per
mixer the launches are

    attention         one projection (q, k, v, gate) -> rotation + append + means of completed blocks (prompts: a launch of their own)
                      -> attention with mixed heads and output gate -> W_o
    gla               one projection (q, k, v, gate, inner half of the decay) -> outer half -> recurrence, norm and gate (decode: one
                      launch) -> W_o
    latent attention  one projection (q, latent, gate; prompts: two) -> norm + append -> absorbed or expanded attention -> gate -> W_o

A layer run (layer i in pass p) has its own rows, state and previous input; the weights of a layer are shared by its runs.
"""
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union

import torch
from torch import nn

from pace_b200.llm.hybrid_cache import BlockSpec, HybridCacheManager, JointSpec, KVSpec, LatentSpec, StateSpec
from pace_b200.llm.models.step_decoder import CheckpointTensors, StepCausalLM, StepModel, mat, vec
from pace_b200.llm.registry import model_registry
from pace_b200.llm.step import Step
from pace_b200.ops import hybrid
from pace_b200.ops.linear import linear
from pace_b200.ops.rotary_embedding import RotaryEmbedding


@dataclass(frozen=True)
class ScalingConfig:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    block: int
    rot_dims: int
    rot_base: float
    scaling: Optional[ScalingConfig]


@dataclass(frozen=True)
class GlaConfig:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[AttentionConfig, GlaConfig, LatentConfig]
    ff: Optional[int]         # None: the layer has no feed-forward


def _mixer_config(kind: str, m: dict):
    if kind == "attention":
        rot, mask = m["rot"], m["mask"]
        s = rot.get("scaling")
        scaling = ScalingConfig(float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"])) if s else None
        c = AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), mask["size"], mask["pool"], rot["dims"],
                            float(rot["base"]), scaling)
        if c.heads % c.kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if c.rot_dims % 2 or not 0 <= c.rot_dims <= c.dim:
            raise ValueError("rotated dimensions come in pairs within a head")
        if c.window < 1 or c.block < 1:
            raise ValueError("a window and a block hold at least one token")
        return c
    if kind == "gla":
        c = GlaConfig(m["heads"], m["dim"], m["vdim"], float(m["tau"]))
        if not c.tau > 0:
            raise ValueError("the root of a decay must be positive")
        return c
    if kind == "latent_attention":
        return LatentConfig(m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"]))
    raise ValueError(f"unknown mixer type {kind!r}")


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class KibotarConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerConfig, ...]
    eps: float
    embedding_scale: float = 1.0
    bigram: Optional[BigramConfig] = None
    loop: Optional[Tuple[int, int, int]] = None    # layers start .. stop - 1 run `times` times in a row, each time behind a vector

    @staticmethod
    def from_dict(c: dict) -> "KibotarConfig":
        layers = []
        for lay in c["layers"]:
            mlp = lay.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            layers.append(LayerConfig(_mixer_config(lay["type"], lay["mixer"]), mlp["ff"] if mlp is not None else None))
        e, lp = c["embedding"], c.get("loop")
        b = e.get("bigram")
        bigram = BigramConfig(b["buckets"], b["mul_prev"], b["mul_cur"]) if b else None
        if bigram is not None and bigram.buckets < 1:
            raise ValueError("a table of token pairs needs a bucket")
        loop = (lp["start"], lp["stop"], lp["times"]) if lp else None
        if loop is not None and (not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1):
            raise ValueError("loop must name a range of layers and a positive count")
        return KibotarConfig(c["vocab"], c["width"], tuple(layers), float(c["norm"]["eps"]), float(e.get("scale", 1.0)), bigram, loop)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, number of the pass it opens or None) in execution order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(start)]
        for t in range(times):
            out += [(i, t if i == start else None) for i in range(start, stop)]
        return out + [(i, None) for i in range(stop, n)]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs())


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


class AttentionMixer(nn.Module):
    def __init__(self, c: AttentionConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c = c
        self.parts = (("q", c.heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.kv_heads * c.vdim))
        self.n_out = c.heads * c.vdim
        self.gate_at = _up8(sum(n for _, n in self.parts))             # the gate's columns begin at 16 bytes
        self.qkvg = mat(self.gate_at + self.n_out, width, dtype=dtype)
        self.bias = nn.Parameter(torch.zeros(self.qkvg.shape[0], dtype=dtype), requires_grad=False)     # zero under the gate
        self.talk = vec((c.heads, c.heads))
        self.sinks = vec(c.heads)                                      # one added to the denominator: a score of 0
        self.o, self.out_bias = mat(width, self.n_out, dtype=dtype), vec(width)
        self.tables = None

    def cache_spec(self) -> JointSpec:
        c = self.c
        return JointSpec((KVSpec(c.kv_heads, c.dim, c.vdim), BlockSpec(c.kv_heads, c.dim, c.vdim, c.block)))

    def prepare(self, max_seq_len: int) -> None:
        """Rotation tables for every position of the longest sequence."""
        c, s = self.c, self.c.scaling
        if c.rot_dims and (self.tables is None or self.tables[0].shape[0] < max_seq_len):
            kind = {"rope_type": "precise"} if s is None else {
                "rope_type": "llama3_precise", "factor": s.factor, "low_freq_factor": s.low, "high_freq_factor": s.high,
                "original_max_position_embeddings": s.original}
            self.tables = RotaryEmbedding(kind, c.rot_dims, max_seq_len, c.rot_base).device_tables(self.qkvg.device)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        W, off = self.qkvg.shape[1], 0
        self.qkvg.zero_()
        for name, n in self.parts:
            self.qkvg[off: off + n].copy_(t.take(pre + name, n, W))
            self.bias[off: off + n].copy_(t.take(f"{pre}{name}.b", n))
            off += n
        self.qkvg[self.gate_at:].copy_(t.take(pre + "g", self.n_out, W))
        self.talk.copy_(t.take(pre + "talk", self.c.heads, self.c.heads))
        self.o.copy_(t.take(pre + "o", W, self.n_out))
        self.out_bias.copy_(t.take(pre + "o.b", W))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c, p = self.c, linear(h, self.qkvg, self.bias)
        heads = hybrid.pooled_attention(step, cache[0], cache[1], p, self.tables, c.heads, c.dim, c.vdim, c.scale, c.window, c.block,
                                        self.sinks, self.talk, p[:, self.gate_at:])
        return linear(heads, self.o)


class GlaMixer(nn.Module):
    def __init__(self, c: GlaConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps, self.dtype, self.width = c, eps, dtype, width
        self.parts = (("q", c.heads * c.dim), ("k", c.heads * c.dim), ("v", c.heads * c.vdim))
        self.n_out, self.out_bias = c.heads * c.vdim, None
        self.gate_at = _up8(sum(n for _, n in self.parts))
        self.low_at = self.gate_at + _up8(self.n_out)
        self.z_bias, self.norm = vec(c.heads * c.dim), vec(c.vdim, 1.0)
        self.o = mat(width, self.n_out, dtype=dtype)
        self.set_rank(16)

    def set_rank(self, rank: int) -> None:
        """The inner size of the decay's low-rank projection, which only a checkpoint's shapes name."""
        self.rank = rank
        with torch.device(self.z_bias.device):
            self.proj = mat(self.low_at + _up8(rank), self.width, dtype=self.dtype)
            self.up = mat(self.c.heads * self.c.dim, _up8(rank), dtype=self.dtype)

    def cache_spec(self) -> StateSpec:
        return StateSpec((("S", (self.c.heads, self.c.dim, self.c.vdim)),))

    def prepare(self, max_seq_len: int) -> None:
        pass

    def load(self, t: CheckpointTensors, pre: str) -> None:
        c, W, off = self.c, self.width, 0
        rank = t.shape(pre + "a1")[0]
        if rank != self.rank:
            self.set_rank(rank)
        self.proj.zero_()
        self.up.zero_()
        for name, n in self.parts:
            self.proj[off: off + n].copy_(t.take(pre + name, n, W))
            off += n
        self.proj[self.gate_at: self.gate_at + self.n_out].copy_(t.take(pre + "g", self.n_out, W))
        self.proj[self.low_at: self.low_at + rank].copy_(t.take(pre + "a1", rank, W))
        self.up[:, :rank].copy_(t.take(pre + "a2", c.heads * c.dim, rank))
        self.z_bias.copy_(t.take(pre + "a2.b", c.heads * c.dim))
        self.norm.copy_(t.take(pre + "norm", c.vdim))
        self.o.copy_(t.take(pre + "o", W, self.n_out))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c, p = self.c, linear(h, self.proj)
        z = linear(p[:, self.low_at:], self.up)
        heads = hybrid.gla(step, p, z, self.z_bias, cache["S"], self.norm, p[:, self.gate_at: self.gate_at + self.n_out], c.tau,
                           c.dim ** -0.5, self.eps)
        return linear(heads, self.o)


class LatentMixer(nn.Module):
    def __init__(self, c: LatentConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        self.nq, self.out_bias = c.heads * c.dim, None
        self.down_at = _up8(self.nq)                                   # rows of the projection: q | latent | gate
        self.gate_at = self.down_at + _up8(c.kv_rank)
        self.proj = mat(self.gate_at + _up8(c.heads), width, dtype=dtype)
        self.kv_norm = vec(c.kv_rank, 1.0)
        self.ukv = mat(c.heads * (c.dim + c.vdim), c.kv_rank, dtype=dtype)      # keys of all heads, then values
        self.o = mat(width, c.heads * c.vdim, dtype=dtype)

    def cache_spec(self) -> LatentSpec:
        return LatentSpec(self.c.kv_rank, 0)

    def prepare(self, max_seq_len: int) -> None:
        pass

    def load(self, t: CheckpointTensors, pre: str) -> None:
        c, W = self.c, self.proj.shape[1]
        self.proj.zero_()
        self.proj[: self.nq].copy_(t.take(pre + "q", self.nq, W))
        self.proj[self.down_at: self.down_at + c.kv_rank].copy_(t.take(pre + "dkv", c.kv_rank, W))
        self.proj[self.gate_at: self.gate_at + c.heads].copy_(t.take(pre + "g", c.heads, W))
        self.kv_norm.copy_(t.take(pre + "dkv.norm", c.kv_rank))
        self.ukv[: self.nq].copy_(t.take(pre + "uk", self.nq, c.kv_rank))
        self.ukv[self.nq:].copy_(t.take(pre + "uv", c.heads * c.vdim, c.kv_rank))
        self.o.copy_(t.take(pre + "o", W, c.heads * c.vdim))

    def forward(self, h: torch.Tensor, step: Step, cache) -> torch.Tensor:
        c, at = self.c, self.down_at
        if step.decode_only:
            p = linear(h, self.proj)
            q, rest = p[:, : self.nq], p[:, at:]
        else:                                    # dense queries for the prompt kernel
            q, rest = linear(h, self.proj[: self.nq]), linear(h, self.proj[at:])
        heads = hybrid.latent_attention(step, cache, rest, None, self.kv_norm, None, self.ukv, c.heads, c.dim, 0, c.vdim, c.scale,
                                        self.eps, None, q=q)
        return linear(hybrid.gate_per_head_(heads, rest[:, self.gate_at - at:], c.heads), self.o)


_MIXERS = {AttentionConfig: AttentionMixer, GlaConfig: GlaMixer, LatentConfig: LatentMixer}


class KibotarLayer(nn.Module):
    """The weights of a layer; the residual stream and the norms around its sublayers are the model's business."""

    def __init__(self, c: LayerConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.mix = _MIXERS[type(c.mixer)](c.mixer, width, eps, dtype)
        self.norm1, self.norm1b, self.shift = vec(width, 1.0), vec(width, 1.0), vec(width)
        self.ff = c.ff
        if c.ff is not None:
            self.norm2, self.norm2b = vec(width, 1.0), vec(width, 1.0)
            self.up, self.down = mat(c.ff, width, dtype=dtype), mat(width, c.ff, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str) -> None:
        W = self.norm1.shape[0]
        for n in ("norm1", "norm1b", "shift") + (("norm2", "norm2b") if self.ff is not None else ()):
            getattr(self, n).copy_(t.take(pre + n, W))
        self.mix.load(t, pre + "mix.")
        if self.ff is not None:
            self.up.copy_(t.take(pre + "mlp.up", self.ff, W))
            self.down.copy_(t.take(pre + "mlp.down", W, self.ff))

    def mlp(self, h: torch.Tensor) -> torch.Tensor:
        return linear(hybrid.relu_squared_(linear(h, self.up)), self.down)


class KibotarModel(StepModel):
    def __init__(self, config: KibotarConfig, dtype: torch.dtype):
        super().__init__()
        self.config, self.dtype = config, dtype
        W = config.hidden_size
        self.embed = mat(config.vocab_size, W, dtype=dtype)
        self.bigram = mat(config.bigram.buckets + 1, W, dtype=dtype) if config.bigram is not None else None
        self.steps = vec((config.loop[2], W)) if config.loop is not None else None
        self.layers = nn.ModuleList([KibotarLayer(c, W, config.eps, dtype) for c in config.layers])
        self.norm = vec(W, 1.0)
        self.runs = config.runs()

    def cache_specs(self) -> list:
        """One per layer run, and what the model remembers: every run's newest mixer input (in front of the shift; twice, since the
        one of the step before is read while that of this step is written) and the newest token."""
        n, W = max(1, len(self.runs)), self.config.hidden_size
        return [self.layers[i].mix.cache_spec() for i, _ in self.runs] + [
            JointSpec((StateSpec((("h", (n, W)), ("next", (n, W)))), StateSpec((("token", ()),), torch.int32)))]

    def prepare(self, max_seq_len: int) -> None:
        for lay in self.layers:
            lay.mix.prepare(max_seq_len)

    def forward_step(self, step: Step, cache: HybridCacheManager) -> torch.Tensor:
        c, eps = self.config, self.config.eps
        cache.begin_step(step)
        shifts, tokens = cache[len(self.runs)]
        before, token = shifts["h"], tokens["token"] if self.bigram is not None else None
        after = before if step.decode_only else shifts["next"]
        b = c.bigram
        x = hybrid.embed_pairs(step, self.embed, c.embedding_scale, self.bigram, token, b.mul_prev if b else 0, b.mul_cur if b else 0)
        y = post = bias = spare = None
        for r, (i, opens) in enumerate(self.runs):
            lay = self.layers[i]
            new, h = hybrid.shift_norm(step, x, lay.norm1, lay.shift, before[:, r], after[:, r], eps, self.dtype, y, bias, post,
                                       self.steps[opens] if opens is not None else None, spare)
            if new is not x:
                x, spare = new, x
            y, post, bias = lay.mix(h, step, cache[r]), lay.norm1b, lay.mix.out_bias
            if lay.ff is not None:
                h = hybrid.residual_norm(step, x, y, post, w_next=lay.norm2, eps=eps, bias=bias)
                y, post, bias = lay.mlp(h), lay.norm2b, None
        h = hybrid.residual_norm(step, x, y, post, w_next=self.norm, eps=eps, bias=bias, dtype=self.dtype)
        if not step.decode_only:
            hybrid.state_commit(step, after, before, token)
        return h


class KibotarForCausalLM(StepCausalLM):
    def __init__(self, config: KibotarConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, KibotarModel(config, dtype), dtype)
        self.lm_head.weight = self.model.embed           # one table reads tokens and makes logits

    def load_head(self, t: CheckpointTensors) -> None:
        m, W = self.model, self.config.hidden_size
        if m.bigram is not None:
            m.bigram.copy_(t.take("bigram", *m.bigram.shape))
        if m.steps is not None:
            m.steps.copy_(t.take("loop.step", self.config.loop[2], W))

    @torch.no_grad()
    def random_init_(self, seed: int, std: float = 0.02) -> "KibotarForCausalLM":
        """Synthetic weights: N(0, std) matrices, unit norms, shifts between 0 and 1, decays of ordinary size, heads mixed a little."""
        g = torch.Generator(device=self.lm_head.weight.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if name.endswith("talk"):
                p.copy_(torch.eye(p.shape[0], device=p.device) + torch.randn(p.shape, generator=g, device=p.device) * 0.1)
            elif name.endswith("shift"):
                p.copy_(torch.rand(p.shape, generator=g, device=p.device))
            elif name.endswith("z_bias"):
                p.copy_(torch.rand(p.shape, generator=g, device=p.device) * 4.0)
            elif p.dim() >= 2:
                p.copy_(torch.randn(p.shape, generator=g, device=p.device) * std)
        return self


model_registry.register("Kibotar", lambda config, dtype: KibotarForCausalLM(KibotarConfig.from_dict(config), dtype),
                        dtypes=(torch.bfloat16, torch.float32))
