"""Lesosun: a decoder whose layers are softmax attention beside a state-space recurrence (both behind short convolutions), or a
gated delta rule with a decay per key channel; a layer's mixer and its feed-forward (dense, or a mixture of experts with identity
experts and a shared one) read two norms of the same residual stream and are added to it together.

Everything runs on a packed ``Step`` of tokens.  Between two layers one kernel takes up everything the first one made - its
product, the chosen experts' rows, the output bias - into the fp32 stream and makes both norms of the second one.  Whatever a layer
multiplies by an output matrix (attention heads, gated state-space outputs, feed-forward activations) lies side by side in one
buffer, so that one product with the matrices side by side is the sum of them all, in fp32 accumulators.  The factors of the two
mixers are in the cached values and in the weight of the state-space norm.  Per mixer the launches are

    parallel       one projection (q, k, v, x, B, C, z, dt) -> convolutions + norms + rotation + append -> attention
                   -> convolution + recurrence (decode: one launch) -> gate and norms
    channel_delta  one projection (q, k, v, beta, the low-rank halves) -> decay and gate -> convolutions + recurrence
                   (decode: one launch) -> norms and gate
"""
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union

import torch
from torch import nn

from pace_b200 import _C
from pace_b200.llm.hybrid_cache import HybridCacheManager, JointSpec, KVSpec, StateSpec
from pace_b200.llm.models.step_decoder import CheckpointTensors, StepCausalLM, StepModel, mat, vec
from pace_b200.llm.registry import model_registry
from pace_b200.llm.step import Step
from pace_b200.ops import hybrid
from pace_b200.ops.linear import linear
from pace_b200.ops.rotary_embedding import RotaryEmbedding

UNIT_EPS = 1e-6          # of the delta rule's unit vectors


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    conv: int
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class SsdConfig:
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: SsdConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    ff: int
    experts: int
    identity: int
    top: int
    scale: float
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[ParallelConfig, DeltaConfig]
    mlp: Union[DenseConfig, MoeConfig, None]


def _mixer_config(kind: str, m: dict):
    if kind == "parallel":
        a, r = m["left"], m["right"]
        left = AttentionConfig(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), float(a["softcap"]), a["conv"],
                               a["rot"]["dims"], float(a["rot"]["base"]))
        right = SsdConfig(r["heads"], r["groups"], r["state"], r["vdim"], r["conv"], r["norm_groups"])
        if left.heads % left.kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if left.rot_dims % 2 or not 0 <= left.rot_dims <= left.dim:
            raise ValueError("rotated dimensions come in pairs within a head")
        if not left.softcap > 0:
            raise ValueError("the cap of the scores must be positive")
        if right.heads % right.groups or (right.heads * right.vdim) % right.norm_groups:
            raise ValueError("heads must be a multiple of groups, the inner width one of the norm's groups")
        if left.conv < 1 or right.conv < 1:
            raise ValueError("a convolution needs at least one tap")
        return ParallelConfig(left, right, float(m["left_scale"]), float(m["right_scale"]))
    if kind == "channel_delta":
        c = DeltaConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
        if c.heads % c.kv_heads:
            raise ValueError("heads must be a multiple of key heads")
        if c.conv < 1:
            raise ValueError("a convolution needs at least one tap")
        return c
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp_config(m: Optional[dict]):
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseConfig(m["ff"])
    if m["kind"] == "moe":
        r, shared = m["router"], m.get("shared")
        c = MoeConfig(m["expert"]["ff"], r["experts"], r.get("identity") or 0, r["top"], float(r["scale"]), shared["ff"] if shared else None)
        if not 1 <= c.top <= c.experts + c.identity or c.experts < 1:
            raise ValueError("a router chooses between one and all of its experts")
        return c
    raise ValueError(f"unknown feed-forward kind {m['kind']!r}")


@dataclass(frozen=True)
class LesosunConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerConfig, ...]
    eps: float
    residual_mult: float
    logit_softcap: float

    @staticmethod
    def from_dict(c: dict) -> "LesosunConfig":
        layers = tuple(LayerConfig(_mixer_config(lay["type"], lay["mixer"]), _mlp_config(lay.get("mlp"))) for lay in c["layers"])
        if not c["logit_softcap"] > 0:
            raise ValueError("the cap of the logits must be positive")
        return LesosunConfig(c["vocab"], c["width"], layers, float(c["norm"]["eps"]), float(c["residual_mult"]),
                             float(c["logit_softcap"]))

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def _starts(sizes) -> Tuple[List[int], int]:
    """Where parts of these sizes begin side by side, each at a multiple of eight (16-byte pieces), and the whole."""
    at, out = 0, []
    for n in sizes:
        out.append(at)
        at += _up8(n)
    return out, at


class ParallelMixer(nn.Module):
    def __init__(self, c: ParallelConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps = c, eps
        a, r = c.left, c.right
        self.parts = (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim))
        self.inner = r.heads * r.vdim
        self.n_left = sum(n for _, n in self.parts)              # channels of the convolutions
        self.n_right = self.inner + 2 * r.groups * r.state
        # rows of the projection: q k v | x B C | z | dt; the convolutions' channels are neighbours
        (self.z_at, self.dt_at), rows = _starts((self.inner, r.heads))
        self.z_at, self.dt_at = (n + _up8(self.n_left + self.n_right) for n in (self.z_at, self.dt_at))
        self.proj = mat(rows + _up8(self.n_left + self.n_right), width, dtype=dtype)
        self.bias = nn.Parameter(torch.zeros(self.proj.shape[0], dtype=dtype), requires_grad=False)     # zero behind v
        self.left_taps, self.right_taps = vec((a.conv, self.n_left)), vec((r.conv, self.n_right))
        self.conv_bias = vec(self.n_right)
        self.q_norm, self.k_norm = vec(a.dim, 1.0), vec(a.dim, 1.0)
        self.dt_bias, self.neg_a, self.d_skip = vec(r.heads), vec(r.heads, -1.0), vec(r.heads, 1.0)
        self.norm = vec(self.inner, c.right_scale)               # times the factor of the branch
        self.out_bias = vec(width)                               # times the factor of the branch
        self.out_sizes = (a.heads * a.vdim, self.inner)
        self.tables = None

    def cache_spec(self) -> JointSpec:
        a, r = self.c.left, self.c.right
        return JointSpec((KVSpec(a.kv_heads, a.dim, a.vdim),
                          StateSpec((("S", (r.heads, r.state, r.vdim)), ("conv", (max(a.conv, r.conv), self.n_left + self.n_right))))))

    def prepare(self, max_seq_len: int) -> None:
        """Rotation tables for every position of the longest sequence."""
        a = self.c.left
        if a.rot_dims and (self.tables is None or self.tables[0].shape[0] < max_seq_len):
            rope = RotaryEmbedding({"rope_type": "precise"}, a.rot_dims, max_seq_len, a.rot_base, is_neox_style=False)
            self.tables = rope.device_tables(self.proj.device)

    def load(self, t: CheckpointTensors, pre: str, outs: List[torch.Tensor]) -> None:
        c, a, r, W, off = self.c, self.c.left, self.c.right, self.proj.shape[1], 0
        left, right = pre + "left.", pre + "right."
        self.proj.zero_()
        for name, n in self.parts:
            self.proj[off: off + n].copy_(t.take(left + name, n, W))
            self.bias[off: off + n].copy_(t.take(f"{left}{name}.b", n))
            self.left_taps[:, off: off + n].copy_(t.take(f"{left}{name}.conv", n, a.conv).t())
            off += n
        self.q_norm.copy_(t.take(left + "q.norm", a.dim))
        self.k_norm.copy_(t.take(left + "k.norm", a.dim))
        w = t.take(right + "in", self.inner + self.n_right + r.heads, W)
        self.proj[off: off + self.n_right].copy_(w[self.inner: self.inner + self.n_right])
        self.proj[self.z_at: self.z_at + self.inner].copy_(w[: self.inner])
        self.proj[self.dt_at: self.dt_at + r.heads].copy_(w[self.inner + self.n_right:])
        self.right_taps.copy_(t.take(right + "conv", self.n_right, r.conv).t())
        self.conv_bias.copy_(t.take(right + "conv.b", self.n_right))
        self.dt_bias.copy_(t.take(right + "dt_bias", r.heads))
        self.neg_a.copy_(-torch.exp(t.take(right + "A_log", r.heads).double()))
        self.d_skip.copy_(t.take(right + "D", r.heads))
        self.norm.copy_(t.take(right + "norm", self.inner).double() * c.right_scale)
        self.out_bias.copy_(t.take(left + "o.b", W).double() * c.left_scale)
        outs[0].copy_(t.take(left + "o", W, self.out_sizes[0]))
        outs[1].copy_(t.take(right + "o", W, self.inner))

    def forward(self, h: torch.Tensor, step: Step, cache, outs: List[torch.Tensor]) -> None:
        c, a, r = self.c, self.c.left, self.c.right
        kv, state = cache
        ring, L, C = state["conv"], self.n_left, self.n_left + self.n_right
        p = linear(h, self.proj, self.bias)
        hybrid.conv_attention(step, kv, p, self.left_taps, ring[:, :, :L], self.q_norm, self.k_norm, self.tables, a.heads, a.dim, a.vdim,
                              a.scale, self.eps, a.softcap, c.left_scale, outs[0])
        y = hybrid.ssd(step, p[:, L:C], p[:, self.dt_at: self.dt_at + r.heads], self.right_taps, self.conv_bias, self.dt_bias,
                       self.neg_a, self.d_skip, r.groups, state["S"], ring[:, :, L:])
        hybrid.part_norm_gate(y, self.norm, p[:, self.z_at: self.z_at + self.inner], self.inner // r.norm_groups, self.eps,
                              gate_first=True, out=outs[1])
        if not step.decode_only:
            hybrid.conv_store(step, p, ring)


class DeltaMixer(nn.Module):
    def __init__(self, c: DeltaConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.c, self.eps, self.dtype, self.width = c, eps, dtype, width
        self.parts = (("q", c.kv_heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.heads * c.vdim))
        self.channels = sum(n for _, n in self.parts)
        self.taps = vec((c.conv, self.channels))
        self.dt_bias, self.neg_a, self.norm = vec(c.heads * c.dim), vec(c.heads, -1.0), vec(c.vdim, 1.0)
        self.out_bias = None
        self.out_sizes = (c.heads * c.vdim,)
        self.set_ranks(c.vdim, c.vdim)

    def set_ranks(self, decay: int, gate: int) -> None:
        """The inner sizes of the two low-rank projections, which only a checkpoint's shapes name."""
        c, dev = self.c, self.taps.device
        self.ranks = (decay, gate)
        # rows of the projection: q k v | beta | decay's inner part | gate's inner part
        (_, self.b_at, self.low_at, self.gate_at), rows = _starts((self.channels, c.heads, decay, gate))
        with torch.device(dev):
            self.proj = mat(rows, self.width, dtype=self.dtype)
            # both outer halves as one product: block diagonal
            self.up_at = _up8(c.heads * c.dim)
            self.up = mat(self.up_at + c.heads * c.vdim, rows - self.low_at, dtype=self.dtype)

    def cache_spec(self) -> StateSpec:
        c = self.c
        return StateSpec((("S", (c.heads, c.dim, c.vdim)), ("conv", (c.conv, self.channels))))

    def prepare(self, max_seq_len: int) -> None:
        pass

    def load(self, t: CheckpointTensors, pre: str, outs: List[torch.Tensor]) -> None:
        c, W, off = self.c, self.width, 0
        ra, rg = t.shape(pre + "a1")[0], t.shape(pre + "g1")[0]
        if (ra, rg) != self.ranks:
            self.set_ranks(ra, rg)
        self.proj.zero_()
        self.up.zero_()
        for name, n in self.parts:
            self.proj[off: off + n].copy_(t.take(pre + name, n, W))
            self.taps[:, off: off + n].copy_(t.take(f"{pre}{name}.conv", n, c.conv).t())
            off += n
        self.proj[self.b_at: self.b_at + c.heads].copy_(t.take(pre + "b", c.heads, W))
        self.proj[self.low_at: self.low_at + ra].copy_(t.take(pre + "a1", ra, W))
        self.proj[self.gate_at: self.gate_at + rg].copy_(t.take(pre + "g1", rg, W))
        nk, nv = c.heads * c.dim, c.heads * c.vdim
        self.up[:nk, :ra].copy_(t.take(pre + "a2", nk, ra))
        at = self.gate_at - self.low_at
        self.up[self.up_at:, at: at + rg].copy_(t.take(pre + "g2", nv, rg))
        self.dt_bias.copy_(t.take(pre + "dt_bias", nk))
        self.neg_a.copy_(-torch.exp(t.take(pre + "A_log", c.heads).double()))
        self.norm.copy_(t.take(pre + "norm", c.vdim))
        outs[0].copy_(t.take(pre + "o", W, nv))

    def forward(self, h: torch.Tensor, step: Step, cache, outs: List[torch.Tensor]) -> None:
        c = self.c
        p = linear(h, self.proj)
        up = linear(p[:, self.low_at:], self.up)
        o = hybrid.delta_rule(step, p, up[:, : c.heads * c.dim], p[:, self.b_at: self.b_at + c.heads], self.taps, self.dt_bias,
                              self.neg_a, c.kv_heads, cache["S"], cache["conv"], UNIT_EPS, c.dim ** -0.5)
        hybrid.part_norm_gate(o, self.norm, up[:, self.up_at:], c.vdim, self.eps, out=outs[0])
        if not step.decode_only:
            hybrid.conv_store(step, p, cache["conv"])


class DenseMlp(nn.Module):
    def __init__(self, c: DenseConfig, width: int, dtype: torch.dtype):
        super().__init__()
        self.ff, self.out_sizes = c.ff, (c.ff,)
        self.gate_up = mat(2 * c.ff, width, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str, outs: List[torch.Tensor]) -> None:
        W = self.gate_up.shape[1]
        self.gate_up[: self.ff].copy_(t.take(pre + "gate", self.ff, W))
        self.gate_up[self.ff:].copy_(t.take(pre + "up", self.ff, W))
        outs[0].copy_(t.take(pre + "down", W, self.ff))

    def forward(self, h: torch.Tensor, status, outs: List[torch.Tensor]) -> Optional[hybrid.Routed]:
        hybrid.glu(linear(h, self.gate_up), _C.ACT_SILU, outs[0])
        return None


class MoeMlp(nn.Module):
    def __init__(self, c: MoeConfig, width: int, dtype: torch.dtype):
        super().__init__()
        self.c, self.out_sizes = c, (c.shared_ff,) if c.shared_ff else ()
        self.router, self.correction = mat(c.experts + c.identity, width, dtype=dtype), vec(c.experts + c.identity)
        self.up, self.down = mat(c.experts, c.ff, width, dtype=dtype), mat(c.experts, width, c.ff, dtype=dtype)
        if c.shared_ff:
            self.shared_up = mat(c.shared_ff, width, dtype=dtype)

    def load(self, t: CheckpointTensors, pre: str, outs: List[torch.Tensor]) -> None:
        c, W = self.c, self.router.shape[1]
        self.router.copy_(t.take(pre + "router", c.experts + c.identity, W))
        self.correction.copy_(t.take(pre + "correction", c.experts + c.identity))
        for e in range(c.experts):
            self.up[e].copy_(t.take(f"{pre}e{e}.up", c.ff, W))
            self.down[e].copy_(t.take(f"{pre}e{e}.down", W, c.ff))
        if c.shared_ff:
            self.shared_up.copy_(t.take(pre + "shared.up", c.shared_ff, W))
            outs[0].copy_(t.take(pre + "shared.down", W, c.shared_ff))

    def forward(self, h: torch.Tensor, status, outs: List[torch.Tensor]) -> hybrid.Routed:
        """The shared expert's activations go beside the mixer's; the chosen experts' rows are summed up behind the layer."""
        c = self.c
        if c.shared_ff:
            hybrid.activate(linear(h, self.shared_up), _C.ACT_GELU_ERF, outs[0])
        routed = hybrid.moe_route(h, self.router, self.correction, c.top, softmax=True, weight_scale=c.scale, identity=c.identity)
        return hybrid.moe_experts(h, routed, self.up, self.down, _C.ACT_GELU_ERF, status, gated=False)


_MIXERS = {ParallelConfig: ParallelMixer, DeltaConfig: DeltaMixer}
_MLPS = {DenseConfig: DenseMlp, MoeConfig: MoeMlp}


class LesosunLayer(nn.Module):
    """The weights of a layer; the residual stream and the norms in front are the model's business."""

    def __init__(self, c: LayerConfig, width: int, eps: float, dtype: torch.dtype):
        super().__init__()
        self.mix = _MIXERS[type(c.mixer)](c.mixer, width, eps, dtype)
        self.norm1, self.norm2, self.mlp = vec(width), None, None
        if c.mlp is not None:
            self.mlp, self.norm2 = _MLPS[type(c.mlp)](c.mlp, width, dtype), vec(width)
        # what the output matrices multiply, side by side
        self.sizes = self.mix.out_sizes + (self.mlp.out_sizes if self.mlp is not None else ())
        self.at, total = _starts(self.sizes)
        self.padded = total != sum(self.sizes)
        self.out = mat(width, total, dtype=dtype)

    def _split(self, x: torch.Tensor) -> Tuple[List[torch.Tensor], List[torch.Tensor]]:
        parts = [x[:, a: a + n] for a, n in zip(self.at, self.sizes)]
        k = len(self.mix.out_sizes)
        return parts[:k], parts[k:]

    def load(self, t: CheckpointTensors, pre: str) -> None:
        self.norm1.copy_(t.take(pre + "norm1", self.norm1.shape[0]))
        self.out.zero_()
        mix, mlp = self._split(self.out)
        self.mix.load(t, pre + "mix.", mix)
        if self.mlp is not None:
            self.norm2.copy_(t.take(pre + "norm2", self.norm2.shape[0]))
            self.mlp.load(t, pre + "mlp.", mlp)

    def forward(self, h1: torch.Tensor, h2: Optional[torch.Tensor], step: Step, cache, status):
        """(sum of the sublayers' products, what a mixture's experts add to it)."""
        acts = (torch.zeros if self.padded else torch.empty)(step.n_tokens, self.out.shape[1], dtype=h1.dtype, device=h1.device)
        mix, mlp = self._split(acts)
        self.mix(h1, step, cache, mix)
        routed = self.mlp(h2, status, mlp) if self.mlp is not None else None
        return linear(acts, self.out), routed


class LesosunModel(StepModel):
    def __init__(self, config: LesosunConfig, dtype: torch.dtype):
        super().__init__()
        self.config, self.dtype = config, dtype
        self.embed, self.embed_norm = mat(config.vocab_size, config.hidden_size, dtype=dtype), vec(config.hidden_size)
        self.layers = nn.ModuleList([LesosunLayer(c, config.hidden_size, config.eps, dtype) for c in config.layers])
        self.norm = vec(config.hidden_size)

    def cache_specs(self) -> list:
        return [lay.mix.cache_spec() for lay in self.layers]

    def prepare(self, max_seq_len: int) -> None:
        for lay in self.layers:
            lay.mix.prepare(max_seq_len)

    def forward_step(self, step: Step, cache: HybridCacheManager) -> torch.Tensor:
        cache.begin_step(step)
        c, status = self.config, cache.pool.status_word()
        x = torch.empty(step.n_tokens, c.hidden_size, dtype=torch.float32, device=self.embed.device)

        def norms(i):                         # of the layer behind: one or two of the same stream, or the last one
            lay = self.layers[i] if i < len(self.layers) else None
            return dict(w_next=lay.norm1 if lay is not None else self.norm, w_next2=lay.norm2 if lay is not None else None,
                        eps=c.eps, weight_offset=1.0)

        h = hybrid.residual_norm(step, x, embed=self.embed, embed_norm=self.embed_norm, restart=True, **norms(0))
        for i, lay in enumerate(self.layers):
            h1, h2 = h if isinstance(h, tuple) else (h, None)
            y, routed = lay(h1, h2, step, cache[i], status)
            h = hybrid.residual_norm(step, x, y, bias=lay.mix.out_bias, routed=routed, y_mul=c.residual_mult, **norms(i + 1))
        return h


class LesosunForCausalLM(StepCausalLM):
    def __init__(self, config: LesosunConfig, dtype: torch.dtype = torch.bfloat16):
        super().__init__(config, LesosunModel(config, dtype), dtype)
        self.lm_head.weight = self.model.embed           # one table reads tokens and makes logits

    def load_head(self, t: CheckpointTensors) -> None:
        self.model.embed_norm.copy_(t.take("embed.norm", self.config.hidden_size))

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return hybrid.soft_cap_(super().logits(hidden), self.config.logit_softcap)

    @torch.no_grad()
    def random_init_(self, seed: int, std: float = 0.02) -> "LesosunForCausalLM":
        """Synthetic weights: N(0, std) matrices, unit norms, taps and decays of ordinary size."""
        g = torch.Generator(device=self.lm_head.weight.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if p.dim() >= 2 or name.endswith("correction"):
                p.copy_(torch.randn(p.shape, generator=g, device=p.device) * (0.3 if name.endswith("taps") else std))
            elif name.endswith("neg_a"):
                p.copy_(-torch.exp(torch.rand(p.shape, generator=g, device=p.device) * 2.0 - 1.0))
            elif name.endswith("dt_bias"):
                p.copy_(torch.rand(p.shape, generator=g, device=p.device) * 4.0 - 6.0)
        return self


model_registry.register("Lesosun", lambda config, dtype: LesosunForCausalLM(LesosunConfig.from_dict(config), dtype),
                        dtypes=(torch.bfloat16, torch.float32))
