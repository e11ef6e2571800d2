"""RotaryEmbedding operator: the reference's front end (pace/ops/rotary_embedding.py:202-485) with
the same constructor arguments, buffers and ``forward`` contract, plus what the fused CUDA path
needs: the table row of every position as an int32 tensor and the fp32 tables on the device.

On the hot path the rotation is not done here: ``KVCacheBase.update_cache_rope`` hands the tables to
``pace_kv_append_rope``, which rotates q and k while it appends k and v (one kernel instead of the
reference's index_select + eight elementwise ops + the append).  ``forward`` keeps the reference's
two return forms for callers that rotate outside the cache.
"""
import math
from functools import partial
from typing import Any, Callable, Dict, Optional, Tuple, Union

import torch
from torch import nn


def _yarn_tables(theta: float, rotary_dim: int, n_rows: int, scaling: Optional[Dict[str, Any]]):
    """fp32 tables from double-precision frequencies and angles.  ``scaling`` (``factor``,
    ``original_max_position_embeddings``, ``beta_fast``, ``beta_slow``): pairs that turn at least ``beta_fast`` times
    within the original length keep their frequency, those that turn at most ``beta_slow`` times have it divided by the
    factor, a linear ramp over the pairs lies in between; cos and sin are multiplied by 0.1 ln(factor) + 1."""
    i = torch.arange(rotary_dim // 2, dtype=torch.float64)
    freq, gain = theta ** (-2.0 * i / rotary_dim), 1.0
    if scaling is not None:
        factor, window = float(scaling["factor"]), float(scaling["original_max_position_embeddings"])
        pair = lambda turns: rotary_dim * math.log(window / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))   # noqa: E731
        lo = max(math.floor(pair(scaling["beta_fast"])), 0)
        hi = min(math.ceil(pair(scaling["beta_slow"])), rotary_dim - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        freq = freq / factor * ramp + freq * (1.0 - ramp)
        gain = 0.1 * math.log(factor) + 1.0
    return _precise_tables(freq, n_rows, gain)


def _precise_tables(freq: torch.Tensor, n_rows: int, gain: float = 1.0):
    angle = torch.arange(n_rows, dtype=torch.float64)[:, None] * freq[None, :]
    return (angle.cos() * gain).float(), (angle.sin() * gain).float()


def _llama3_frequencies(freq: torch.Tensor, scaling: Dict[str, Any]) -> torch.Tensor:
    """Wavelengths shorter than the original length / ``high_freq_factor`` keep their frequency, those longer than length /
    ``low_freq_factor`` have it divided by the factor, in between lies a blend."""
    f, lo, hi = scaling["factor"], scaling["low_freq_factor"], scaling["high_freq_factor"]
    window = scaling["original_max_position_embeddings"]
    wavelength = 2 * math.pi / freq
    blend = (window / wavelength - lo) / (hi - lo) if lo != hi else 0
    mixed = (1 - blend) * freq / f + blend * freq
    return torch.where(wavelength < window / hi, freq, torch.where(wavelength > window / lo, freq / f, mixed))


def _frequencies(theta: float, rotary_dim: int, divide_by=None) -> torch.Tensor:
    exponents = torch.arange(0, rotary_dim, 2, dtype=torch.float) / rotary_dim
    freq = theta ** exponents
    if divide_by:
        freq = torch.tensor(divide_by, dtype=torch.float32) * freq
    return 1.0 / freq


def _tables(freq: torch.Tensor, n_rows, gain: float = 1.0) -> Tuple[torch.Tensor, torch.Tensor]:
    angle = torch.einsum("i,j -> ij", torch.arange(n_rows, dtype=torch.float), freq)
    return angle.cos() * gain, angle.sin() * gain


class RotaryEmbedding(nn.Module):
    """``rope_scaling`` selects the variant through ``rope_type`` (or the older ``type``) key:
    ``default``, ``linear`` (``scaling_factor``), ``dynamic`` (NTK, ``scaling_factor``), ``llama3``
    (``factor``, ``low_freq_factor``, ``high_freq_factor``, ``original_max_position_embeddings``) and
    ``longrope`` (``short_factor``, ``long_factor``, optional ``attention_factor``; keyword
    ``original_max_position_embeddings``), ``yarn`` (``factor``, ``original_max_position_embeddings``, ``beta_fast``,
    ``beta_slow``), ``precise`` (no scaling) and ``llama3_precise`` (as ``llama3``).  Tables are fp32 ``[rows, rotary_dim / 2]``;
    those of the last three come from double-precision angles (an fp32 product of position and frequency is off by up to half an ulp of the angle)."""

    def __init__(self, rope_scaling: Optional[Dict[str, Any]], rotary_dim: int, max_position_embeddings: int,
                 rope_theta: float, partial_rotary_factor: float = 1.0, dtype: Optional[torch.dtype] = None,
                 backend_impl=None, is_neox_style: bool = True, **rope_kwargs):
        super().__init__()
        if partial_rotary_factor < 1.0:
            rotary_dim = int(rotary_dim * partial_rotary_factor)
        self.rotary_dim = rotary_dim
        self.partial_rotary_factor = partial_rotary_factor
        self.rope_kwargs = rope_kwargs
        self.rope_scaling = rope_scaling
        self.rope_type = "default" if rope_scaling is None else rope_scaling.get("rope_type", rope_scaling.get("type"))
        self.max_position_embeddings = max_position_embeddings
        self.rope_theta = rope_theta
        self.is_neox_style = is_neox_style
        self.original_max_position_embeddings = None
        kind, R, N = self.rope_type, rotary_dim, max_position_embeddings
        if kind == "default":
            cos, sin = _tables(_frequencies(rope_theta, R), N)
        elif kind == "linear":
            # (the reference scales cos and sin themselves by the factor, rotary_embedding.py:124-136)
            cos, sin = _tables(_frequencies(rope_theta, R), N, rope_scaling["scaling_factor"])
        elif kind == "dynamic":
            f = rope_scaling["scaling_factor"]
            rows = N * f
            theta = rope_theta * ((f * rows / N) - (f - 1)) ** (R / (R - 2))
            cos, sin = _tables(_frequencies(theta, R), rows)
        elif kind == "llama3":
            cos, sin = _tables(_llama3_frequencies(_frequencies(rope_theta, R), rope_scaling), N)
        elif kind == "llama3_precise":
            freq = rope_theta ** (-2.0 * torch.arange(R // 2, dtype=torch.float64) / R)
            cos, sin = _precise_tables(_llama3_frequencies(freq, rope_scaling), N)
        elif kind == "longrope":
            window = rope_kwargs.get("original_max_position_embeddings", N)
            self.original_max_position_embeddings = window
            ratio = N / window
            gain = 1.0 if ratio <= 1.0 else math.sqrt(1 + math.log(ratio) / math.log(window))
            if rope_scaling.get("attention_factor") is not None:
                gain = rope_scaling["attention_factor"]
            short = _tables(_frequencies(rope_theta, R, rope_scaling["short_factor"]), window, gain)
            long = _tables(_frequencies(rope_theta, R, rope_scaling["long_factor"]), N, gain)
            cos, sin = torch.cat([short[0], long[0]]), torch.cat([short[1], long[1]])
        elif kind in ("yarn", "precise"):
            cos, sin = _yarn_tables(rope_theta, R, N, rope_scaling if kind == "yarn" else None)
        else:
            raise ValueError(f"Unsupported RoPE type: {kind}")
        self.register_buffer("cos_cache", cos.contiguous(), persistent=False)
        self.register_buffer("sin_cache", sin.contiguous(), persistent=False)
        self._device_tables = {}

    # ---- what the fused kernel takes ----------------------------------------------------------
    def table_rows(self, position_ids: torch.Tensor, offsets: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Row of the tables each position reads, int32 and contiguous (rotary_embedding.py:382-396:
        longrope moves every index to the long table as soon as one position leaves the original window)."""
        idx = position_ids
        if self.rope_type == "longrope":
            k = self.original_max_position_embeddings
            idx = idx + (torch.any(position_ids > k).to(idx.dtype) * k)
            if offsets is not None:
                idx = idx + offsets
        return idx.to(torch.int32).contiguous()

    def device_tables(self, device) -> Tuple[torch.Tensor, torch.Tensor]:
        key = str(torch.device(device))
        if key not in self._device_tables:
            self._device_tables[key] = (self.cos_cache.to(device=device, dtype=torch.float32).contiguous(),
                                        self.sin_cache.to(device=device, dtype=torch.float32).contiguous())
        return self._device_tables[key]

    # ---- the reference's forward contract -------------------------------------------------------
    def forward(self, x: torch.Tensor, position_ids: torch.Tensor, return_cos_sin: bool = False,
                offsets: Optional[torch.Tensor] = None) -> Union[Callable, Tuple[torch.Tensor, torch.Tensor]]:
        rows = self.table_rows(position_ids, offsets).long().flatten()
        cos = self.cos_cache.to(x.device).index_select(0, rows).unflatten(0, position_ids.shape).to(x.dtype)
        sin = self.sin_cache.to(x.device).index_select(0, rows).unflatten(0, position_ids.shape).to(x.dtype)
        if return_cos_sin:
            return cos, sin
        return partial(self.apply_rotary_emb, cos=cos, sin=sin, unsqueeze_dim=1)

    def _rotate(self, x, cos, sin, unsqueeze_dim, is_neox_style):
        cos, sin = cos.unsqueeze(unsqueeze_dim), sin.unsqueeze(unsqueeze_dim)
        R = self.rotary_dim
        turn, keep = x[..., :R], x[..., R:]
        if is_neox_style:
            a, b = turn[..., : R // 2], turn[..., R // 2:]
        else:
            a, b = turn[..., ::2], turn[..., 1::2]
        ra, rb = a * cos - b * sin, b * cos + a * sin
        turned = torch.cat((ra, rb), dim=-1) if is_neox_style else torch.stack((ra, rb), dim=-1).flatten(-2)
        return torch.cat((turned, keep), dim=-1) if keep.shape[-1] else turned

    def apply_rotary_emb(self, query, key, cos, sin, unsqueeze_dim: int = 1, is_neox_style: Optional[bool] = None):
        """query / key ``[B, heads, S, D]``, cos / sin ``[B, S, rotary_dim / 2]`` in their dtype."""
        style = self.is_neox_style if is_neox_style is None else is_neox_style
        return self._rotate(query, cos, sin, unsqueeze_dim, style), self._rotate(key, cos, sin, unsqueeze_dim, style)

    def extra_repr(self):
        return (f"rope_type={self.rope_type}, rotary_dim={self.rotary_dim}, "
                f"max_position_embeddings={self.max_position_embeddings}, rope_theta={self.rope_theta}")
