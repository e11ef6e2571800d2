"""What decoders that run on a packed ``Step`` have in common: parameters, checkpoint reading, and the forward forms
that the schedulers and generation loops call.  A model brings ``forward_step`` and what its layers remember."""
from typing import Dict, List, Optional, Sequence, Tuple

import torch
from torch import nn

from pace_b200.llm.cache import KVCacheType
from pace_b200.llm.hybrid_cache import HybridCacheManager
from pace_b200.llm.outputs import ModelOutput
from pace_b200.llm.step import Step
from pace_b200.ops import hybrid


def vec(n, value: float = 0.0) -> nn.Parameter:
    """A small constant of a layer (norm weight, bias, taps): fp32 whatever the activations are."""
    return nn.Parameter(torch.full((n,) if isinstance(n, int) else n, value, dtype=torch.float32), requires_grad=False)


def mat(*shape: int, dtype: torch.dtype) -> nn.Parameter:
    return nn.Parameter(torch.empty(*shape, dtype=dtype), requires_grad=False)


class CheckpointTensors:
    """A checkpoint's tensors, handed out by name with their shapes checked; knows which were never asked for."""

    def __init__(self, tensors: Dict[str, torch.Tensor]):
        self.tensors, self.used = tensors, set()

    def shape(self, name: str) -> Tuple[int, ...]:
        """For sizes that only the checkpoint names."""
        if name not in self.tensors:
            raise KeyError(f"checkpoint has no tensor {name}")
        return tuple(self.tensors[name].shape)

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


class StepModel(nn.Module):
    """Embedding, layers and last norm.  Subclasses define ``config.vocab_size``, ``forward_step`` and
    ``cache_specs``."""

    def forward_step(self, step: Step, cache: HybridCacheManager) -> torch.Tensor:
        """Hidden rows behind the last norm, ``[n_tokens, width]`` in the step's token order."""
        raise NotImplementedError

    def cache_specs(self) -> list:
        """What every layer run remembers (``KVSpec``, ``LatentSpec``, ``StateSpec`` or ``JointSpec``), in execution order."""
        raise NotImplementedError

    def prepare(self, max_seq_len: int) -> None:
        """Called when a cache for sequences of up to ``max_seq_len`` tokens is made."""

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
        self.weight = mat(vocab, width, dtype=dtype)


class StepCausalLM(nn.Module):
    """A ``StepModel`` with its head."""

    def __init__(self, config, model: StepModel, dtype: torch.dtype):
        super().__init__()
        # bf16 products accumulate in fp32 to the end; fp32 products stay out of the reduced-precision modes
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.config, self.dtype, self.vocab_size = config, dtype, config.vocab_size
        self.model = model
        self.lm_head = _Head(config.vocab_size, config.hidden_size, dtype)

    # -- weights and caches --------------------------------------------------------------------------
    def load_head(self, t: CheckpointTensors) -> None:
        self.lm_head.weight.copy_(t.take("head", *self.lm_head.weight.shape))

    @torch.no_grad()
    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        """``embed``, ``l<i>.*`` (layers with a ``load`` method), ``final.norm``, what ``load_head`` takes; nothing may be left
        over."""
        t, V, W = CheckpointTensors(tensors), self.config.vocab_size, self.config.hidden_size
        self.model.embed.copy_(t.take("embed", V, W))
        done = set()
        for i, lay in enumerate(self.model.layers):
            if id(lay) not in done:               # a layer that shares another one's weights is the same module
                lay.load(t, f"l{i}.")
                done.add(id(lay))
        self.model.norm.copy_(t.take("final.norm", W))
        self.load_head(t)
        if t.unused():
            raise ValueError(f"checkpoint tensors without a place in the model: {t.unused()[:8]}")

    def new_cache(self, batch: int, pool_tokens: int, max_seq_len: int,
                  cache_type: KVCacheType = KVCacheType.DYNAMIC) -> HybridCacheManager:
        """Pools and states for ``batch`` rows; called by the schedulers and generation loops."""
        self.model.prepare(max_seq_len)
        return HybridCacheManager(self.model.cache_specs(), batch, pool_tokens, max_seq_len, self.dtype,
                                  self.lm_head.weight.device, cache_type)

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
