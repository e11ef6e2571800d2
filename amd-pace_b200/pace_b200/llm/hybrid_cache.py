"""Caches of hybrid decoders: paged K/V for attention layers, fixed-size recurrent states for the others.

A model describes what each of its layer runs remembers (``KVSpec``, ``BlockSpec``, ``LatentSpec``, ``StateSpec``, or a ``JointSpec`` of
them; a layer that runs several times has one entry per run; what the model itself remembers is one more entry).  ``HybridCacheManager`` keeps one paged pool (``KVPool`` under a
``KVCacheManager``) per distinct K/V geometry and one state array per recurrent run, all indexed by the same
batch rows, and presents what the generation loops use of ``KVCacheManager``: lengths per row, recycling of
finished rows, beam gather, the switches of graph capture, status checks.

K and V rows: bf16 with head sizes up to 128 are stored as 64- or 128-element rows (zero-filled), which the
tensor-core attention kernels read; anything else (fp32, larger heads) as opaque rows for the general kernel.
Latent rows are opaque rows of one plane, padded to a multiple of eight elements.  The rows of pooled blocks live in a pool of their
own whose pages cover as many blocks as the token pages cover tokens; it counts in tokens and is large enough for whatever fits the
token pool.  States are fp32 (unless their spec says otherwise).  A state is never cleared: a sequence whose first position is 0 starts from zeros, so a row
that is used again needs nothing but its length set back.
"""
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple, Union

import torch

from pace_b200 import _C
from pace_b200.llm.cache import KVCacheManager, KVCacheType, KVPool, PagedKV, physical_page_tokens
from pace_b200.llm.step import Step


@dataclass(frozen=True)
class KVSpec:
    kv_heads: int
    dim: int          # per-head key size
    vdim: int         # per-head value size


@dataclass(frozen=True)
class BlockSpec:
    """Beside a ``KVSpec`` of the same sizes: a key and a value row for every whole block of ``block`` tokens."""
    kv_heads: int
    dim: int
    vdim: int
    block: int


@dataclass(frozen=True)
class LatentSpec:
    """One row per token for all heads: a latent (keys and values are made from it) and a rotated key part."""
    rank: int
    rot_dim: int


@dataclass(frozen=True)
class StateSpec:
    """Shapes per sequence of a recurrent run's arrays."""
    shapes: Tuple[Tuple[str, Tuple[int, ...]], ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class JointSpec:
    """A layer run that remembers several things (mixers side by side): its cache is the ``JointCache`` of theirs."""
    parts: Tuple[Union[KVSpec, BlockSpec, LatentSpec, StateSpec], ...]


def kv_row(spec: Union[KVSpec, BlockSpec, LatentSpec], dtype: torch.dtype) -> Tuple[int, int]:
    """(pool head_dim in 16-bit units, row format) that holds the keys and values of a layer."""
    if isinstance(spec, LatentSpec):
        n = (spec.rank + spec.rot_dim + 7) // 8 * 8
        return (n if dtype == torch.bfloat16 else 2 * n), _C.ROWS_SHARED
    widest = max(spec.dim, spec.vdim)
    if dtype == torch.bfloat16:
        if widest <= 128:
            return (64 if widest <= 64 else 128), _C.ROWS_BF16
        return (widest + 7) // 8 * 8, _C.ROWS_OPAQUE
    if dtype == torch.float32:
        return (widest + 3) // 4 * 4 * 2, _C.ROWS_OPAQUE
    raise TypeError(f"caches hold bfloat16 or float32 rows, got {dtype}")


class StateCache:
    """A recurrent run's arrays, ``[slots, ...]`` each."""

    def __init__(self, manager: "HybridCacheManager", spec: StateSpec, slots: int, device):
        self.manager = manager
        self.arrays: Dict[str, torch.Tensor] = {
            name: torch.zeros((slots,) + tuple(shape), dtype=spec.dtype, device=device) for name, shape in spec.shapes}

    def __getitem__(self, name: str) -> torch.Tensor:
        return self.arrays[name]

    @property
    def seq_lens(self) -> List[int]:
        return self.manager.seq_lens

    @property
    def seq_len(self) -> int:
        return max(self.manager.seq_lens, default=0)


class JointCache(tuple):
    """The caches of a ``JointSpec``; its parts have the same lengths."""

    @property
    def seq_lens(self) -> List[int]:
        return self[0].seq_lens

    @property
    def seq_len(self) -> int:
        return self[0].seq_len


class PoolSet:
    """What callers ask of "the pool" when there are several (or none).  Pools of blocks follow the token pools and never run out
    before them: free pages are those of the token pools."""

    def __init__(self, pools: List[KVPool], n_pages: int, block_pools: Sequence[KVPool] = ()):
        self.pools, self.n_pages = pools, n_pages
        self.token_pools = [p for p in pools if p not in block_pools]

    @property
    def host_free_pages(self) -> int:
        return min((p.host_free_pages for p in self.token_pools), default=self.n_pages)

    @property
    def shared_pages(self) -> bool:
        return any(p.shared_pages for p in self.pools)

    def query(self) -> Tuple[int, int]:
        bits, free = 0, self.n_pages
        for p in self.pools:
            b, f = p.query()
            bits, free = bits | b, min(free, f) if p in self.token_pools else free
        return bits, free

    def status_word(self) -> Optional[torch.Tensor]:
        """Where kernels that belong to no pool report (None: there is no pool)."""
        return self.pools[0].status_word() if self.pools else None

    def check_status(self) -> None:
        for p in self.pools:
            p.check_status()

    def clear_status(self) -> None:
        for p in self.pools:
            p.clear_status()


class _GroupConfig:
    def __init__(self, n: int):
        self.num_hidden_layers = n


class HybridCacheManager:
    """``specs``: one (``KVSpec``, ``BlockSpec``, ``LatentSpec``, ``StateSpec`` or ``JointSpec``) per layer run.  ``pool_tokens``: tokens the K/V pools hold for all rows together (rounded
    down to pages); ``batch``: rows, each with a slot in every pool and state array."""

    def __init__(self, specs: Sequence[Union[KVSpec, LatentSpec, StateSpec, JointSpec]], batch: int, pool_tokens: int, max_seq_len: int,
                 dtype: torch.dtype, device, cache_type: KVCacheType = KVCacheType.DYNAMIC):
        self.batch, self.max_seq_len, self.dtype = batch, max_seq_len, dtype
        self.device = torch.device(device)
        self.num_layers = len(specs)
        joint = [len(s.parts) if isinstance(s, JointSpec) else 0 for s in specs]
        specs = [p for s in specs for p in (s.parts if isinstance(s, JointSpec) else (s,))]
        self._lens = [0] * batch
        self.page_tokens = physical_page_tokens(None)
        n_pages = max(1, pool_tokens // self.page_tokens)
        max_pages = min(n_pages, (max_seq_len + self.page_tokens - 1) // self.page_tokens)
        by_geometry: Dict[Tuple[int, int, int, int], List[int]] = {}
        for i, s in enumerate(specs):
            if not isinstance(s, StateSpec):
                key = (getattr(s, "kv_heads", 1),) + kv_row(s, dtype) + (s.block if isinstance(s, BlockSpec) else 0,)
                by_geometry.setdefault(key, []).append(i)
        self.groups: List[KVCacheManager] = []
        block_pools: List[KVPool] = []
        self.caches: List[object] = [None] * len(specs)
        for (heads, units, fmt, block), runs in by_geometry.items():
            if block == 0:
                pool = KVPool(len(runs), heads, units, self.page_tokens, n_pages, max_seqs=batch, max_pages_per_seq=max_pages,
                              device=self.device, row_format=fmt)
            else:          # every row of the batch may leave the rest of a page empty
                per = self.page_tokens * block
                most = (max_pages * self.page_tokens + per - 1) // per
                pool = KVPool(len(runs), heads, units, per, min(n_pages * self.page_tokens // per + batch, most * batch), max_seqs=batch,
                              max_pages_per_seq=most, device=self.device, row_format=fmt, row_tokens=block)
                block_pools.append(pool)
            mgr = KVCacheManager(_GroupConfig(len(runs)), max_seq_len, cache_type, pool=pool)
            mgr.open_batch(batch)
            for j, run in enumerate(runs):
                self.caches[run] = mgr[j]
            self.groups.append(mgr)
        self.states: List[StateCache] = []
        for i, s in enumerate(specs):
            if isinstance(s, StateSpec):
                self.caches[i] = StateCache(self, s, batch, self.device)
                self.states.append(self.caches[i])
        parts = iter(self.caches)
        self.caches = [JointCache(next(parts) for _ in range(n)) if n else next(parts) for n in joint]
        self.pool = PoolSet([g.pool for g in self.groups], n_pages, block_pools)
        # rows map to slots 1:1: every pool is this manager's own
        self.slots = list(range(batch))
        self._decode_step: Optional[Step] = None
        self._static = self._capturing = self._skip_reserve = False
        self.defer_appends = False          # (accepted for the generation loops; rows are stored by the layers themselves)

    # -- what the generation loops use ---------------------------------------------------------
    def __getitem__(self, run: int):
        return self.caches[run]

    def __len__(self) -> int:
        return max(self._lens, default=0)

    @property
    def seq_lens(self) -> List[int]:
        return list(self._lens)

    def _switch(name):
        def get(self):
            return getattr(self, "_" + name)

        def put(self, value):
            setattr(self, "_" + name, value)
            for g in self.groups:
                setattr(g, {"static": "static_launch"}.get(name, name), value)
        return property(get, put)

    static_launch = _switch("static")
    capturing = _switch("capturing")
    skip_reserve = _switch("skip_reserve")
    del _switch

    def commit(self) -> None:
        pass

    def advance_host_mirror(self, n: int) -> bool:
        """Every row took ``n`` tokens in a replayed step; True when a row needs a new page."""
        grow = False
        for g in self.groups:
            grow |= g.advance_host_mirror(n)
        self._lens = [x + n for x in self._lens]
        return grow

    def begin_step(self, step: Step) -> None:
        """Pages for the step's tokens and the new lengths, on the host and on the device, before any layer runs
        (the layers store their rows at the positions the step names)."""
        counts = [0] * self.batch
        for b, c in zip(step.rows, step.counts):
            if self._lens[b] + c > self.max_seq_len:
                raise RuntimeError(f"sequence of {self._lens[b] + c} tokens exceeds max_seq_len {self.max_seq_len}")
            counts[b] = c
        for g in self.groups:
            g.advance_step(counts, step.slot, step.count, step.max_count)
        if not self._capturing:
            self._lens = [x + c for x, c in zip(self._lens, counts)]

    def step(self, counts: Sequence[int], tokens: torch.Tensor, vocab: int, base: Optional[Sequence[int]] = None) -> Step:
        return Step(counts, self._lens, self.slots, tokens, vocab, self.device, base)

    def decode_step(self) -> Step:
        """The fixed step of one token per row whose ids and positions the device supplies (``set_decode``)."""
        if self._decode_step is None:
            self._decode_step = Step([1] * self.batch, [0] * self.batch, self.slots,
                                     torch.zeros(self.batch, dtype=torch.long), 1, self.device)
            self._decode_step.max_keys = self.max_seq_len     # positions come from the device
        return self._decode_step

    def recycle(self, batch_indices: Sequence[int]) -> None:
        """Ends the sequences of these rows: pages go back, lengths to zero; the states are stale from here on and
        the next sequence of a row starts from zeros by its position."""
        for g in self.groups:
            g.recycle(batch_indices)
        for b in batch_indices:
            self._lens[int(b)] = 0

    def update_cache_with_beam_indices(self, beam_idx: torch.Tensor) -> None:
        """Row i continues old row ``beam_idx[i]``: index-only on the pools, a copy of the (small) states."""
        for g in self.groups:
            g.update_cache_with_beam_indices(beam_idx)
        idx = beam_idx.to(self.device).long()
        for s in self.states:
            for name, x in s.arrays.items():
                s.arrays[name].copy_(x.index_select(0, idx))
        self._lens = [self._lens[j] for j in beam_idx.tolist()]

    def remove_cache(self, remove_len) -> None:
        """Attention-only stacks roll back like ``KVCacheManager``; a recurrent state holds no past to go back to."""
        n = remove_len.tolist() if isinstance(remove_len, torch.Tensor) else remove_len
        n = [int(x) for x in n] if isinstance(n, (list, tuple)) else [int(n)] * self.batch
        if not any(n):
            return
        if self.states:
            raise NotImplementedError("recurrent states cannot be rolled back (speculative decoding needs attention-only models)")
        for g in self.groups:
            g.remove_cache(n)
        self._lens = [have - r for have, r in zip(self._lens, n)]

    def release(self) -> None:
        for g in self.groups:
            g.release()

    def bytes_per_token(self) -> int:
        """K/V bytes one cached token takes over all layer runs (blocks: its share of a row)."""
        return sum(g.num_layers * (1 if g.pool.desc.row_format == _C.ROWS_SHARED else 2) * g.pool.n_kv_heads *
                   g.pool.head_dim * 2 // max(1, g.pool.desc.row_tokens) for g in self.groups)
