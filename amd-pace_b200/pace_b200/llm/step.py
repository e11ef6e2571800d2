"""The tokens of one forward pass, packed back to back, as the kernels see them (C struct pace_step_t).

An entry is a sequence that takes part; entries that bring one token come first, so that their attention can
run on the decode kernels and the others' on the prefill kernels.  Everything the kernels need - token ids,
positions, entry boundaries, slots, the rows of the attention staging buffers - is one int32 buffer built on
the host and copied once.
"""
import ctypes as C
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from pace_b200 import _C


@dataclass
class KeyRows:
    """Keys of several entries back to back: entry i owns [cu[i], cu[i + 1]), its first key has position first_pos[i]."""
    total: int
    slot: torch.Tensor
    pos: torch.Tensor
    cu: torch.Tensor
    first_pos: torch.Tensor


class Step:
    """``counts[b]`` new tokens for batch row b (zero: sits out), first position ``starts[b]``, state and cache
    slot ``slots[b]``.  ``tokens`` is a flat integer tensor (host or device) in which row b's tokens begin at
    ``base[b]`` (default: packed back to back in batch order)."""

    def __init__(self, counts: Sequence[int], starts: Sequence[int], slots: Sequence[int], tokens: torch.Tensor,
                 vocab: int, device, base: Optional[Sequence[int]] = None):
        counts = [int(c) for c in counts]
        if base is None:
            base, off = [], 0
            for c in counts:
                base.append(off)
                off += c
        live = [b for b, c in enumerate(counts) if c > 0]
        self.rows = [b for b in live if counts[b] == 1] + [b for b in live if counts[b] > 1]   # batch row of each entry
        self.counts = [counts[b] for b in self.rows]
        self.starts = [int(starts[b]) for b in self.rows]
        self.n_decode = sum(1 for c in self.counts if c == 1)
        self.n_tokens, self.n_entries = sum(self.counts), len(self.rows)
        if self.n_entries == 0:
            raise ValueError("a step needs at least one token")
        self.max_count = max(self.counts)
        # last position of any entry + 1, as far as the host knows (``set_decode``: whoever supplies positions raises it)
        self.max_keys = max(s + c for s, c in zip(self.starts, self.counts))
        self._key_rows: Dict[tuple, "KeyRows"] = {}
        T, E, Ed = self.n_tokens, self.n_entries, self.n_decode
        n = np.asarray(self.counts, dtype=np.int64)
        cu = np.concatenate([[0], np.cumsum(n)])
        entry = np.repeat(np.arange(E), n)
        local = np.arange(T) - cu[entry]
        pos = local + np.asarray(self.starts, dtype=np.int64)[entry]
        # staging rows: one per decode entry, then max_count per entry of the others
        q_row = np.where(entry < Ed, entry, Ed + (entry - Ed) * self.max_count + local)
        self.staging_rows = Ed + (E - Ed) * self.max_count
        src = np.asarray([base[b] for b in self.rows], dtype=np.int64)[entry] + local
        tok = np.zeros(T, dtype=np.int64)
        if not tokens.is_cuda:
            tok = tokens.reshape(-1).numpy().astype(np.int64)[src]
            if tok.min() < 0 or tok.max() >= vocab:
                raise ValueError(f"token ids must lie in [0, {vocab})")
        # (batch row, local token) of a packed row, for callers that ask for logits by place
        self.first_row: Dict[int, int] = {b: int(cu[i]) for i, b in enumerate(self.rows)}
        self.last_rows: List[int] = [int(x) - 1 for x in cu[1:]]
        self._slots = [int(slots[b]) for b in self.rows]
        parts = [tok, entry, pos, q_row, cu, np.asarray(self.starts), np.asarray([slots[b] for b in self.rows]), n]
        if tokens.is_cuda:
            parts.append(src)
        host = torch.from_numpy(np.concatenate(parts).astype(np.int32))
        device = torch.device(device)
        self.device = device
        # the pageable copy is complete on the host side when the call returns, so `host` may go
        self._buf = host.to(device) if device.type != "cuda" else host.pin_memory().to(device, non_blocking=True)
        views, off = [], 0
        for p in parts:
            views.append(self._buf[off: off + len(p)])
            off += len(p)
        (self.token, self.tok_entry, self.tok_pos, self.q_row, self.cu, self.start, self.slot, self.count) = views[:8]
        if tokens.is_cuda:
            self.token.copy_(tokens.reshape(-1).index_select(0, views[8]))
        self.struct = _C.StepStruct(n_tokens=T, n_entries=E, max_count=self.max_count, reserved=0)
        for name in ("token", "tok_entry", "tok_pos", "q_row", "cu", "start", "slot"):
            setattr(self.struct, name, getattr(self, name).data_ptr())

    @property
    def handle(self) -> int:
        """The step as the ``torch.ops.pace_b200`` ops name it: the address of its descriptor."""
        return C.addressof(self.struct)

    @property
    def decode_only(self) -> bool:
        return self.max_count == 1

    def key_rows(self, window: Optional[int], first_entry: int) -> "KeyRows":
        """The keys that entries ``first_entry`` .. see through a sliding window (None: all), listed for gathering."""
        key = (window, first_entry)
        if key not in self._key_rows:
            lo = [max(0, s - window + 1) if window else 0 for s in self.starts[first_entry:]]
            hi = [s + c for s, c in zip(self.starts[first_entry:], self.counts[first_entry:])]
            n = np.asarray(hi) - np.asarray(lo)
            cu = np.concatenate([[0], np.cumsum(n)])
            pos = np.arange(cu[-1]) - np.repeat(cu[:-1], n) + np.repeat(lo, n)
            slot = np.repeat(self._slots[first_entry:], n)
            host = torch.from_numpy(np.concatenate([slot, pos, cu, lo]).astype(np.int32))
            dev = host if self.device.type != "cuda" else host.pin_memory().to(self.device, non_blocking=True)
            T, E = int(cu[-1]), len(lo)
            self._key_rows[key] = KeyRows(T, dev[:T], dev[T: 2 * T], dev[2 * T: 2 * T + E + 1], dev[2 * T + E + 1:])
        return self._key_rows[key]

    def set_decode(self, next_token: torch.Tensor, position: torch.Tensor) -> None:
        """Token ids and positions (int64 ``[n_entries]``, on the device) of a one-token-per-entry step; stream
        ordered, so a recorded step can be replayed with what the previous one produced."""
        if not self.decode_only:
            raise ValueError("set_decode needs a step of one token per entry")
        torch.ops.pace_b200.step_decode(self.token, self.tok_pos, self.start, next_token, position)
