"""Recurrent state of sequences, beside the paged cache.

A sequence of a model with recurrent layers owns one slot, and a slot has two rows.  A pass reads the row that holds the
state after the tokens before its first one and writes the other row, so the state before a pass survives it: a pass can run
again from the same position (a graph's warm-up run, a decode step that was launched ahead and dropped, a verification of
drafts of which some are rejected) and finds what it found the first time.  A pass from position 0 reads nothing: a slot that
is used again needs no clearing.

A row holds ``state_floats`` 32-bit numbers (every recurrent layer's part at its offset) and the sequence's last token.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass
from typing import Deque, Dict, Optional, Tuple

import torch


@dataclass
class _Entry:
    slot: int
    pos: int = 0                 # tokens that row 2 * slot + bank has seen
    bank: int = 0
    before: int = -1             # tokens that the other row has seen; -1: none that can be used


class StateSlots:
    def __init__(self, slots: int, floats: int, device=None):
        if slots <= 0:
            raise ValueError("a model with recurrent state needs at least one state slot")
        self.slots, self.floats = slots, floats
        self._free: Deque[int] = deque(range(slots))
        self._seqs: Dict[int, _Entry] = {}
        self.rows: Optional[torch.Tensor] = None
        self.last_token: Optional[torch.Tensor] = None
        if device is not None:
            self.rows = torch.zeros(2 * slots, max(4, floats), dtype=torch.float32, device=device)
            self.last_token = torch.zeros(2 * slots, dtype=torch.int32, device=device)

    @staticmethod
    def bytes_per_slot(floats: int) -> int:
        return 2 * (max(4, floats) + 1) * 4

    @property
    def num_free(self) -> int:
        return len(self._free)

    @property
    def total_bytes(self) -> int:
        return self.slots * self.bytes_per_slot(self.floats)

    def allocate(self, seq_id: int) -> None:
        if seq_id in self._seqs:
            raise ValueError(f"sequence {seq_id} already has a state slot")
        if not self._free:
            raise RuntimeError(f"no state slot left for sequence {seq_id} ({self.slots} in use)")
        self._seqs[seq_id] = _Entry(self._free.popleft())

    def free(self, seq_id: int) -> None:
        e = self._seqs.pop(seq_id, None)
        if e is not None:
            self._free.append(e.slot)

    def fork(self, src_id: int, dst_id: int) -> None:
        self.allocate(dst_id)
        s, d = self._seqs[src_id], self._seqs[dst_id]
        d.pos, d.bank, d.before = s.pos, s.bank, s.before
        if self.rows is not None:
            for t in (self.rows, self.last_token):
                t[2 * d.slot: 2 * d.slot + 2].copy_(t[2 * s.slot: 2 * s.slot + 2])

    def advance(self, seq_id: int, start: int, tokens: int) -> Tuple[int, int]:
        """(row to read or -1, row to write) of a pass over ``tokens`` tokens from position ``start``."""
        e = self._seqs[seq_id]
        if start == 0:
            read, bank = -1, 1 - e.bank
        elif start == e.pos:
            read, bank = 2 * e.slot + e.bank, 1 - e.bank
        elif start == e.before:
            read, bank = 2 * e.slot + 1 - e.bank, e.bank
        else:
            raise RuntimeError(f"sequence {seq_id}: the state at position {start} is not held (positions {e.pos} and "
                               f"{e.before} are)")
        e.before, e.pos, e.bank = (start if read >= 0 else -1), start + tokens, bank
        return read, 2 * e.slot + bank

    def position(self, seq_id: int) -> int:
        return self._seqs[seq_id].pos

    def destroy(self) -> None:
        self.rows = self.last_token = None
        self._seqs.clear()
        self._free.clear()
