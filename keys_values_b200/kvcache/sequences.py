"""State of the sequences a model is working on, one slot per sequence.

A model whose rows may have different lengths keeps, per slot: the position of the next token, the previous
token, and state of the edges between sublayers where there is one (fp32: the token shift's last normed input per layer; the last inputs
of every sublayer, if these pass a convolution, in rings: position p in row p mod taps). Slots are handed
out and taken back like cache blocks; a slot that starts at position 0 never reads what an earlier owner left.

A pass (:class:`SequencePass`) names the slots of its rows, the position each row starts at and how many of its
tokens are real. Everything a kernel needs is in device tensors, so a single-token pass can be captured in a CUDA graph;
host mirrors of the positions serve argument checks and launch shapes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch


@dataclass
class SequencePass:
    slots: torch.Tensor  # (B,) int32
    start: torch.Tensor  # (B,) int32: position of the row's first token
    count: torch.Tensor  # (B,) int32: real tokens of the row
    slots_host: Tuple[int, ...]
    start_host: Tuple[int, ...]
    count_host: Tuple[int, ...]
    length: int  # tokens per row, padding included

    @property
    def max_start(self) -> int:
        return max(self.start_host)

    @property
    def max_end(self) -> int:
        return max(s + n for s, n in zip(self.start_host, self.count_host))


class SequenceTable:
    def __init__(self, n_slots: int, device, shift_layers: int = 0, width: int = 0, conv_edges: int = 0, taps: int = 0,
                 dtype: torch.dtype = torch.float32):
        """``conv_edges``: sublayers whose input passes a convolution of ``taps``; these inputs are kept as ``dtype``."""
        if n_slots <= 0:
            raise ValueError("n_slots must be positive")
        self.n_slots = n_slots
        self.device = torch.device(device)
        with torch.inference_mode(False):
            self.pos = torch.zeros(n_slots, dtype=torch.int32, device=self.device)
            self.prev_token = torch.zeros(n_slots, dtype=torch.int32, device=self.device)
            self.shift = torch.zeros((shift_layers, n_slots, width), dtype=torch.float32, device=self.device) if shift_layers else None
            self.conv = torch.zeros((conv_edges, n_slots, taps, width), dtype=dtype, device=self.device) if conv_edges else None
        self._consts: Dict[Tuple[int, ...], torch.Tensor] = {}
        self.reset()

    # ------------------------------------------------------------------ slots
    def reset(self) -> None:
        """Every slot is free and at position 0; the next pass takes the first slots for its rows."""
        self.pos.zero_()
        self.pos_host: List[int] = [0] * self.n_slots
        self._free = list(range(self.n_slots))
        self.batch: Optional[Tuple[int, ...]] = None

    def acquire(self) -> int:
        """A free slot, at position 0."""
        if not self._free:
            raise RuntimeError(f"all {self.n_slots} sequence slots are in use")
        return self._free.pop(0)

    def release(self, slot: int) -> None:
        if slot in self._free or not 0 <= slot < self.n_slots:
            raise ValueError(f"slot {slot} is not in use")
        self.pos[slot] = 0
        self.pos_host[slot] = 0
        self._free.append(slot)
        self._free.sort()
        if self.batch is not None and slot in self.batch:
            self.batch = tuple(s for s in self.batch if s != slot)

    def live(self) -> int:
        return self.n_slots - len(self._free)

    def set_batch(self, slots: Sequence[int]) -> None:
        """Slots of the rows of the following passes."""
        slots = tuple(int(s) for s in slots)
        if len(set(slots)) != len(slots) or any(s in self._free or not 0 <= s < self.n_slots for s in slots):
            raise ValueError(f"slots {slots} must be distinct and acquired")
        self.batch = slots

    # ----------------------------------------------------------------- passes
    def _const(self, values: Tuple[int, ...]) -> torch.Tensor:
        """Small int32 tensor that stays: single-token passes find theirs here, so a captured step copies nothing and its
        graph can keep reading it."""
        t = self._consts.get(values)
        if t is None:
            with torch.inference_mode(False):
                t = self._consts[values] = torch.tensor(values, dtype=torch.int32, device=self.device)
        return t

    def begin(self, batch_size: int, length: int, counts: Optional[Sequence[int]] = None) -> SequencePass:
        if not self.batch:
            if batch_size > self.n_slots:
                raise ValueError(f"batch size {batch_size} exceeds the {self.n_slots} sequence slots")
            self.set_batch([self.acquire() for _ in range(batch_size)])
        if len(self.batch) != batch_size:
            raise ValueError(f"batch size {batch_size} differs from the {len(self.batch)} sequences of the batch")
        counts = (length,) * batch_size if counts is None else tuple(int(n) for n in counts)
        if len(counts) != batch_size or any(not 0 <= n <= length for n in counts):
            raise ValueError(f"counts {counts} must give 0 .. {length} tokens for each of {batch_size} rows")
        slots = self.batch
        start = self.pos[:batch_size] if slots == tuple(range(batch_size)) else self.pos.index_select(0, self._const(slots))
        count = self._const(counts) if length == 1 else torch.tensor(counts, dtype=torch.int32, device=self.device)
        return SequencePass(self._const(slots), start, count, slots, tuple(self.pos_host[s] for s in slots), counts, length)

    def finish(self, seq: SequencePass, idx: torch.Tensor) -> None:
        from keys_values_b200.ops import layers as L

        L.sequence_advance(idx, self.pos, self.prev_token, seq)
        for s, n in zip(seq.slots_host, seq.count_host):
            self.pos_host[s] += n

    def advance_host(self) -> None:
        """One token of every row of the batch has been processed by a replayed graph."""
        for s in self.batch:
            self.pos_host[s] += 1

    def size_estimate(self) -> int:
        """Bits held on the device."""
        return 64 * self.n_slots + sum(8 * t.numel() * t.element_size() for t in (self.shift, self.conv) if t is not None)
