"""Cache of a grouped-query attention layer: rotated keys and values.

One row per token and key/value head, ``[keys (padded to a multiple of 8, one per map) | value (the same)]``. Prompts and single
tokens attend over the cache as it lies. A layer that sees every earlier position keeps position p of the sequence in slot s in row p
of that slot. A layer that looks back a bounded way (a window or chunks) needs the rows of that span and of the pass at hand: if
the cache is longer, the first positions that stay visible have rows of their own and the others share a ring
(:class:`keys_values_b200.ops.layers.RowPlan`), in tiles of the attention kernels, so that a tile never wraps.
"""
from __future__ import annotations

from typing import Optional

import torch

from keys_values_b200.config import Config
from keys_values_b200.kvcache.layer_cache import MAX_PASS_TOKENS, LayerCache
from keys_values_b200.ops.layers import RowPlan


TILE = 128  # rows of the widest tile of the attention kernels


def tiles(n: int) -> int:
    return (n + TILE - 1) // TILE * TILE


class GroupedKVCache(LayerCache):
    kind = "grouped_attention"
    # tokens of a pass that a ring takes besides the span of its layer
    max_pass = MAX_PASS_TOKENS

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **_ignored):
        from keys_values_b200.models.grouped_attention import grouped_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device)
        s = self.shape = grouped_shape(config.layers[block_idx]["mixer"])
        self.plan = RowPlan()
        if s.span:
            head, ring = tiles(s.keep), tiles(s.span + self.max_pass)
            if head + ring < cache_length:
                self.plan = RowPlan(head, ring)
        self.length = cache_length if not self.plan.ring else sum(self.plan)  # rows of a slot

    @property
    def rows(self) -> Optional[torch.Tensor]:
        """``(turns, max_batch_size, length, kv_heads, shape.row)``."""
        return None if self.buffers_ is None else self.buffers_[0]

    @property
    def current_length(self) -> int:
        return min(self.input_pos, self.length)

    def check_capacity(self, end: int) -> None:
        if end > self.cache_length and not self.plan.ring:
            raise IndexError(f"layer {self.block_idx}: {end} tokens exceed the cache of {self.cache_length}")

    def check_pass(self, seq) -> None:
        super().check_pass(seq)
        if self.plan.ring and seq.length > self.plan.ring - self.shape.span:
            raise IndexError(f"layer {self.block_idx}: a pass of {seq.length} tokens exceeds the ring of {self.plan.ring} (take smaller portions)")

    def _shapes(self, dtype):
        s = self.shape
        return {"keys_values": ((self.max_batch_size, self.length, s.kv_heads, s.row), dtype)}

    def token_positions(self) -> torch.Tensor:
        """``(B, 1, current_length)`` int32: position held by every row, −1 for empty ones."""
        seq = self.sequences
        pos = torch.tensor([seq.pos_host[s] for s in seq.batch], dtype=torch.int32)[:, None]
        row = torch.arange(self.current_length, dtype=torch.int32)[None]
        if self.plan.ring:
            head, ring = self.plan
            row = torch.where(row < head, row, pos - 1 - (pos - 1 - row) % ring)
            row = torch.where((row >= 0) & ((row >= head) | (torch.arange(row.shape[1])[None] < head)), row, torch.full_like(row, -1))
        return torch.where(row < pos, row, torch.full_like(row, -1))[:, None].to(self.device or "cpu")
