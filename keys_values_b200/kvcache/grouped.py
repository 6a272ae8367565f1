"""Cache of a grouped-query attention layer: rotated keys and values.

One row per token and key/value head, ``[keys (padded to a multiple of 8, one per map) | value (the same)]``. Prompts and single
tokens attend over the cache as it lies. A layer that sees every earlier position keeps position p of the sequence in slot s in row p
of that slot. A layer that looks back a bounded way (a window or chunks) needs the rows of that span and of the pass at hand: if
the cache is longer, the first positions that stay visible have rows of their own and the others share a ring
(:class:`keys_values_b200.ops.layers.RowPlan`), in tiles of the attention kernels, so that a tile never wraps.

A window with pooled blocks has the rows of the blocks ahead of a ring of tokens: row b of the first ones holds the means of keys and values
of block b, written by the pass that brings the block's last token.

A layer that takes the keys and values of an earlier layer holds none (:class:`BorrowedKVCache`).
"""
from __future__ import annotations

from typing import Optional, Tuple

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

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.grouped_attention import grouped_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        s = self.shape = grouped_shape(self.spec)
        self.plan = RowPlan()
        if s.pool:
            self.plan = RowPlan(tiles(cache_length // s.pool), min(tiles(s.span + self.max_pass), tiles(cache_length)))
        elif s.span:
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

    @property
    def wraps(self) -> bool:
        """Whether positions of a sequence share rows."""
        return self.plan.ring > 0 and (not self.shape.pool or self.plan.ring < self.cache_length)

    def check_capacity(self, end: int) -> None:
        if end > self.cache_length and (self.shape.pool or not self.plan.ring):
            raise IndexError(f"layer {self.block_idx}: {end} tokens exceed the cache of {self.cache_length}")

    def check_pass(self, seq) -> None:
        super().check_pass(seq)
        if self.wraps and seq.length > self.plan.ring - self.shape.span:
            raise IndexError(f"layer {self.block_idx}: a pass of {seq.length} tokens exceeds the ring of {self.plan.ring} (take smaller portions)")

    def _shapes(self, dtype):
        s = self.shape
        return {"keys_values": ((self.max_batch_size, self.length, s.kv_heads, s.row), dtype)}

    def token_positions(self) -> torch.Tensor:
        """``(B, 1, current_length)`` int32: position held by every row, −1 for empty ones."""
        seq = self.sequences
        pos = torch.tensor([seq.pos_host[s] for s in seq.batch], dtype=torch.int32)[:, None]
        row = torch.arange(self.current_length, dtype=torch.int32)[None]
        if self.shape.pool:  # of the tokens; the rows of blocks hold none
            row = pos - 1 - (pos - 1 - torch.arange(min(self.input_pos, self.plan.ring), dtype=torch.int32)[None]) % self.plan.ring
            row = torch.where(row >= 0, row, torch.full_like(row, -1))
        elif self.plan.ring:
            head, ring = self.plan
            row = torch.where(row < head, row, pos - 1 - (pos - 1 - row) % ring)
            row = torch.where((row >= 0) & ((row >= head) | (torch.arange(row.shape[1])[None] < head)), row, torch.full_like(row, -1))
        return torch.where(row < pos, row, torch.full_like(row, -1))[:, None].to(self.device or "cpu")


class BorrowedKVCache(LayerCache):
    """Stands for the cache of an earlier layer (``kv_from``), which this layer reads and never writes."""

    kind = "grouped_attention"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        if self.spec.get("kv_from") is None:
            raise ValueError(f"layer {block_idx} has keys and values of its own")
        self._source: Tuple[GroupedKVCache, ...] = ()

    def get_source(self) -> GroupedKVCache:
        if not self._source:
            raise ValueError(f"the cache of layer {self.block_idx} stands for that of layer {self.spec['kv_from']}: assign both to a model")
        return self._source[0]

    def set_source(self, cache: GroupedKVCache) -> None:
        self._source = (cache,)  # not a module of this one

    @property
    def plan(self) -> RowPlan:
        return self.get_source().plan

    @property
    def current_length(self) -> int:
        return self.get_source().current_length

    def allocate(self, device, dtype):
        return self.get_source().allocate(device, dtype)

    def _shapes(self, dtype):
        return {}

    def token_positions(self) -> torch.Tensor:
        return self.get_source().token_positions()
