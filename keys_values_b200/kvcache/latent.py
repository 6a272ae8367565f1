"""Cache of a latent-attention layer: one row per token, shared by all heads.

A row holds the normed latent (from which every head's unrotated key and value follow by a matrix product) and the rotated
key part. A layer that sees a window of W tokens keeps the rows of the last W positions in a ring (position p in
slot ``p mod length``), so single-token steps attend over the ring as it lies, without masks or position tables; a
layer without a window keeps ``cache_length`` rows and refuses more. Sequences of a batch may have different lengths: positions
come from the model's :class:`keys_values_b200.kvcache.sequences.SequenceTable`.
"""
from __future__ import annotations

from typing import Optional

import torch

from keys_values_b200.config import Config
from keys_values_b200.kvcache.layer_cache import LayerCache


class LatentKVCache(LayerCache):
    kind = "latent_attention"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.layered import latent_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        spec = self.spec
        self.window: Optional[int] = spec.get("window")
        self.shape = latent_shape(spec)
        self.ring_length = cache_length if self.window is None else min(cache_length, self.window)

    @property
    def ring(self) -> Optional[torch.Tensor]:
        """``(turns, max_batch_size, ring_length, shape.row)``."""
        return None if self.buffers_ is None else self.buffers_[0]

    @property
    def current_length(self) -> int:
        return min(self.input_pos, self.ring_length)

    def check_capacity(self, end: int) -> None:
        """Raises if positions up to ``end`` cannot all stay visible as long as the layer's window wants."""
        if end > self.ring_length and (self.window is None or self.ring_length < self.window):
            raise IndexError(f"layer {self.block_idx}: {end} tokens exceed the cache of {self.ring_length}")

    def _shapes(self, dtype):
        return {"latents": ((self.max_batch_size, self.ring_length, self.shape.row), dtype)}

    def token_positions(self) -> torch.Tensor:
        """``(B, 1, ring_length)`` int32: position held by every slot of the ring, −1 for empty ones."""
        seq = self.sequences
        pos = torch.tensor([seq.pos_host[s] for s in seq.batch], dtype=torch.int64)[:, None]
        slot = torch.arange(self.ring_length)[None]
        held = pos - 1 - (pos - 1 - slot) % self.ring_length
        return torch.where((held >= 0) & (pos > 0), held, torch.full_like(held, -1)).to(torch.int32)[:, None].to(self.device or "cpu")
