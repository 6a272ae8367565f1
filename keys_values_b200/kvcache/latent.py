"""Cache of a latent-attention layer: one row per token, shared by all heads.

A row holds the normed latent (from which every head's unrotated key and value follow by a matrix product) and the rotated
key part. A layer that sees a window of W tokens keeps the rows of the last W positions in a ring (position p in
slot ``p mod length``), so single-token steps attend over the ring as it lies, without masks or position tables; a
layer without a window keeps ``cache_length`` rows and refuses more. Sequences of a batch may have different lengths: positions
come from the model's :class:`keys_values_b200.kvcache.sequences.SequenceTable`.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from keys_values_b200.config import Config
from keys_values_b200.kvcache.base import KVCache, KVCacheParams, bits_for_torch_dtype


class LatentKVCache(KVCache):
    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **_ignored):
        from keys_values_b200.models.layered import latent_shape

        if config.layers is None or config.layers[block_idx]["mixer"]["kind"] != "latent_attention":
            raise ValueError(f"layer {block_idx} of {config.name!r} has no latent attention")
        super().__init__(config, max_batch_size, cache_length, block_idx, dtype)
        spec = config.layers[block_idx]["mixer"]
        self.window: Optional[int] = spec.get("window")
        self.shape = latent_shape(spec)
        self.ring_length = cache_length if self.window is None else min(cache_length, self.window)
        self._device = None if device is None else torch.device(device)
        self.ring: Optional[torch.Tensor] = None  # (max_batch_size, ring_length, shape.row)
        # SequenceTable of the model the cache is assigned to
        self.sequences = None

    @classmethod
    def from_config(cls, config: Config, max_batch_size: int, cache_length: int, block_idx: int, device=None, dtype=None, **kwargs):
        return cls(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)

    # ------------------------------------------------------------- properties
    @property
    def device(self):
        return self._device if self.ring is None else self.ring.device

    @property
    def input_pos(self) -> int:
        if self.sequences is None or not self.sequences.batch:
            return 0
        return max(self.sequences.pos_host[s] for s in self.sequences.batch)

    @property
    def batch_size(self) -> Optional[int]:
        return None if self.sequences is None or not self.sequences.batch else len(self.sequences.batch)

    @property
    def current_length(self) -> int:
        return min(self.input_pos, self.ring_length)

    @property
    def max_prefill_length(self) -> Optional[int]:
        return None  # a pass may have any length

    def max_forward_length(self) -> int:
        return self.config.block_size

    def check_capacity(self, end: int) -> None:
        """Raises if positions up to ``end`` cannot all stay visible as long as the layer's window wants."""
        if end > self.ring_length and (self.window is None or self.ring_length < self.window):
            raise IndexError(f"layer {self.block_idx}: {end} tokens exceed the cache of {self.ring_length}")

    # ---------------------------------------------------------------- storage
    def allocate(self, device, dtype) -> torch.Tensor:
        dtype = self._dtype or dtype
        if self.ring is None or self.ring.device != torch.device(device) or self.ring.dtype != dtype:
            with torch.inference_mode(False):
                self.ring = torch.zeros((self.max_batch_size, self.ring_length, self.shape.row), dtype=dtype, device=device)
        return self.ring

    def deallocate_buffers(self) -> None:
        self.ring = None

    def token_positions(self) -> torch.Tensor:
        """``(B, 1, ring_length)`` int32: position held by every slot of the ring, −1 for empty ones."""
        seq = self.sequences
        pos = torch.tensor([seq.pos_host[s] for s in seq.batch], dtype=torch.int64)[:, None]
        slot = torch.arange(self.ring_length)[None]
        held = pos - 1 - (pos - 1 - slot) % self.ring_length
        return torch.where((held >= 0) & (pos > 0), held, torch.full_like(held, -1)).to(torch.int32)[:, None].to(self.device or "cpu")

    def get_keys_values(self):
        return None  # keys and values exist per pass only

    def forward(self, *args, **kwargs):
        raise NotImplementedError("latent caches are driven by LatentAttention")

    def advance_host_counters(self) -> None:
        pass  # the model's SequenceTable counts

    # ------------------------------------------------------------------ sizes
    def size_estimate(self) -> Tuple[int, Dict[str, int]]:
        sz = self.max_batch_size * self.ring_length * self.shape.row * bits_for_torch_dtype(self.dtype or torch.float32)
        return sz, {"latents": sz}

    @classmethod
    def size_estimate_apriori(cls, params: KVCacheParams, **kwargs):
        raise NotImplementedError("sizes of latent caches depend on the layer; create them and call size_estimate")

    def clone(self, device=None) -> "LatentKVCache":
        other = LatentKVCache(self.config, self.max_batch_size, self.cache_length, self.block_idx, dtype=self._dtype, device=device or self._device)
        if self.ring is not None:
            other.ring = self.ring.clone() if device is None else self.ring.to(device, copy=True)
        return other
