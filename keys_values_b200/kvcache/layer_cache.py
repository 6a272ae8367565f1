"""Caches of models that are described layer by layer: what a mixer keeps per sequence, with one slot per sequence.

Positions, slots and batches belong to the model's :class:`keys_values_b200.kvcache.sequences.SequenceTable`; a cache
only owns memory of fixed size and address, so any single-token pass can be captured in a CUDA graph. A layer that is run
several times in a pass (``config.loop``) has one region per run (``turns``) in its cache.
"""
from __future__ import annotations

from typing import Any, Dict, Optional, Tuple, Type

import torch

from keys_values_b200.config import Config
from keys_values_b200.kvcache.base import KVCache, KVCacheParams, bits_for_torch_dtype


# tokens that one pass of a chunked prefill takes at most, all rows together; rings of bounded layers have room for as many
MAX_PASS_TOKENS = 16384


class LayerCache(KVCache):
    kind: str  # of the mixer that the cache serves

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, spec=None, **_ignored):
        """``spec``: description of the mixer, if it is a part of the layer's."""
        self.spec: Dict[str, Any] = (None if config.layers is None else config.layers[block_idx]["mixer"]) if spec is None else spec
        if self.spec is None or self.spec["kind"] != self.kind:
            raise ValueError(f"layer {block_idx} of {config.name!r} has no {self.kind.replace('_', ' ')} mixer")
        super().__init__(config, max_batch_size, cache_length, block_idx, dtype)
        self.turns = config.layer_turns(block_idx)
        self._device = None if device is None else torch.device(device)
        self.buffers_: Optional[Tuple[torch.Tensor, ...]] = None
        # SequenceTable of the model the cache is assigned to
        self.sequences = None

    @classmethod
    def from_config(cls, config: Config, max_batch_size: int, cache_length: int, block_idx: int, device=None, dtype=None, **kwargs):
        if cls is LayerCache:
            spec = {"kind": None} if config.layers is None else config.layers[block_idx]["mixer"]
            return layer_cache_class(spec)(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        return cls(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)

    # ------------------------------------------------------------- properties
    @property
    def device(self):
        return self._device if self.buffers_ is None else self.buffers_[0].device

    @property
    def input_pos(self) -> int:
        if self.sequences is None or not self.sequences.batch:
            return 0
        return max(self.sequences.pos_host[s] for s in self.sequences.batch)

    @property
    def batch_size(self) -> Optional[int]:
        return None if self.sequences is None or not self.sequences.batch else len(self.sequences.batch)

    @property
    def max_prefill_length(self) -> Optional[int]:
        return None  # a pass may have any length

    def max_forward_length(self) -> int:
        return self.config.block_size

    def check_capacity(self, end: int) -> None:
        """Raises if positions up to ``end`` cannot all be kept as long as the layer needs them."""

    def check_pass(self, seq) -> None:
        """Raises if the pass cannot be worked on."""
        self.check_capacity(seq.max_end)

    # ---------------------------------------------------------------- storage
    def _shapes(self, dtype: torch.dtype) -> Dict[str, Tuple[Tuple[int, ...], torch.dtype]]:
        """Name, shape (of one turn) and type of every buffer."""
        raise NotImplementedError

    def allocate(self, device, dtype) -> Tuple[torch.Tensor, ...]:
        """The buffers ``(turns, max_batch_size, ...)``, made on first use."""
        dtype = self._dtype or dtype
        shapes = self._shapes(dtype)
        held = self.buffers_
        if held is None or held[0].device != torch.device(device) or any(t.dtype != d for t, (_, d) in zip(held, shapes.values())):
            with torch.inference_mode(False):
                self.buffers_ = tuple(torch.zeros((self.turns, *shape), dtype=d, device=device) for shape, d in shapes.values())
        return self.buffers_

    def deallocate_buffers(self) -> None:
        self.buffers_ = None

    def get_keys_values(self):
        return None

    def forward(self, *args, **kwargs):
        raise NotImplementedError("caches of described layers are driven by their mixers")

    def advance_host_counters(self) -> None:
        pass  # the model's SequenceTable counts

    # ------------------------------------------------------------------ sizes
    def size_estimate(self) -> Tuple[int, Dict[str, int]]:
        sizes = {}
        for name, (shape, dtype) in self._shapes(self._dtype or torch.float32).items():
            n = self.turns * bits_for_torch_dtype(dtype)
            for x in shape:
                n *= x
            sizes[name] = n
        return sum(sizes.values()), sizes

    @classmethod
    def size_estimate_apriori(cls, params: KVCacheParams, **kwargs):
        raise NotImplementedError("sizes of these caches depend on the layer; create them and call size_estimate")

    def clone(self, device=None) -> "LayerCache":
        other = type(self)(self.config, self.max_batch_size, self.cache_length, self.block_idx, dtype=self._dtype, device=device or self._device,
                           spec=self.spec)
        if self.buffers_ is not None:
            other.buffers_ = tuple(t.clone() if device is None else t.to(device, copy=True) for t in self.buffers_)
        return other


class SideBySideCache(LayerCache):
    """Caches of two mixers that read the same input, each of the class that its mixer needs."""

    kind = "side_by_side"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, spec=None, **kwargs):
        self.parts: Tuple[LayerCache, ...] = ()
        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, spec=spec)
        self.parts = tuple(layer_cache_class(s)(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, spec=s, **kwargs)
                           for s in (self.spec["left"], self.spec["right"]))

    @property
    def sequences(self):
        return self._sequences

    @sequences.setter
    def sequences(self, value) -> None:
        self._sequences = value
        for p in self.parts:
            p.sequences = value

    @property
    def device(self):
        return self.parts[0].device

    @property
    def current_length(self) -> int:
        return max(p.current_length for p in self.parts)

    def check_capacity(self, end: int) -> None:
        for p in self.parts:
            p.check_capacity(end)

    def check_pass(self, seq) -> None:
        for p in self.parts:
            p.check_pass(seq)

    def deallocate_buffers(self) -> None:
        for p in self.parts:
            p.deallocate_buffers()

    def token_positions(self) -> torch.Tensor:
        return self.parts[0].token_positions()

    def size_estimate(self) -> Tuple[int, Dict[str, int]]:
        total, sizes = 0, {}
        for side, p in zip(("left", "right"), self.parts):
            n, detail = p.size_estimate()
            total += n
            sizes.update({f"{side}.{k}": v for k, v in detail.items()})
        return total, sizes

    def clone(self, device=None) -> "SideBySideCache":
        other = super().clone(device)
        other.parts = tuple(p.clone(device) for p in self.parts)
        return other


def layer_cache_class(spec: Dict[str, Any]) -> Type[LayerCache]:
    """The cache class that serves the mixer described by ``spec``."""
    from keys_values_b200.kvcache.grouped import BorrowedKVCache, GroupedKVCache
    from keys_values_b200.kvcache.latent import LatentKVCache
    from keys_values_b200.kvcache.recurrent import GatedLinearCache, GatedRecurrenceCache, RetentionCache, StateSpaceCache

    if spec.get("kv_from") is not None:
        return BorrowedKVCache
    classes = {c.kind: c for c in (LatentKVCache, GroupedKVCache, StateSpaceCache, RetentionCache, GatedLinearCache, GatedRecurrenceCache, SideBySideCache)}
    if spec["kind"] not in classes:
        raise ValueError(f"no cache for mixers of kind {spec['kind']!r}")
    return classes[spec["kind"]]
