"""State of a recurrent layer: per sequence the fp32 state of every head and, where the layer has a short convolution, its last
inputs.

The state ``(heads, state, vdim)`` has its sizes padded to multiples of 8 (padding stays zero). The convolution's inputs lie in
a ring of ``taps`` rows, position p in row ``p mod taps``: one row more than the convolution looks back, so that a step
writes a row that none of its readers wants. A sequence that starts at position 0 reads neither, so slots need no clearing.
"""
from __future__ import annotations

from typing import Optional

import torch

from keys_values_b200.config import Config
from keys_values_b200.kvcache.layer_cache import LayerCache


class RecurrentCache(LayerCache):
    """Holds a state per sequence and no tokens."""

    @property
    def state(self) -> Optional[torch.Tensor]:
        """``(turns, max_batch_size, heads, np, vdp)`` fp32."""
        return None if self.buffers_ is None else self.buffers_[0]

    @property
    def current_length(self) -> int:
        return self.input_pos

    def _shapes(self, dtype):
        s = self.shape
        return {"state": ((self.max_batch_size, s.heads, s.np, s.vdp), torch.float32)}

    def token_positions(self) -> torch.Tensor:
        raise NotImplementedError("a recurrent state holds no tokens")


class RetentionCache(RecurrentCache):
    kind = "retention"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.retention import retention_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        self.shape = retention_shape(self.spec)


class GatedLinearCache(RecurrentCache):
    kind = "gated_linear_attention"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.gated_linear import gated_linear_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        self.shape = gated_linear_shape(self.spec)


class GatedRecurrenceCache(RecurrentCache):
    """One number per channel instead of a matrix per head: state ``(turns, max_batch_size, channels)``."""

    kind = "gated_recurrence"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.gated_recurrence import recurrence_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        self.shape = recurrence_shape(self.spec)

    @property
    def conv(self) -> Optional[torch.Tensor]:
        """``(turns, max_batch_size, taps, channels)``."""
        return None if self.buffers_ is None else self.buffers_[1]

    def _shapes(self, dtype):
        s = self.shape
        return {"state": ((self.max_batch_size, s.channels), torch.float32), "conv": ((self.max_batch_size, s.taps, s.channels), dtype)}


class StateSpaceCache(RecurrentCache):
    kind = "mamba2"

    def __init__(self, config: Config, max_batch_size: int, cache_length: int, block_idx: int, dtype=None, device=None, **kwargs):
        from keys_values_b200.models.state_space import state_shape

        super().__init__(config, max_batch_size, cache_length, block_idx, dtype=dtype, device=device, **kwargs)
        self.shape = state_shape(self.spec)

    @property
    def conv(self) -> Optional[torch.Tensor]:
        """``(turns, max_batch_size, taps, channels)``."""
        return None if self.buffers_ is None else self.buffers_[1]

    def _shapes(self, dtype):
        return {**super()._shapes(dtype), "conv": ((self.max_batch_size, self.shape.taps, self.shape.channels), dtype)}
