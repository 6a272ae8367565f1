"""Two mixers that read the same input and whose results are added, each with a factor.

Description: ``left`` and ``right`` (descriptions of mixers), ``left_scale`` and ``right_scale``. The input projections of both are one product
and so are the output projections: the mixers leave their results, factors applied, side by side in one buffer. A mixer can be part of this if
it has ``core`` (from its input projection to what its output projection reads), ``inner`` and packed weights ``in``, ``bias`` and ``proj``.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch
import torch.nn.functional as F

from keys_values_b200.config import Config
from keys_values_b200.kvcache.sequences import SequencePass
from keys_values_b200.models.gated_recurrence import GatedRecurrence
from keys_values_b200.models.grouped_attention import GroupedAttention
from keys_values_b200.models.packed import Packed

PARTS = {"grouped_attention": GroupedAttention, "gated_recurrence": GatedRecurrence}


class SideBySide(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        spec = config.layers[block_idx]["mixer"]
        for side in ("left", "right"):
            if spec[side]["kind"] not in PARTS:
                raise ValueError(f"layer {block_idx}: mixer {spec[side]['kind']!r} beside another one")
            if spec[side].get("kv_from") is not None:
                raise NotImplementedError(f"layer {block_idx}: keys and values of another layer beside another mixer")
        self.left, self.right = (PARTS[spec[s]["kind"]](config, block_idx, spec=spec[s], scale=float(spec[f"{s}_scale"])) for s in ("left", "right"))
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx

    def _make_pack(self) -> Dict[str, Optional[torch.Tensor]]:
        a, b = self.left.packed(), self.right.packed()
        bias = None
        if a["bias"] is not None or b["bias"] is not None:
            bias = torch.cat([w["in"].new_zeros(w["in"].shape[0]) if w["bias"] is None else w["bias"] for w in (a, b)])
        return {"in": torch.cat((a["in"], b["in"])), "bias": bias, "proj": torch.cat((a["proj"], b["proj"]), dim=1), "cols": a["in"].shape[0]}

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; the caches of both take the pass."""
        w, n = self.packed(), self.left.inner
        u = F.linear(x, w["in"], w["bias"])
        y = torch.empty((*x.shape[:2], n + self.right.inner), dtype=x.dtype, device=x.device)
        left, right = self.kv_cache.parts
        self.left.core(u[..., : w["cols"]], seq, turn, left, y[..., :n])
        self.right.core(u[..., w["cols"] :], seq, turn, right, y[..., n:])
        return F.linear(y, w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.layer_cache import SideBySideCache

        if not isinstance(cache, SideBySideCache):
            raise ValueError(f"layer {self.block_idx} needs a SideBySideCache")
        self.left.check_kv_cache(cache.parts[0])
        self.right.check_kv_cache(cache.parts[1])

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.layer_cache import SideBySideCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = SideBySideCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
