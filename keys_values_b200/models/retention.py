"""Retention mixer (linear attention with a fixed decay per head) of models described layer by layer.

Queries and keys are rotated (as in :mod:`keys_values_b200.models.grouped_attention`), keys scaled by dim^(−1/2). Per head, in fp32 and
carried per sequence by :class:`keys_values_b200.kvcache.recurrent.RetentionCache`: S_t = decay S_(t−1) + k_t v_t^T, o_t = S_t^T q_t.
o is RMS-normed per head without a weight, multiplied with silu of a gate projection and projected.

Several new tokens: queries and keys leave their product in fp32 and are rounded once, after the rotation; the recurrence is the
chunked kernel of the state-space mixers with a fixed decay. One new token: one product for everything, in fp32, and one kernel from
there to the gated output.
"""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from keys_values_b200.config import Config
from keys_values_b200.kvcache.sequences import SequencePass
from keys_values_b200.models.grouped_attention import rotation_frequencies
from keys_values_b200.models.packed import Packed, pad_groups, pad_last
from keys_values_b200.ops import layers as L

# log2 of the smallest decay that the chunked kernel tells from zero: a token further on nothing is left of a state either way
MIN_LOG2_DECAY = -100.0


def retention_shape(spec: Dict[str, Any]) -> L.RetentionShape:
    s = L.RetentionShape(heads=spec["n_head"], dim=spec["dim"], vdim=spec["v_dim"], rot_dims=spec.get("rope_dims") or 0)
    if s.rot_dims % 2 or s.rot_dims > s.dim:
        raise ValueError(f"{s.rot_dims} of {s.dim} dimensions rotated")
    if len(spec["decay"]) != s.heads or not all(0 <= d <= 1 for d in spec["decay"]):
        raise ValueError(f"decay must have a number in [0, 1] for each of {s.heads} heads")
    return s


class Retention(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        spec = config.layers[block_idx]["mixer"]
        s = self.shape = retention_shape(spec)
        self.spec = spec
        self.eps = config.norm_eps
        self.qkvg = nn.Linear(config.n_embd, 2 * s.heads * (s.dim + s.vdim), bias=False)  # rows queries | keys | values | gate
        self.proj = nn.Linear(s.heads * s.vdim, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        s, dev = self.shape, self.proj.weight.device
        qk, vg = torch.split(self.qkvg.weight, [2 * s.heads * s.dim, 2 * s.heads * s.vdim])
        decay = torch.tensor(self.spec["decay"], dtype=torch.float64)
        return {
            "in": torch.cat((pad_groups(qk, 2 * s.heads, s.np), pad_groups(vg, 2 * s.heads, s.vdp))).contiguous(),
            "decay": decay.to(device=dev, dtype=torch.float32),
            "log2_decay": decay.log2().clamp(min=MIN_LOG2_DECAY).to(device=dev, dtype=torch.float32),
            "freq": rotation_frequencies(self.spec).to(device=dev, dtype=torch.float32),
            "proj": pad_last(self.proj.weight.view(-1, s.heads, s.vdim), s.vdp).view(-1, s.inner),
        }

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; the states of the sequences move on."""
        s, w = self.shape, self.packed()
        B, T, width = x.shape
        state = self.kv_cache.allocate(x.device, x.dtype)[0][turn]
        flat = x.reshape(-1, width)
        if T == 1:
            u = L.linear_fp32(flat, w["in"]).view(B, T, -1)
            return F.linear(L.retention_step(u, w["freq"], w["decay"], state, seq, s, self.eps, x.dtype), w["proj"])
        qk = L.retention_prep(L.linear_fp32(flat, w["in"][: s.qk]).view(B, T, -1), w["freq"], seq, s, x.dtype)
        vg = F.linear(x, w["in"][s.qk :])
        y = L.retention_scan(qk, vg, w["decay"], w["log2_decay"], state, seq, s)
        return F.linear(L.head_norm_gate(y, vg[..., s.inner :], s, self.eps), w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.recurrent import RetentionCache

        if not isinstance(cache, RetentionCache) or cache.shape != self.shape:
            raise ValueError(f"layer {self.block_idx} needs a RetentionCache of its own sizes")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.recurrent import RetentionCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = RetentionCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
