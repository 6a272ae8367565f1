"""Mamba-2 mixer (state-space duality) of models described layer by layer.

One library product gives gate z, x, B, C and the step sizes dt. x, B and C pass a short causal convolution with silu. Per head,
with decay a_t = exp(−exp(A_log) · dt_t): S_t = a_t S_(t−1) + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t, in fp32 and carried per
sequence by :class:`keys_values_b200.kvcache.recurrent.StateSpaceCache`. y · silu(z) is RMS-normed in equal parts and projected.

Several new tokens: convolution, then a kernel that takes the tokens chunk by chunk (products within a chunk, the state between
chunks). One new token: convolution, decay, state and output are one kernel.
"""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from keys_values_b200.config import Config
from keys_values_b200.kvcache.sequences import SequencePass
from keys_values_b200.models.packed import Packed, pad_groups, pad_last
from keys_values_b200.ops import layers as L


def state_shape(spec: Dict[str, Any]) -> L.StateShape:
    s = L.StateShape(heads=spec["n_head"], vdim=spec["v_dim"], state=spec["state"], groups=spec["groups"],
                     norm_groups=spec["norm_groups"], taps=spec["conv"])
    if s.heads % s.groups or (s.heads * s.vdim) % s.norm_groups or s.taps < 1:
        raise ValueError(f"sizes of a state-space mixer do not fit each other: {s}")
    return s


class Mamba2Mixer(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        s = self.shape = state_shape(config.layers[block_idx]["mixer"])
        self.eps = config.norm_eps
        inner, bc = s.heads * s.vdim, s.groups * s.state
        self.proj_in = nn.Linear(config.n_embd, 2 * inner + 2 * bc + s.heads, bias=False)  # rows z | x | B | C | dt
        self.conv = nn.Parameter(torch.zeros(inner + 2 * bc, s.taps))
        self.conv_bias = nn.Parameter(torch.zeros(inner + 2 * bc))
        self.dt_bias = nn.Parameter(torch.zeros(s.heads))
        self.a_log = nn.Parameter(torch.zeros(s.heads))
        self.skip = nn.Parameter(torch.ones(s.heads))
        self.norm = nn.Parameter(torch.ones(inner))
        self.proj = nn.Linear(inner, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx
        self.reset_parameters()

    def reset_parameters(self) -> None:
        """Decay rates 1 … 16, step sizes around 0.02."""
        with torch.no_grad():
            nn.init.normal_(self.conv, std=self.shape.taps**-0.5)
            self.a_log.copy_(torch.linspace(1, 16, self.shape.heads).log())
            self.dt_bias.fill_(-4.0)

    def _pad_channels(self, w: torch.Tensor) -> torch.Tensor:
        """Rows ``x | B | C`` with every head and every group padded."""
        s = self.shape
        inner, bc = s.heads * s.vdim, s.groups * s.state
        x, b, c = torch.split(w, [inner, bc, bc])
        return torch.cat((pad_groups(x, s.heads, s.vdp), pad_groups(b, s.groups, s.np), pad_groups(c, s.groups, s.np)))

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        s = self.shape
        inner = s.heads * s.vdim
        w = self.proj_in.weight
        z, rest, dt = w[:inner], w[inner : w.shape[0] - s.heads], w[w.shape[0] - s.heads :]
        joint = torch.cat((pad_groups(z, s.heads, s.vdp), self._pad_channels(rest), dt))
        return {
            "in": F.pad(joint, (0, 0, 0, s.ld - joint.shape[0])).contiguous(),
            "conv": self._pad_channels(self.conv.float()).t().contiguous(),  # (taps, channels)
            "conv_bias": self._pad_channels(self.conv_bias.float()),
            "dt_bias": self.dt_bias.float().contiguous(),
            "a_log": self.a_log.float().contiguous(),
            "skip": self.skip.float().contiguous(),
            "norm": pad_groups(self.norm.float(), s.heads, s.vdp),
            "proj": pad_last(self.proj.weight.view(-1, s.heads, s.vdim), s.vdp).view(-1, s.heads * s.vdp),
        }

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; state and convolution inputs of the sequences move on."""
        s, w = self.shape, self.packed()
        u = F.linear(x, w["in"])
        state, ring = (t[turn] for t in self.kv_cache.allocate(x.device, x.dtype))
        if x.shape[1] == 1:
            y = L.state_step(u, w["conv"], w["conv_bias"], w["dt_bias"], w["a_log"], w["skip"], ring, state, seq, s)
        else:
            xbc = L.short_conv(u, s.inner, w["conv"], w["conv_bias"], ring, seq)
            y = L.state_scan(u, xbc, w["dt_bias"], w["a_log"], w["skip"], state, seq, s)
        return F.linear(L.gated_group_norm(y, u, w["norm"], s, self.eps), w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.recurrent import StateSpaceCache

        if not isinstance(cache, StateSpaceCache) or cache.shape != self.shape:
            raise ValueError(f"layer {self.block_idx} needs a StateSpaceCache of its own sizes")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.recurrent import StateSpaceCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = StateSpaceCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
