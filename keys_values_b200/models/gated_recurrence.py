"""Gated recurrence per channel (Griffin's recurrent block with its real-gated linear recurrent unit) of models described layer by layer.

Two branches: y = gelu(W_y h + b) and x, W_x h + b after a short causal convolution with a bias. Gates r and i are sigmoids of square products
of x with biases, each within one of ``blocks`` equal parts of the channels. Per channel, in fp32 and carried per sequence by
:class:`keys_values_b200.kvcache.recurrent.GatedRecurrenceCache`: log a = −8 r softplus(lam), S_t = a S_(t−1) + sqrt(1 − a²) i x. The
result S · y is projected.

Several new tokens: convolution, the gates' products (library, fp32 results), then one kernel from there to S · y. One new token: everything
between the projections is one kernel.
"""
from __future__ import annotations

import math
from typing import Any, Dict, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from keys_values_b200.config import Config
from keys_values_b200.kvcache.sequences import SequencePass
from keys_values_b200.models.packed import Packed, pad_groups, pad_last
from keys_values_b200.ops import layers as L

RATE = -8.0  # logarithm of the decay at an open gate, in units of softplus(lam)


def recurrence_shape(spec: Dict[str, Any]) -> L.RecurrenceShape:
    s = L.RecurrenceShape(width=spec["width"], blocks=spec["blocks"], taps=spec["conv"])
    if s.blocks < 1 or s.width % s.blocks or s.taps < 1:
        raise ValueError(f"sizes of a gated recurrence do not fit each other: {s}")
    return s


class GatedRecurrence(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None, spec: Optional[Dict[str, Any]] = None, scale: float = 1.0) -> None:
        """``scale``: factor of the result."""
        super().__init__()
        s = self.shape = recurrence_shape(config.layers[block_idx]["mixer"] if spec is None else spec)
        self.scale = float(scale)
        self.proj_in = nn.Linear(config.n_embd, 2 * s.width, bias=True)  # rows y | x
        self.conv = nn.Parameter(torch.zeros(s.width, s.taps))
        self.conv_bias = nn.Parameter(torch.zeros(s.width))
        self.gate_r = nn.Parameter(torch.zeros(s.blocks, s.part, s.part))  # (out, in) of every part
        self.gate_i = nn.Parameter(torch.zeros(s.blocks, s.part, s.part))
        self.gate_r_bias = nn.Parameter(torch.zeros(s.blocks, s.part))
        self.gate_i_bias = nn.Parameter(torch.zeros(s.blocks, s.part))
        self.lam = nn.Parameter(torch.zeros(s.width))
        self.proj = nn.Linear(s.width, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx
        self.reset_parameters()

    def reset_parameters(self) -> None:
        """Decays 0.9 … 0.999 at an open gate."""
        s = self.shape
        with torch.no_grad():
            nn.init.normal_(self.conv, std=s.taps**-0.5)
            for w in (self.gate_r, self.gate_i):
                nn.init.normal_(w, std=s.part**-0.5)
            wanted = torch.linspace(0.9, 0.999, s.width).log() / RATE
            self.lam.copy_(torch.log(torch.expm1(wanted)))

    @property
    def inner(self) -> int:
        return self.shape.inner

    def _make_pack(self) -> Dict[str, Optional[torch.Tensor]]:
        s = self.shape

        def channels(w: torch.Tensor) -> torch.Tensor:
            return pad_groups(w.float(), s.blocks, s.pp)

        def gate(w: torch.Tensor) -> torch.Tensor:
            return F.pad(w.transpose(1, 2), (0, s.pp - s.part, 0, s.pp - s.part))

        return {
            "in": pad_groups(self.proj_in.weight, 2 * s.blocks, s.pp).contiguous(),
            "bias": pad_groups(self.proj_in.bias, 2 * s.blocks, s.pp).contiguous(),
            "mix": L.RecurrenceWeights(
                conv=channels(self.conv).t().contiguous(), conv_bias=channels(self.conv_bias), gates=torch.cat((gate(self.gate_r), gate(self.gate_i)), -1).contiguous(),
                bias_r=channels(self.gate_r_bias.view(-1)), bias_i=channels(self.gate_i_bias.view(-1)),
                rate=channels(RATE / math.log(2.0) * F.softplus(self.lam.double(), threshold=1e9)),
            ),
            "proj": pad_last(self.proj.weight.view(-1, s.blocks, s.part), s.pp).view(-1, s.channels),
        }

    def core(self, u: torch.Tensor, seq: SequencePass, turn: int, cache, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """From the input projection ``u (B, T, ·)`` to what the output projection reads, ``(B, T, inner)``."""
        s, w = self.shape, self.packed()
        state, ring = (t[turn] for t in cache.allocate(u.device, u.dtype))
        if out is None:
            out = torch.empty((*u.shape[:2], s.inner), dtype=u.dtype, device=u.device)
        return L.gated_recurrence(u, w["mix"], ring, state, seq, s, self.scale, out)

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; state and convolution inputs of the sequences move on."""
        w = self.packed()
        return F.linear(self.core(F.linear(x, w["in"], w["bias"]), seq, turn, self.kv_cache), w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.recurrent import GatedRecurrenceCache

        if not isinstance(cache, GatedRecurrenceCache) or cache.shape != self.shape:
            raise ValueError(f"layer {self.block_idx} needs a GatedRecurrenceCache of its own sizes")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.recurrent import GatedRecurrenceCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = GatedRecurrenceCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
