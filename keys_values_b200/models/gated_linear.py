"""Gated linear attention of models described layer by layer: a linear attention whose decay is a number per token and key channel.

Per head, in fp32 and carried per sequence by :class:`keys_values_b200.kvcache.recurrent.GatedLinearCache`: S_t = diag(alpha_t) S_(t−1) +
k_t v_t^T, o_t = S_t^T q_t dim^(−1/2), with alpha = sigmoid(z)^(1 / tau) and z a low-rank projection of the input (``rank``) with a bias. o is
RMS-normed per head with one weight for all heads, multiplied with silu of a gate projection and projected.

Several new tokens: queries, keys and the low-rank input leave their product in fp32; one kernel makes the decays of 128 tokens at a time and
rounds queries and keys once, with the decay since (up to) the middle of the chunk in them, which leaves a masked product for the
chunked kernel of the other recurrences. One new token: one product for everything, in fp32, and one kernel from there to the gated output.
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

# bias of the decays of padded key channels: they keep their (zero) state
KEEP = 30.0


def gated_linear_shape(spec: Dict[str, Any]) -> L.GatedLinearShape:
    s = L.GatedLinearShape(heads=spec["n_head"], dim=spec["dim"], vdim=spec["v_dim"], rank=spec["rank"], tau=float(spec["tau"]))
    if min(s.heads, s.dim, s.vdim, s.rank) < 1 or not s.tau > 0:
        raise ValueError(f"sizes of a gated linear attention: {s}")
    return s


class GatedLinearAttention(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None, spec: Optional[Dict[str, Any]] = None) -> None:
        super().__init__()
        s = self.shape = gated_linear_shape(config.layers[block_idx]["mixer"] if spec is None else spec)
        self.eps = config.norm_eps
        self.parts = [2 * s.heads * s.dim, s.rank, 2 * s.heads * s.vdim]
        self.proj_in = nn.Linear(config.n_embd, sum(self.parts), bias=False)  # rows queries | keys | low rank | values | gate
        self.decay = nn.Parameter(torch.zeros(s.heads * s.dim, s.rank))
        self.decay_bias = nn.Parameter(torch.zeros(s.heads * s.dim))
        self.norm = nn.Parameter(torch.ones(s.vdim))
        self.proj = nn.Linear(s.heads * s.vdim, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx
        self.reset_parameters()

    def reset_parameters(self) -> None:
        """Decays around 0.97 to 0.999 at tau = 16."""
        with torch.no_grad():
            nn.init.normal_(self.decay, std=self.shape.rank**-0.5)
            self.decay_bias.copy_(torch.linspace(0.5, 4.5, self.decay_bias.numel()))

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        s = self.shape
        qk, low, vg = torch.split(self.proj_in.weight, self.parts)
        bias = F.pad(self.decay_bias.float().view(s.heads, s.dim), (0, s.np - s.dim), value=KEEP)
        return {
            "in": torch.cat((pad_groups(qk, 2 * s.heads, s.np), pad_groups(low, 1, s.rp), pad_groups(vg, 2 * s.heads, s.vdp))).contiguous(),
            "decay": pad_groups(self.decay.float(), s.heads, s.np).t().contiguous(),
            "decay_bias": bias.reshape(-1).contiguous(),
            "norm": pad_last(self.norm.float(), s.vdp),
            "proj": pad_last(self.proj.weight.view(-1, s.heads, s.vdim), s.vdp).view(-1, s.inner),
        }

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; the states of the sequences move on."""
        s, w = self.shape, self.packed()
        B, T, width = x.shape
        state = self.kv_cache.allocate(x.device, x.dtype)[0][turn]
        decay = L.DecayWeights(w["decay"], w["decay_bias"])
        flat = x.reshape(-1, width)
        if T == 1:
            u = L.linear_fp32(flat, w["in"]).view(B, T, -1)
            return F.linear(L.gated_linear_step(u, decay, w["norm"], state, seq, s, self.eps, x.dtype), w["proj"])
        n = s.qk + s.rp
        vg = F.linear(x, w["in"][n:])
        y = L.gated_linear_scan(L.linear_fp32(flat, w["in"][:n]).view(B, T, -1), vg, decay, state, seq, s)
        return F.linear(L.head_norm_gate(y, vg[..., s.inner :], s, self.eps, w["norm"]), w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.recurrent import GatedLinearCache

        if not isinstance(cache, GatedLinearCache) or cache.shape != self.shape:
            raise ValueError(f"layer {self.block_idx} needs a GatedLinearCache of its own sizes")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.recurrent import GatedLinearCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = GatedLinearCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
