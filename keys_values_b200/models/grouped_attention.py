"""Grouped-query attention of models described layer by layer, with its variants as entries of the description:

* ``qkv_bias``: the projections of queries, keys and values have biases;
* ``qk_norm``: RMS norm over the whole query and the whole key projection (``True``), or over every head with one weight for all heads
  (``"head"``) or without a weight (``"unit"``), before the rotation (without a weight the same as after it);
* ``temperature``: a learned factor of the scores per head;
* ``rope_base``, ``rope_dims``, ``rope_scale``: rotation of the first ``rope_dims`` dimensions of every head (pairs i and
  i + rope_dims / 2), angles position · base^(−2i / rope_dims) / rope_scale; ``rope_bands``: frequencies stretched by their wavelength,
  see :func:`band_frequencies`; ``rope_interleaved``: the pairs are 2i and 2i + 1 (the rows of the projections are put into the other
  order, alike for queries and keys, when the weights are packed);
* ``shared_value``: the values are the keys as projected (no norm, no rotation, no value projection);
* ``softcap``: scores become softcap · tanh(score / softcap);
* ``window`` and ``keep_first``: a position sees the last ``window`` positions and the first ``keep_first`` of the sequence;
  ``chunk``: it sees its own part of ``chunk`` positions; ``window`` and ``pool``: beside the window it sees the means of keys and of values
  of all blocks of ``pool`` positions that end before the window;
* ``kv_from``: the keys and values are those in the cache of an earlier layer, which has the same heads, sizes and rotation;
* ``sink``: one more term in the denominator of the softmax, exp(0) (``True``) or learned per head (``"learned"``);
* ``gate``: the heads' outputs are multiplied with sigmoid of one more projection of the mixer's input, one number per coordinate
  (``True``) or per head (``"head"``);
* ``differential``: every head has two queries and two keys over the same values; the result is the first map less lambda times the
  second, RMS-normed per head and times 1 − differential. lambda = exp(lq1 · lk1) − exp(lq2 · lk2) + differential.

Queries, keys, values and gate are one library product; one kernel norms, rotates and writes keys and values to the cache;
attention reads the cache as it lies and applies masks, difference and gate.
"""
from __future__ import annotations

import math
from dataclasses import replace
from typing import Any, Dict, Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from keys_values_b200.config import Config
from keys_values_b200.kvcache.sequences import SequencePass
from keys_values_b200.models.packed import Packed, pad_groups, pad_last
from keys_values_b200.ops import layers as L


def band_frequencies(freq: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequencies for contexts longer than the ``original`` one: wavelengths above original / low are stretched by ``factor``, those below
    original / high are left, between them the two are blended linearly in original / wavelength."""
    turns = original * freq / (2 * math.pi)  # of a pair over the original context
    share = (turns - low) / (high - low)
    blend = torch.where(turns < low, torch.zeros_like(share), torch.where(turns > high, torch.ones_like(share), share))
    return freq * (blend + (1 - blend) / factor)


def rotation_frequencies(spec: Dict[str, Any]) -> torch.Tensor:
    """Angle per position of every rotated pair, float64."""
    dims = spec.get("rope_dims") or 0
    if not dims:
        return torch.empty(0, dtype=torch.float64)
    freq = float(spec["rope_base"]) ** (torch.arange(dims // 2, dtype=torch.float64) * (-2.0 / dims)) / float(spec.get("rope_scale") or 1.0)
    return band_frequencies(freq, **spec["rope_bands"]) if spec.get("rope_bands") else freq


def grouped_shape(spec: Dict[str, Any]) -> L.GroupedShape:
    diff = spec.get("differential")
    s = L.GroupedShape(
        heads=spec["n_head"], kv_heads=spec["n_kv_head"], dim=spec["dim"], vdim=spec["v_dim"], rot_dims=spec.get("rope_dims") or 0,
        shared_value=bool(spec.get("shared_value")), gate=bool(spec.get("gate")), sink=bool(spec.get("sink")), scale=float(spec["scale"]),
        maps=1 if diff is None else 2, head_norm=spec.get("qk_norm") in ("head", "unit"), gate_per_head=spec.get("gate") == "head",
        softcap=float(spec.get("softcap") or 0.0), window=spec.get("window") or 0, keep=spec.get("keep_first") or 0 if spec.get("window") else 0,
        chunk=spec.get("chunk") or 0, post=1.0 if diff is None else 1.0 - float(diff), pool=spec.get("pool") or 0, borrowed=spec.get("kv_from") is not None,
    )
    if s.heads % s.kv_heads or s.rot_dims % 2 or s.rot_dims > s.dim:
        raise ValueError(f"attention of {s.heads} heads on {s.kv_heads} with {s.rot_dims} of {s.dim} dimensions rotated")
    if s.shared_value and (s.vdim != s.dim or s.maps != 1):
        raise ValueError(f"values that are the keys have one map and {s.dim} dimensions, not {s.vdim}")
    if not s.scale > 0 or s.softcap < 0:
        raise ValueError("attention scale must be positive, a soft cap not negative")
    if s.window and s.chunk:
        raise ValueError("a layer has a window or chunks, not both")
    if s.pool < 0 or s.pool and (not s.window or s.keep):
        raise ValueError("pooled blocks go with a window, and without kept first positions")
    if s.borrowed and s.shared_value:
        raise ValueError("values that are the keys cannot be another layer's")
    if s.maps == 2 and (s.sink or s.gate):
        raise NotImplementedError("differential attention with a sink or a gate")
    return s


def check_source(config: Config, block_idx: int) -> None:
    """Raises unless layer ``block_idx`` can use the keys and values of the layer that it names."""
    mixer = config.layers[block_idx]["mixer"]
    j = mixer["kv_from"]
    source = config.layers[j]["mixer"] if 0 <= j < block_idx else {}
    if source.get("kind") != "grouped_attention" or source.get("kv_from") is not None:
        raise ValueError(f"layer {block_idx} takes keys and values of layer {j}, which is no earlier attention layer with its own")
    if config.layer_turns(j) != config.layer_turns(block_idx):
        raise ValueError(f"layers {j} and {block_idx}, which share keys and values, are not run equally often")
    a, b = grouped_shape(source), grouped_shape(mixer)
    if (a.kv_heads, a.dim, a.vdim, a.maps) != (b.kv_heads, b.dim, b.vdim, b.maps) or not torch.equal(rotation_frequencies(source), rotation_frequencies(mixer)) \
            or bool(source.get("rope_interleaved")) != bool(mixer.get("rope_interleaved")):
        raise ValueError(f"layers {j} and {block_idx}, which share keys and values, differ in their sizes or their rotation")
    if a.pool or b.pool or a.span and (a.keep, a.chunk, a.window) != (b.keep, b.chunk, b.window):
        raise NotImplementedError(f"layer {j} does not keep all that layer {block_idx} sees")


class GroupedAttention(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None, spec: Optional[Dict[str, Any]] = None, scale: float = 1.0) -> None:
        """``scale``: factor of the result."""
        super().__init__()
        spec = config.layers[block_idx]["mixer"] if spec is None else spec
        s = self.shape = grouped_shape(spec)
        if s.borrowed:
            check_source(config, block_idx)
        self.result_scale = float(scale)
        self.spec = spec
        self.eps = config.norm_eps
        # rows: queries, keys (head by head, the maps of a head in a row), values (unless they are the keys, or both another layer's), gate
        H, G = s.heads * s.maps, s.kv_heads * s.maps
        self.parts = [H * s.dim]
        if not s.borrowed:
            self.parts += [G * s.dim] + ([] if s.shared_value else [s.kv_heads * s.vdim])
        self.gate_rows = 0 if not s.gate else s.heads if s.gate_per_head else s.heads * s.vdim
        self.qkv = nn.Linear(config.n_embd, sum(self.parts) + self.gate_rows, bias=False)
        self.qkv_bias = nn.Parameter(torch.zeros(sum(self.parts))) if spec.get("qkv_bias") else None
        norm = spec.get("qk_norm")
        if norm == "unit":
            norm = None  # nothing to learn
        self.norm_q = nn.Parameter(torch.ones(s.dim if norm == "head" else H * s.dim)) if norm else None
        self.norm_k = nn.Parameter(torch.ones(s.dim if norm == "head" else G * s.dim)) if norm else None
        self.temperature = nn.Parameter(torch.ones(s.heads)) if spec.get("temperature") else None
        self.sink = nn.Parameter(torch.zeros(s.heads)) if spec.get("sink") == "learned" else None
        # rows lq1, lk1, lq2, lk2
        self.map_weights = nn.Parameter(torch.zeros(4, s.dim)) if s.maps == 2 else None
        self.proj = nn.Linear(s.heads * s.vdim, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx

    @property
    def inner(self) -> int:
        return self.shape.inner

    def _halves(self, w: torch.Tensor, heads: int) -> torch.Tensor:
        """Rows of ``heads`` heads whose rotated pairs are neighbours, put so that the pairs are half of the rotated rows apart."""
        s = self.shape
        if not self.spec.get("rope_interleaved") or not s.rot_dims:
            return w
        order = torch.cat((torch.arange(0, s.rot_dims, 2), torch.arange(1, s.rot_dims, 2), torch.arange(s.rot_dims, s.dim))).to(w.device)
        return w.view(heads, s.dim, *w.shape[1:])[:, order].reshape(w.shape)

    def _pad_rows(self, w: torch.Tensor, gate: bool) -> torch.Tensor:
        """Rows of the joint projection, every head padded and the whole padded to its leading dimension."""
        s = self.shape
        parts = list(torch.split(w, self.parts + ([self.gate_rows] if gate and self.gate_rows else [])))
        H, G = s.heads * s.maps, s.kv_heads * s.maps
        out = [pad_groups(self._halves(parts[0], H), H, s.dimp)]
        if not s.borrowed:
            out.append(pad_groups(self._halves(parts[1], G), G, s.dimp))
            if not s.shared_value:
                out.append(pad_groups(parts[2], s.kv_heads, s.vdp))
        if gate and self.gate_rows:
            out.append(pad_groups(parts[-1], s.heads, s.gate_cols))
        out = torch.cat(out)
        return F.pad(out, (0, 0) * (out.ndim - 1) + (0, s.ld - out.shape[0])).contiguous()

    def _pad_norm(self, w: Optional[torch.Tensor], heads: int) -> Optional[torch.Tensor]:
        s = self.shape
        if self.spec.get("qk_norm") == "unit":
            return torch.ones(s.dimp, device=self.proj.weight.device)
        if w is None:
            return None
        w = self._halves(w.float(), 1 if s.head_norm else heads * s.maps)
        return pad_last(w, s.dimp) if s.head_norm else pad_groups(w, heads * s.maps, s.dimp)

    def _make_pack(self) -> Dict[str, Any]:
        s = self.shape
        if s.maps == 2:
            a = self.map_weights.double()
            lam = float(torch.exp((a[0] * a[1]).sum()) - torch.exp((a[2] * a[3]).sum())) + float(self.spec["differential"])
            s = replace(s, lam=lam, eps=self.eps)
        if self.result_scale != 1.0:
            s = replace(s, post=s.post * self.result_scale)
        w = self.qkv.weight
        return {
            "shape": s,
            "in": self._pad_rows(w, True),
            "bias": None if self.qkv_bias is None else self._pad_rows(self.qkv_bias, False),
            "norm_q": self._pad_norm(self.norm_q, s.heads),
            "norm_k": self._pad_norm(self.norm_k, s.kv_heads),
            "temperature": None if self.temperature is None else self.temperature.float().contiguous(),
            "sink": None if self.sink is None else self.sink.float().contiguous(),
            "freq": rotation_frequencies(self.spec).to(device=w.device, dtype=torch.float32),
            "proj": pad_last(self.proj.weight.view(-1, s.heads, s.vdim), s.vdp).view(-1, s.heads * s.vdp),
        }

    def core(self, u: torch.Tensor, seq: SequencePass, turn: int, cache, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """From the input projection ``u (B, T, ·)`` to what the output projection reads, ``(B, T, inner)``."""
        w = self.packed()
        s, plan = w["shape"], cache.plan
        rows = cache.allocate(u.device, u.dtype)[0][turn]
        q = L.grouped_prep(u, w["norm_q"], w["norm_k"], w["freq"], rows, seq, s, self.eps, plan, w["temperature"])
        return L.grouped_attend(q, u, rows, seq, s, w["sink"], plan, out)

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; the cache takes the keys and values of the pass."""
        w = self.packed()
        return F.linear(self.core(F.linear(x, w["in"], w["bias"]), seq, turn, self.kv_cache), w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.grouped import BorrowedKVCache, GroupedKVCache

        if self.shape.borrowed:
            if not isinstance(cache, BorrowedKVCache):
                raise ValueError(f"layer {self.block_idx} has no keys and values of its own")
        elif not isinstance(cache, GroupedKVCache) or cache.shape != self.shape:
            raise ValueError(f"layer {self.block_idx} needs a GroupedKVCache of its own sizes")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.layer_cache import LayerCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = LayerCache.from_config(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)
