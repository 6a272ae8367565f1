"""Ops of models that are described layer by layer (fp32 residual stream, latent attention, routed experts).

A CUDA tensor is always served by the kernels of ``libkvb200_layers.so`` (bf16 or fp32; anything else
raises), a CPU tensor by the PyTorch restatement in :mod:`keys_values_b200.ops.layers_reference`.

``seq`` is the :class:`keys_values_b200.kvcache.sequences.SequencePass` of the pass: slots, start positions and
token counts of its rows.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class LatentShape:
    """Sizes of one latent attention; the padded ones are multiples of 8."""

    heads: int
    dim: int
    rot: int
    vdim: int
    kv_rank: int
    rot_dims: int

    @property
    def dimp(self) -> int:
        return round8(self.dim)

    @property
    def rp(self) -> int:
        return round8(self.rot)

    @property
    def vdp(self) -> int:
        return round8(self.vdim)

    @property
    def kvp(self) -> int:
        return round8(self.kv_rank)

    @property
    def row(self) -> int:
        """Width of a latent row: latent and rotated key part."""
        return self.kvp + self.rp


def _impl(t: torch.Tensor):
    if t.is_cuda:
        from keys_values_b200.ops import layers_cuda as impl
    else:
        from keys_values_b200.ops import layers_reference as impl
    return impl


# ---- layer edges
def embed_edge(idx, prev_token, embed, bigram, buckets, mul_prev, mul_cur, hist, gain, shift, state, h, hs, seq, eps) -> None:
    """``hist (B, T, width)`` fp32 = token (+ bigram) embedding; then norm and token shift of the first layer, see
    :func:`layer_edge`. A bigram row is ``(previous · mul_prev + current · mul_cur) mod buckets``; a sequence's first
    token has row ``buckets``."""
    _impl(idx).embed_edge(idx, prev_token, embed, bigram, buckets, mul_prev, mul_cur, hist, gain, shift, state, h, hs, seq, eps)


def layer_edge(x_in, mix, experts, hist, n_hist: int, coef, x_out, gain, shift, state, h, hs, seq, eps) -> None:
    """``new = x_in + mix + Σ_k weight_k · expert output_k``; ``x_out = Σ_j coef[j] · hist[j]`` with ``hist[n_hist] = new``
    (``coef None``: ``x_out = new``); ``h = x_out / rms · gain``; ``hs = h + (h of the token before − h) · shift``, with the
    ``state (slots, width)`` holding h of every sequence's last token. ``experts``: ``(out, row, weight)`` of
    :func:`routed_experts` or ``None``. ``gain None`` stops after ``x_out``, ``shift None`` after ``h``."""
    out, row, weight = experts if experts is not None else (None, None, None)
    _impl(x_in).layer_edge(x_in, mix, out, row, weight, hist, n_hist, coef, x_out, gain, shift, state, h, hs, seq, eps)


def scalar_rmsnorm(x: torch.Tensor, gain: torch.Tensor, eps: float, dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rows of ``x (n, width)`` fp32 divided by their root mean square, times the number ``gain``."""
    return _impl(x).scalar_rmsnorm(x, rows, gain, eps, dtype)


def sequence_advance(idx, pos, prev_token, seq) -> None:
    _impl(idx).sequence_advance(idx, pos, prev_token, seq)


# ---- products whose result stays in 32 bits
def linear_fp32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``x (n, k) · weight (m, k)^T`` with an fp32 result (the inputs keep their type)."""
    if x.dtype == torch.float32 and weight.dtype == torch.float32:
        return x @ weight.t()
    if x.is_cuda:
        return torch.mm(x, weight.t(), out_dtype=torch.float32)
    return x.float() @ weight.float().t()


# ---- latent attention
def latent_prep(qkv, norm_w, freq, latent, ring, seq, P: int, shape: LatentShape, eps: float) -> torch.Tensor:
    """Split of the joint projection ``qkv (B, T, ·)``, norm of the latents, rotation. Returns padded queries
    ``(B, T, heads, dimp + rp)``; latent rows go to ``latent[:, P:]`` and those of the last tokens of every sequence (at most
    the ring's length) into ``ring``, either of which may be ``None``."""
    return _impl(qkv).latent_prep(qkv, norm_w, freq, latent, ring, seq, P, shape, eps)


def ring_gather(ring, latent, seq, P: int) -> None:
    """``latent[:, :P]`` = rows of the ``P`` positions before the pass (zero where a sequence has none)."""
    if P > 0:
        _impl(ring).ring_gather(ring, latent, seq, P)


def latent_attend(q, kv, latent, seq, P: int, shape: LatentShape, window: int, scale: float) -> torch.Tensor:
    """``q (B, T, heads, dimp + rp)`` against ``kv (B, P + T, heads, dimp + vdp)`` and the rotated key parts of
    ``latent (B, P + T, row)``; ``window`` 0: every earlier token. Returns ``(B, T, heads · vdp)``."""
    return _impl(q).latent_attend(q, kv, latent, seq, P, shape, window, scale)


def latent_decode(q_abs, q, ring, seq, shape: LatentShape, scale: float) -> torch.Tensor:
    """One token per sequence over its ring, in latent space: ``q_abs (heads, B, kvp)`` → ``(heads, B, kvp)``."""
    return _impl(q).latent_decode(q_abs, q, ring, seq, shape, scale)


# ---- routed experts
ACTIVATIONS = {"none": 0, "relu_squared": 1}


def routed_experts(h, logits, up, down, top: int, activation: str, renormalize: bool, n_up: int, n_down: int):
    """Softmax over all experts' ``logits (n, E)``, the ``top`` largest per token, ``down_e · act(up_e · h)`` of each.
    Returns ``(out, row (n, top), weight (n, top))``; choice ``k`` of token ``n`` is ``weight[n, k] · out[row[n, k]]``."""
    return _impl(h).moe_forward(h, logits, up, down, top, ACTIVATIONS[activation], renormalize, n_up, n_down)
