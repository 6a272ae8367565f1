"""Ops of models that are described layer by layer (fp32 residual stream, latent and grouped attention, state-space
recurrence, retention, gated linear attention, gated recurrence per channel, routed experts).

A CUDA tensor is always served by the kernels of ``libkvb200_layers.so`` (bf16 or fp32; anything else
raises), a CPU tensor by the PyTorch restatement in :mod:`keys_values_b200.ops.layers_reference`.

``seq`` is the :class:`keys_values_b200.kvcache.sequences.SequencePass` of the pass: slots, start positions and
token counts of its rows.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import NamedTuple, Optional

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


@dataclass(frozen=True)
class GroupedShape:
    """Sizes and constants of one grouped-query attention; padded sizes are multiples of 8. The joint projection has the
    columns ``[queries: heads · maps · dimp | keys: kv_heads · maps · dimp | values: kv_heads · vdp (not with shared_value) |
    gate: heads · vdp, or heads (gate_per_head)]``, every head padded with zeros, the whole to a multiple of 8.

    ``maps = 2``: differential attention, every head has two queries and two keys over the same values; the result is
    ``norm(map 1 − lam · map 2) · post``, the norm an RMS norm of the head without a weight.
    Position i sees j <= i, and only ``i − j < window`` or ``j < keep`` (``window > 0``), or its own part of ``chunk`` positions
    (``chunk > 0``). ``pool > 0``: it also sees, as one key and one value each, the means of all blocks of ``pool`` positions that end
    before its window. ``softcap > 0``: scores become softcap · tanh(score / softcap). One map: the result is multiplied by ``post``.

    ``borrowed``: the keys and values are those of another layer; the projection has columns for queries and gate only."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    shared_value: bool
    gate: bool
    sink: bool
    scale: float
    maps: int = 1
    head_norm: bool = False
    gate_per_head: bool = False
    softcap: float = 0.0
    window: int = 0
    keep: int = 0
    chunk: int = 0
    lam: float = 0.0
    post: float = 1.0
    eps: float = 0.0
    pool: int = 0
    borrowed: bool = False

    @property
    def dimp(self) -> int:
        return round8(self.dim)

    @property
    def vdp(self) -> int:
        return round8(self.vdim)

    @property
    def row(self) -> int:
        """Width of a cache row: the keys of all maps and the value of one key/value head."""
        return self.maps * self.dimp + self.vdp

    @property
    def value_col(self) -> int:
        """First value column of the joint projection."""
        return (self.heads + (0 if self.shared_value or self.borrowed else self.kv_heads)) * self.maps * self.dimp

    @property
    def gate_col(self) -> int:
        return self.value_col if self.borrowed else (self.heads + self.kv_heads) * self.maps * self.dimp + (0 if self.shared_value else self.kv_heads * self.vdp)

    @property
    def gate_cols(self) -> int:
        """Gate columns per head."""
        return 0 if not self.gate else 1 if self.gate_per_head else self.vdp

    @property
    def ld(self) -> int:
        """Columns of the joint projection."""
        return round8(self.gate_col + self.heads * self.gate_cols)

    @property
    def span(self) -> int:
        """Positions a query looks back at most, itself included, kept ones and means of blocks aside (but a block's positions stay until its
        mean is taken); 0: all."""
        return max(self.chunk or self.window, self.pool)

    @property
    def inner(self) -> int:
        """Columns of the result."""
        return self.heads * self.vdp


class RowPlan(NamedTuple):
    """Where the positions of a sequence lie: ``ring = 0`` position p in row p; else the first ``head`` positions have rows of
    their own and position p >= head has row ``head + (p − head) mod ring``; with pooled blocks the first ``head`` rows are those of the
    blocks, and position p has row ``head + p mod ring``. Both are multiples of 128."""

    head: int = 0
    ring: int = 0


@dataclass(frozen=True)
class RetentionShape:
    """Sizes of one retention mixer; padded sizes are multiples of 8. The projection has the columns ``[queries: heads · np |
    keys: heads · np | values: heads · vdp | gate: heads · vdp]``, every head padded with zeros."""

    heads: int
    dim: int
    vdim: int
    rot_dims: int

    @property
    def np(self) -> int:
        return round8(self.dim)

    @property
    def vdp(self) -> int:
        return round8(self.vdim)

    @property
    def qk(self) -> int:
        """Columns of queries and keys."""
        return 2 * self.heads * self.np

    @property
    def inner(self) -> int:
        return self.heads * self.vdp

    @property
    def key_scale(self) -> float:
        return self.dim**-0.5


@dataclass(frozen=True)
class GatedLinearShape:
    """Sizes of one gated linear attention; padded sizes are multiples of 8. The projection has the columns ``[queries: heads · np |
    keys: heads · np | low-rank input of the decays: rp | values: heads · vdp | gate: heads · vdp]``, every head padded with zeros."""

    heads: int
    dim: int
    vdim: int
    rank: int
    tau: float

    @property
    def np(self) -> int:
        return round8(self.dim)

    @property
    def vdp(self) -> int:
        return round8(self.vdim)

    @property
    def rp(self) -> int:
        return round8(self.rank)

    @property
    def qk(self) -> int:
        """Columns of queries and keys."""
        return 2 * self.heads * self.np

    @property
    def keys(self) -> int:
        """Key channels of all heads, each with a decay of its own."""
        return self.heads * self.np

    @property
    def inner(self) -> int:
        return self.heads * self.vdp

    @property
    def query_scale(self) -> float:
        return self.dim**-0.5


class DecayWeights(NamedTuple):
    """Second half of the decays' projection: ``weight (rank, keys)`` and ``bias (keys,)``, fp32."""

    weight: torch.Tensor
    bias: torch.Tensor


@dataclass(frozen=True)
class RecurrenceShape:
    """Sizes of one gated recurrence per channel. ``blocks`` equal parts of the channels, each padded to a multiple of 8, with gates that are
    square products within a part. The projection has the columns ``[y: channels | x: channels]``."""

    width: int
    blocks: int
    taps: int

    @property
    def part(self) -> int:
        return self.width // self.blocks

    @property
    def pp(self) -> int:
        return round8(self.part)

    @property
    def channels(self) -> int:
        """Padded width."""
        return self.blocks * self.pp

    @property
    def inner(self) -> int:
        return self.channels


class RecurrenceWeights(NamedTuple):
    """``conv (taps, channels)``, ``conv_bias``, ``bias_r``, ``bias_i`` and ``rate`` (log2 of the decay at an open gate) ``(channels,)``, all fp32;
    ``gates (blocks, pp, 2 · pp)`` in the model's type: columns of the decay gates, then of the input gates of a part."""

    conv: torch.Tensor
    conv_bias: torch.Tensor
    gates: torch.Tensor
    bias_r: torch.Tensor
    bias_i: torch.Tensor
    rate: torch.Tensor


class EdgeTokens(NamedTuple):
    """What an edge between sublayers needs to know of its tokens: the pass; ``table`` (a vector per position is added to the stream); ``conv
    (taps, width)`` fp32 and its ``ring (slots, taps, width)`` (what the sublayer reads, h, passes a causal convolution, whose last row meets the
    token itself; the ring keeps the last h of every sequence, position p in row p mod taps)."""

    seq: object
    table: Optional[torch.Tensor] = None
    conv: Optional[torch.Tensor] = None
    ring: Optional[torch.Tensor] = None


@dataclass(frozen=True)
class RouterRule:
    """How a router scores and chooses: ``score`` ``"softmax"`` or ``"sigmoid"``; ``groups`` of neighbouring experts, of which the
    ``keep`` best (by the sum of their two largest choice scores) stay in the choice; ``renormalize``: the chosen scores are divided by
    their sum + ``eps``."""

    score: str = "softmax"
    groups: int = 1
    keep: int = 1
    renormalize: bool = False
    eps: float = 0.0


@dataclass(frozen=True)
class StateShape:
    """Sizes of one state-space mixer; padded sizes are multiples of 8. The joint projection has the columns
    ``[z: heads · vdp | x: heads · vdp | B: groups · np | C: groups · np | dt: heads]``, every head and group padded with
    zeros; x, B and C are the channels of the convolution."""

    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int

    @property
    def vdp(self) -> int:
        return round8(self.vdim)

    @property
    def np(self) -> int:
        return round8(self.state)

    @property
    def inner(self) -> int:
        """Padded width of z, x and y."""
        return self.heads * self.vdp

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.np

    @property
    def dt_col(self) -> int:
        return self.inner + self.channels

    @property
    def ld(self) -> int:
        """Columns of the joint projection."""
        return round8(self.dt_col + self.heads)


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


def norm_edge(x_in, sub, after, x_out, before, h, idx, embed, step, eps: float, center: bool, experts=None, tokens: Optional[EdgeTokens] = None) -> None:
    """``x = x_in + norm(s) · after`` with ``s = sub + Σ_k weight_k · expert output_k`` (``x_in``, ``sub`` or ``experts`` ``None``:
    without it; ``after`` ``None``: ``s`` as it is), then ``x += embed[idx] + step`` (each unless ``None``); ``x_out = x`` (fp32, may be
    ``x_in``) and, unless ``h`` is ``None``, ``h = norm(x) · before`` (``before`` ``None``: ``h = x``). The norm takes the mean off if
    ``center``. ``experts``: ``(out, row, weight)`` of :func:`routed_experts`. ``tokens``: see :class:`EdgeTokens`; a single
    token passes the convolution in the same kernel."""
    impl = _impl(x_out)
    if tokens is None or tokens.conv is None or tokens.seq.length == 1:
        impl.norm_edge(x_in, sub, after, x_out, before, h, idx, embed, step, eps, center, experts, tokens)
        return
    plain = torch.empty_like(h)
    impl.norm_edge(x_in, sub, after, x_out, before, plain, idx, embed, step, eps, center, experts, tokens._replace(conv=None, ring=None))
    impl.short_conv(plain, 0, tokens.conv, None, tokens.ring, tokens.seq, False, h)


def row_norm(x: torch.Tensor, weight: torch.Tensor, eps: float, center: bool, dtype: torch.dtype) -> torch.Tensor:
    """Norm of the rows of ``x (n, width)`` fp32, times ``weight (width,)`` fp32."""
    return _impl(x).row_norm(x, weight, eps, center, dtype)


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


# ---- grouped-query attention
def grouped_prep(qkv, norm_q, norm_k, freq, rows, seq, shape: GroupedShape, eps: float, plan: RowPlan = RowPlan(), q_scale=None) -> torch.Tensor:
    """Norm (unless ``norm_q`` is ``None``) and rotation of queries and keys of the joint projection ``qkv (B, T, ·)``. The norm goes over
    a whole projection or (``head_norm``) over every head and map with weights of one head; ``q_scale (heads,)`` multiplies queries. Returns
    queries ``(B, T, heads · maps, dimp)``; ``[keys of the maps | value]`` of every real token goes to its place in ``rows (slots, length,
    kv_heads, row)`` (unless they are ``borrowed``), and the means of blocks that the pass completes to theirs."""
    return _impl(qkv).grouped_prep(qkv, norm_q, norm_k, freq, rows, seq, shape, eps, plan, q_scale)


def grouped_attend(q, qkv, rows, seq, shape: GroupedShape, sink=None, plan: RowPlan = RowPlan(), out=None) -> torch.Tensor:
    """Causal attention of ``q (B, T, heads · maps, dimp)`` over ``rows``, which hold the pass already; with the gate of ``qkv``
    applied. ``sink (heads,)`` fp32: logarithms of what shapes with a sink add to the denominators (``None``: zeros). Returns
    ``(B, T, heads · vdp)``, in ``out`` if that is given (rows of any leading dimension)."""
    return _impl(q).grouped_attend(q, qkv, rows, seq, shape, sink, plan, out)


# ---- retention
def retention_prep(qk, freq, seq, shape: RetentionShape, dtype: torch.dtype) -> torch.Tensor:
    """``qk (B, T, shape.qk)`` fp32, queries and keys as projected → the same rotated, keys times dim^(−1/2), as ``dtype``."""
    return _impl(qk).retention_prep(qk, freq, seq, shape, dtype)


def retention_scan(qk, v, decay, log2_decay, state, seq, shape: RetentionShape) -> torch.Tensor:
    """``S_t = decay S_(t−1) + k_t v_t^T``, ``o_t = S_t^T q_t`` per head over the tokens of a pass, from and to ``state (slots, heads, np,
    vdp)`` fp32. ``v``: rows of any leading dimension whose first ``inner`` columns are the values. Returns ``(B, T, inner)``."""
    return _impl(qk).retention_scan(qk, v, decay, log2_decay, state, seq, shape)


def head_norm_gate(y, gate, shape, eps: float, weight=None) -> torch.Tensor:
    """``y (B, T, inner)`` divided by every head's root mean square, times ``weight (vdp,)`` (``None``: without), times silu of ``gate`` (rows of
    any leading dimension)."""
    return _impl(y).head_norm_gate(y, gate, shape, eps, weight)


def retention_step(u, freq, decay, state, seq, shape: RetentionShape, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """The three above for one token per sequence, from the fp32 projections ``u (B, 1, qk + 2 inner)``; all of it in fp32."""
    return _impl(u).retention_step(u, freq, decay, state, seq, shape, eps, dtype)


# ---- gated linear attention
def gated_linear_scan(qka, v, decay: DecayWeights, state, seq, shape: GatedLinearShape) -> torch.Tensor:
    """``S_t = diag(alpha_t) S_(t−1) + k_t v_t^T``, ``o_t = S_t^T q_t · query_scale`` per head over the tokens of a pass, from and to ``state
    (slots, heads, np, vdp)`` fp32. ``qka (B, T, qk + rp)`` fp32: queries, keys and input a of the decays ``alpha = sigmoid(weight^T a +
    bias)^(1 / tau)``; ``v``: rows of any leading dimension whose first ``inner`` columns are the values. Returns ``(B, T, inner)``."""
    return _impl(qka).gated_linear_scan(qka, v, decay, state, seq, shape)


def gated_linear_step(u, decay: DecayWeights, weight, state, seq, shape: GatedLinearShape, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """The scan, norm (times ``weight (vdp,)``) and gate for one token per sequence, from the fp32 projections ``u (B, 1, qk + rp + 2 inner)``; all
    of it in fp32."""
    return _impl(u).gated_linear_step(u, decay, weight, state, seq, shape, eps, dtype)


# ---- gated recurrence per channel
def gated_recurrence(u, w: RecurrenceWeights, ring, state, seq, shape: RecurrenceShape, scale: float, out) -> torch.Tensor:
    """``u (B, T, 2 · channels)``: y and x. x passes a causal convolution (its inputs before the pass come from ``ring``), gives gates r and i, and
    ``S_t = a S_(t−1) + sqrt(1 − a²) i x`` with ``log2 a = rate · r``, from and to ``state (slots, channels)`` fp32. Returns ``out (B, T, channels)``
    = S · gelu(y) · ``scale``, zero in padding. u and out: rows of any leading dimension."""
    return _impl(u).gated_recurrence(u, w, ring, state, seq, shape, scale, out)


# ---- state-space recurrence
def short_conv(u, col: int, w, bias, ring, seq, silu: bool = True, out=None) -> torch.Tensor:
    """Causal convolution ``w (taps, channels)`` with bias (unless ``None``) and silu (or without) over the channels of ``u (B, T, ·)`` from ``col`` on; the inputs before the
    pass come from ``ring (slots, taps, channels)``, which takes the last ones of the pass. Returns ``(B, T, channels)``."""
    return _impl(u).short_conv(u, col, w, bias, ring, seq, silu, out)


def state_scan(u, xbc, dt_bias, a_log, skip, state, seq, shape: StateShape) -> torch.Tensor:
    """The recurrence over the tokens of a pass, from and to ``state (slots, heads, np, vdp)`` fp32; step sizes from the last
    columns of ``u``. Returns ``y (B, T, inner)``, zero in padding."""
    return _impl(u).state_scan(u, xbc, dt_bias, a_log, skip, state, seq, shape)


def state_step(u, w, bias, dt_bias, a_log, skip, ring, state, seq, shape: StateShape) -> torch.Tensor:
    """:func:`short_conv` and :func:`state_scan` for one token per sequence, ``u (B, 1, ld)``."""
    return _impl(u).state_step(u, w, bias, dt_bias, a_log, skip, ring, state, seq, shape)


def gated_group_norm(y, u, weight, shape: StateShape, eps: float) -> torch.Tensor:
    """``y · silu(z)`` (z from ``u``), RMS-normed in ``norm_groups`` equal parts of the unpadded width, times ``weight``."""
    return _impl(y).gated_group_norm(y, u, weight, shape, eps)


def activate(x: torch.Tensor, activation: str) -> torch.Tensor:
    """Activation of a product's result, in place."""
    return x if activation == "none" else _impl(x).activate(x, ACTIVATIONS[activation])


def glu(x: torch.Tensor, ff: int, limit: Optional[float] = None) -> torch.Tensor:
    """``x (n, 2 · round8(ff))`` = ``[gate | up]`` → ``silu(gate) · up (n, round8(ff))``, zero in the padding. With a ``limit``: the clamped unit
    ``g · sigmoid(1.702 g) · (u + 1)`` with ``g = min(gate, limit)`` and u = up clamped to ±limit."""
    return _impl(x).glu(x, ff, limit)


# ---- routed experts. silu_gated: the rows of gate and up projection in turns, act(up h) = silu(gate h) · (up h)
ACTIVATIONS = {"none": 0, "relu_squared": 1, "silu_gated": 2}


def routed_experts(h, logits, up, down, top: int, activation: str, rule: RouterRule, n_up: int, n_down: int, correction=None):
    """Scores of all experts from ``logits (n, E)``, the ``top`` of every token by score + ``correction (E,)``, ``down_e · act(up_e · h)`` of
    each; ``n_up`` results of the activation, ``n_down`` outputs. Returns ``(out, row (n, top), weight (n, top))``; choice ``k`` of token
    ``n`` is ``weight[n, k] · out[row[n, k]]``."""
    return _impl(h).moe_forward(h, logits, up, down, top, ACTIVATIONS[activation], rule, n_up, n_down, correction)
