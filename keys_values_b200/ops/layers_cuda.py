"""ctypes bindings to ``libkvb200_layers.so``: kernels of models that are described layer by layer.

Same conventions as :mod:`keys_values_b200.ops.cuda` (outputs allocated with torch, raw pointers plus the
current stream, status code checked); launches are counted and device-side errors reported through
the same status word.
"""
from __future__ import annotations

import ctypes
import functools
from typing import Optional

import torch

from keys_values_b200.ops import cuda as _base
from keys_values_b200.ops.cuda import NativeError, _check, _count, _ll, _p, _stream, status_word

_LIB = None
LIB_PATH = _base._ROOT / "libkvb200_layers.so"
_CODE = {torch.float32: 0, torch.bfloat16: 1}
# True: the CUDA-core kernels serve bf16 too (comparisons in tests and benchmarks)
FORCE_SIMPLE = False


class _Attention(ctypes.Structure):
    """``kvb_attention`` of ``kvb200_layers.h``."""

    _fields_ = [(n, ctypes.c_int) for n in ("heads", "kv_heads", "maps", "dim", "dimp", "vdim", "vdp", "rot_dims", "value_col", "head_norm",
                                            "window", "keep", "chunk", "head", "ring", "sink", "gate_cols")]
    _fields_ += [(n, ctypes.c_float) for n in ("scale", "softcap", "lam", "post", "eps")]
    _fields_ += [("pool", ctypes.c_int), ("borrowed", ctypes.c_int), ("out_ld", ctypes.c_longlong), ("sink_w", ctypes.c_void_p), ("q_scale", ctypes.c_void_p)]


class _Router(ctypes.Structure):
    """``kvb_router`` of ``kvb200_layers.h``."""

    _fields_ = [(n, ctypes.c_int) for n in ("score", "groups", "keep", "renormalize")] + [("eps", ctypes.c_float), ("correction", ctypes.c_void_p)]


class _EdgeTokens(ctypes.Structure):
    """``kvb_edge_tokens`` of ``kvb200_layers.h``."""

    _fields_ = [(n, ctypes.c_void_p) for n in ("slots", "start", "count")] + [("T", ctypes.c_int), ("taps", ctypes.c_int), ("table", ctypes.c_void_p),
                ("table_rows", ctypes.c_longlong), ("conv_w", ctypes.c_void_p), ("conv_ring", ctypes.c_void_p)]


class _GatedLinear(ctypes.Structure):
    """``kvb_gated_linear`` of ``kvb200_layers.h``."""

    _fields_ = [(n, ctypes.c_void_p) for n in ("input", "w", "bias")] + [("ld", ctypes.c_longlong)]
    _fields_ += [(n, ctypes.c_int) for n in ("heads", "np", "rank")] + [("inv_tau", ctypes.c_float), ("q_scale", ctypes.c_float)]


class _GatedRecurrence(ctypes.Structure):
    """``kvb_gated_recurrence`` of ``kvb200_layers.h``."""

    _fields_ = [(n, ctypes.c_void_p) for n in ("conv", "conv_bias", "bias_r", "bias_i", "rate", "gates")]
    _fields_ += [(n, ctypes.c_int) for n in ("blocks", "pp", "taps")] + [("scale", ctypes.c_float)]


def _ptr(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


@functools.lru_cache(maxsize=512)
def _attention(s, plan, eps: float, sink: Optional[int] = None, q_scale: Optional[int] = None, out_ld: int = 0) -> _Attention:
    return _Attention(s.heads, s.kv_heads, s.maps, s.dim, s.dimp, s.vdim, s.vdp, s.rot_dims, s.value_col, int(s.head_norm), s.window, s.keep,
                      s.chunk, plan.head, plan.ring, int(s.sink), s.gate_cols, s.scale, s.softcap, s.lam, s.post, eps,
                      s.pool, int(s.borrowed), out_ld or s.inner, sink, q_scale)


def lib():
    global _LIB
    if _LIB is None:
        if not LIB_PATH.exists():
            raise NativeError(f"{LIB_PATH} is missing: run `python -m keys_values_b200.build_ext`")
        _LIB = ctypes.CDLL(str(LIB_PATH))
        _LIB.kvb_grouped_decode_scratch_bytes.restype = ctypes.c_longlong
        _LIB.kvb_state_scan_tc_scratch_bytes.restype = ctypes.c_longlong
        _LIB.kvb_latent_decode_scratch_bytes.restype = ctypes.c_longlong
        _LIB.kvb_gated_linear_scan_tc_scratch_bytes.restype = ctypes.c_longlong
    return _LIB


def code(dtype: torch.dtype) -> int:
    try:
        return _CODE[dtype]
    except KeyError:
        raise NativeError(f"dtype {dtype}: these kernels exist for bfloat16 and float32")


def _f(x: float) -> ctypes.c_float:
    return ctypes.c_float(float(x))


def _contiguous(*tensors) -> None:
    for t in tensors:
        if t is not None and not t.is_contiguous():
            raise NativeError("layer kernels take contiguous tensors")


# ---------------------------------------------------------------------------------------------- layer edges
def embed_edge(idx, prev_token, embed, bigram, buckets, mul_prev, mul_cur, hist, gain, shift, state, h, hs, seq, eps) -> None:
    B, T = idx.shape
    _contiguous(idx, embed, bigram, hist, gain, shift, state, h, hs)
    _check(lib().kvb_embed_edge(_p(idx), _p(prev_token), _p(embed), _p(bigram), _ll(buckets), _ll(mul_prev), _ll(mul_cur), _p(hist),
                                _p(gain), _p(shift), _p(state), _p(h), _p(hs), _p(seq.slots), _p(seq.start), _p(seq.count), B, T,
                                embed.shape[1], _ll(embed.shape[0]), _f(eps), code(embed.dtype), _p(status_word(idx.device)),
                                _stream(idx)), "embed_edge")
    _count()


def layer_edge(x_in, mix, expert_out, expert_row, expert_w, hist, n_hist, coef, x_out, gain, shift, state, h, hs, seq, eps) -> None:
    B, T, width = x_in.shape
    _contiguous(x_in, mix, expert_out, expert_row, expert_w, coef, x_out, gain, shift, state, h, hs)
    top = 0 if expert_w is None else expert_w.shape[1]
    ld = 0 if expert_out is None else expert_out.shape[1]
    _check(lib().kvb_layer_edge(_p(x_in), _p(mix), _p(expert_out), _p(expert_row), _p(expert_w), top, _ll(ld), _p(hist), n_hist,
                                _ll(0 if hist is None else hist.stride(0)), _p(coef), _p(x_out), _p(gain), _p(shift), _p(state), _p(h),
                                _p(hs), _p(seq.slots), _p(seq.start), _p(seq.count), B, T, width, _f(eps), code(mix.dtype),
                                _stream(x_in)), "layer_edge")
    _count()


def scalar_rmsnorm(x, rows, gain, eps, dtype) -> torch.Tensor:
    n = x.shape[0] if rows is None else rows.numel()
    y = torch.empty((n, x.shape[1]), dtype=dtype, device=x.device)
    _contiguous(x, rows, gain)
    _check(lib().kvb_scalar_rmsnorm(_p(x), _p(rows), _p(gain), _p(y), _ll(n), x.shape[1], _f(eps), code(dtype), _stream(x)), "scalar_rmsnorm")
    _count()
    return y


def sequence_advance(idx, pos, prev_token, seq) -> None:
    B, T = idx.shape
    _contiguous(idx)
    _check(lib().kvb_sequence_advance(_p(idx), _p(pos), _p(prev_token), _p(seq.slots), _p(seq.count), B, T, _stream(idx)), "sequence_advance")
    _count()


# ------------------------------------------------------------------------------------------- latent attention
def latent_prep(qkv, norm_w, freq, latent, ring, seq, P, shape, eps) -> torch.Tensor:
    """``qkv (B, T, ·)`` → padded queries ``(B, T, heads, dimp + rp)``; latent rows go to ``latent`` and into ``ring``."""
    B, T, ld = qkv.shape
    s = shape
    q = torch.empty((B, T, s.heads, s.dimp + s.rp), dtype=qkv.dtype, device=qkv.device)
    _contiguous(qkv, norm_w, freq, latent, ring)
    _check(lib().kvb_latent_prep(_p(qkv), _ll(ld), _p(norm_w), _p(freq), _p(q), _p(latent), _p(ring), _p(seq.slots), _p(seq.start),
                                 _p(seq.count), B, T, P, 0 if ring is None else ring.shape[1], s.heads, s.dim, s.dimp, s.rot, s.rot_dims,
                                 s.rp, s.kv_rank, s.kvp, _f(eps), code(qkv.dtype), _stream(qkv)), "latent_prep")
    _count()
    return q


def ring_gather(ring, latent, seq, P) -> None:
    B, n, lw = latent.shape
    _check(lib().kvb_ring_gather(_p(ring), _p(latent), _p(seq.slots), _p(seq.start), B, n - P, P, ring.shape[1], lw, code(ring.dtype),
                                 _stream(ring)), "ring_gather")
    _count()


def latent_attend(q, kv, latent, seq, P, shape, window, scale) -> torch.Tensor:
    B, T = q.shape[:2]
    s = shape
    out = torch.empty((B, T, s.heads * s.vdp), dtype=q.dtype, device=q.device)
    _contiguous(q, kv, latent)
    args = (B, T, P, s.heads, s.dimp, s.rp, s.kvp, s.vdp, int(window), _f(scale))
    if q.dtype == torch.bfloat16 and not FORCE_SIMPLE and lib().kvb_latent_attend_tc_supported(s.dimp, s.rp, s.vdp):
        _check(lib().kvb_latent_attend_tc(_p(q), _p(kv), _p(latent), _p(out), _p(seq.start), *args, _p(status_word(q.device)), _stream(q)),
               "latent_attend_tc")
    else:
        _check(lib().kvb_latent_attend(_p(q), _p(kv), _p(latent), _p(out), _p(seq.start), *args, code(q.dtype), _stream(q)), "latent_attend")
    _count()
    return out


def latent_decode(q_abs, q, ring, seq, shape, scale) -> torch.Tensor:
    """``q_abs (heads, B, kvp)``, ``q (B, 1, heads, dimp + rp)`` → weighted latents ``(heads, B, kvp)``."""
    s = shape
    H, B, kvp = q_abs.shape
    C = ring.shape[1]
    out = torch.empty_like(q_abs)
    _contiguous(q_abs, q, ring)
    nbytes = int(lib().kvb_latent_decode_scratch_bytes(B, H, kvp, s.rp, C))
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device)
    _check(lib().kvb_latent_decode(_p(q_abs), _p(q), _p(ring), _p(out), _p(scratch), _p(seq.slots), _p(seq.start), B,
                                   ring.shape[0], H, s.dimp, s.rp, kvp, C, _f(scale), code(q.dtype), int(FORCE_SIMPLE), _p(status_word(q.device)), _stream(q)), "latent_decode")
    _count()
    return out


# ------------------------------------------------------------------------------------------ sequential layers
def _edge_tokens(tokens):
    if tokens is None:
        return None
    seq, table, conv, ring = tokens
    _contiguous(table, conv, ring)
    return ctypes.byref(_EdgeTokens(seq.slots.data_ptr(), seq.start.data_ptr(), seq.count.data_ptr(), seq.length, 0 if conv is None else conv.shape[0],
                                    _ptr(table), 0 if table is None else table.shape[0], _ptr(conv), _ptr(ring)))


def norm_edge(x_in, sub, after, x_out, before, h, idx, embed, step, eps, center, experts=None, tokens=None) -> None:
    width = x_out.shape[-1]
    out, row, weight = experts if experts is not None else (None, None, None)
    _contiguous(x_in, sub, after, x_out, before, h, idx, embed, step, out, row, weight)
    dtype = next((t.dtype for t in (sub, out, h, embed) if t is not None), torch.float32)
    _check(lib().kvb_norm_edge(_p(x_in), _p(sub), _p(out), _p(row), _p(weight), 0 if weight is None else weight.shape[1],
                               _ll(0 if out is None else out.shape[1]), _p(after), _p(x_out), _p(before), _p(h), _p(idx), _p(embed),
                               _ll(0 if embed is None else embed.shape[0]), _p(step), _ll(x_out.numel() // width), width, _f(eps), int(center),
                               code(dtype), _edge_tokens(tokens), _p(status_word(x_out.device)), _stream(x_out)), "norm_edge")
    _count()


def row_norm(x, weight, eps, center, dtype) -> torch.Tensor:
    n, width = x.shape
    y = torch.empty((n, width), dtype=dtype, device=x.device)
    _contiguous(x, weight)
    _check(lib().kvb_norm_edge(_p(x), None, None, None, None, 0, _ll(0), None, None, _p(weight), _p(y), None, None, _ll(0), None, _ll(n), width, _f(eps), int(center),
                               code(dtype), None, _p(status_word(x.device)), _stream(x)), "row_norm")
    _count()
    return y


def activate(x, act: int) -> torch.Tensor:
    _contiguous(x)
    _check(lib().kvb_activate(_p(x), _ll(x.numel()), act, code(x.dtype), _stream(x)), "activate")
    _count()
    return x


# ------------------------------------------------------------------------------------------ grouped attention
def grouped_prep(qkv, norm_q, norm_k, freq, rows, seq, s, eps, plan, q_scale=None) -> torch.Tensor:
    B, T, _ = qkv.shape
    ld = _rows_of(qkv)
    q = torch.empty((B, T, s.heads * s.maps, s.dimp), dtype=qkv.dtype, device=qkv.device)
    _contiguous(norm_q, norm_k, freq, rows, q_scale)
    a = _attention(s, plan, eps, None, _ptr(q_scale))
    _check(lib().kvb_grouped_prep(_p(qkv), _ll(ld), _p(norm_q), _p(norm_k), _p(freq), _p(q), _p(rows), _p(seq.slots), _p(seq.start),
                                  _p(seq.count), B, T, rows.shape[1], ctypes.byref(a), code(qkv.dtype), _stream(qkv)), "grouped_prep")
    _count(2 if s.pool and T > 1 else 1)
    return q


def grouped_attend(q, qkv, rows, seq, s, sink, plan, out=None) -> torch.Tensor:
    B, T = q.shape[:2]
    if out is None:
        out = torch.empty((B, T, s.inner), dtype=q.dtype, device=q.device)
    _contiguous(q, rows, sink)
    gate = qkv.data_ptr() + s.gate_col * qkv.element_size() if s.gate else None
    gate_args = (ctypes.c_void_p(gate), _ll(_rows_of(qkv) if s.gate else 0))
    where = (_p(seq.slots), _p(seq.start))
    length = rows.shape[1]
    a = ctypes.byref(_attention(s, plan, s.eps, _ptr(sink), None, _rows_of(out)))
    fast = q.dtype == torch.bfloat16 and not FORCE_SIMPLE
    if fast and T == 1 and lib().kvb_grouped_decode_supported(a):
        nbytes = int(lib().kvb_grouped_decode_scratch_bytes(B, length, a))
        scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device) if nbytes else None
        _check(lib().kvb_grouped_decode(_p(q), _p(rows), *gate_args, _p(out), _p(scratch), *where, B, rows.shape[0], length, a,
                                        _p(status_word(q.device)), _stream(q)), "grouped_decode")
        _count(2 if nbytes else 1)
        return out
    if fast and T > 1 and lib().kvb_grouped_attend_tc_supported(a):
        _check(lib().kvb_grouped_attend_tc(_p(q), _p(rows), *gate_args, _p(out), *where, B, T, rows.shape[0], length, a,
                                           _p(status_word(q.device)), _stream(q)), "grouped_attend_tc")
    else:
        _check(lib().kvb_grouped_attend(_p(q), _p(rows), *gate_args, _p(out), *where, B, T, length, a, code(q.dtype), _stream(q)), "grouped_attend")
    _count()
    return out


# --------------------------------------------------------------------------------------------------- retention
def _rows_of(t: torch.Tensor) -> int:
    """Leading dimension of a view of equal columns of contiguous rows ``(B, T, ·)``."""
    B, T, _ = t.shape
    if t.stride(2) != 1 or (B > 1 and t.stride(0) != T * t.stride(1)):
        raise NativeError("rows must lie one behind the other")
    return t.stride(1)


def retention_prep(qk, freq, seq, s, dtype) -> torch.Tensor:
    B, T, _ = qk.shape
    out = torch.empty((B, T, s.qk), dtype=dtype, device=qk.device)
    _check(lib().kvb_retention_prep(_p(qk), _ll(_rows_of(qk)), _p(freq), _p(out), _p(seq.start), B, T, s.heads, s.np, s.rot_dims, _f(s.key_scale),
                                    code(dtype), _stream(qk)), "retention_prep")
    _count()
    return out


def retention_scan(qk, v, decay, log2_decay, state, seq, s) -> torch.Tensor:
    B, T, ldqk = qk.shape
    y = torch.empty((B, T, s.inner), dtype=qk.dtype, device=qk.device)
    _contiguous(qk, state)
    where = (_p(seq.slots), _p(seq.start), _p(seq.count), B, T, s.heads, s.vdp, s.np)
    if qk.dtype == torch.bfloat16 and not FORCE_SIMPLE and lib().kvb_state_scan_tc_supported(s.heads, s.heads, s.vdp, s.np):
        nbytes = int(lib().kvb_state_scan_tc_scratch_bytes(B, T, s.heads, s.heads, s.vdp, s.np))
        scratch = torch.empty(nbytes, dtype=torch.uint8, device=qk.device) if nbytes else None
        _check(lib().kvb_retention_scan_tc(_p(v), _ll(_rows_of(v)), _p(qk), _ll(ldqk), _p(log2_decay), _p(state), _p(y), _p(scratch), *where,
                                           _p(status_word(qk.device)), _stream(qk)), "retention_scan_tc")
        _count(3 if nbytes else 1)
        return y
    _check(lib().kvb_retention_scan(_p(v), _ll(_rows_of(v)), _p(qk), _ll(ldqk), _p(decay), _p(state), _p(y), *where, code(qk.dtype), _stream(qk)),
           "retention_scan")
    _count()
    return y


def head_norm_gate(y, gate, s, eps, weight=None) -> torch.Tensor:
    out = torch.empty_like(y)
    _contiguous(y, weight)
    _check(lib().kvb_head_norm_gate(_p(y), _p(gate), _ll(_rows_of(gate)), _p(weight), _p(out), _ll(y.numel() // s.inner), s.heads, s.vdim, s.vdp, _f(eps),
                                    code(y.dtype), _stream(y)), "head_norm_gate")
    _count()
    return out


def retention_step(u, freq, decay, state, seq, s, eps, dtype) -> torch.Tensor:
    B, _, ld = u.shape
    out = torch.empty((B, 1, s.inner), dtype=dtype, device=u.device)
    _contiguous(u, state)
    _check(lib().kvb_retention_step(_p(u), _ll(ld), _p(freq), _p(decay), _p(state), _p(out), _p(seq.slots), _p(seq.start), _p(seq.count), B,
                                    s.heads, s.vdim, s.vdp, s.np, s.rot_dims, _f(s.key_scale), _f(eps), code(dtype), _stream(u)), "retention_step")
    _count()
    return out


# --------------------------------------------------------------------------------------- gated linear attention
# rank of the decays' projection that the kernel in front of the chunked scan has room for
GATED_LINEAR_MAX_RANK = 256


def _gated_linear(u, decay, s) -> _GatedLinear:
    _contiguous(u, *decay)
    return _GatedLinear(u.data_ptr(), decay.weight.data_ptr(), decay.bias.data_ptr(), u.shape[-1], s.heads, s.np, s.rank, 1.0 / s.tau, s.query_scale)


def gated_linear_scan(qka, v, decay, state, seq, s) -> torch.Tensor:
    B, T, _ = qka.shape
    y = torch.empty((B, T, s.inner), dtype=v.dtype, device=v.device)
    _contiguous(state)
    g = _gated_linear(qka, decay, s)
    where, stream = (_p(seq.slots), _p(seq.start), _p(seq.count), B, T), _stream(qka)
    far = None
    if v.dtype == torch.bfloat16 and not FORCE_SIMPLE and s.rank <= GATED_LINEAR_MAX_RANK and lib().kvb_state_scan_tc_supported(s.heads, s.heads, s.vdp, s.np):
        chunks = (T + 127) // 128
        qk = torch.empty((B, T, s.qk), dtype=v.dtype, device=v.device)
        factor = torch.empty((B, chunks, s.keys, 2), dtype=torch.float32, device=v.device)
        far = torch.empty((B, s.heads), dtype=torch.int32, device=v.device)
        _check(lib().kvb_gated_linear_prep(ctypes.byref(g), _p(qk), _p(factor), _p(far), _p(seq.count), B, T, stream), "gated_linear_prep")
        nbytes = int(lib().kvb_gated_linear_scan_tc_scratch_bytes(B, T, s.heads, s.vdp, s.np))
        scratch = torch.empty(nbytes, dtype=torch.uint8, device=v.device) if nbytes else None
        _check(lib().kvb_gated_linear_scan_tc(_p(v), _ll(_rows_of(v)), _p(qk), _p(factor), _p(far), _p(state), _p(y), _p(scratch), *where, s.heads,
                                              s.vdp, s.np, _p(status_word(v.device)), stream), "gated_linear_scan_tc")
        _count(4 if nbytes else 2)
    # after the chunked kernel: the heads whose decays are beyond its range, usually none
    _check(lib().kvb_gated_linear_scan(ctypes.byref(g), _p(v), _ll(_rows_of(v)), _p(state), _p(y), _p(far), *where, s.vdp, code(v.dtype), stream),
           "gated_linear_scan")
    _count()
    return y


def gated_linear_step(u, decay, weight, state, seq, s, eps, dtype) -> torch.Tensor:
    B = u.shape[0]
    out = torch.empty((B, 1, s.inner), dtype=dtype, device=u.device)
    _contiguous(weight, state)
    g = _gated_linear(u, decay, s)
    _check(lib().kvb_gated_linear_step(ctypes.byref(g), s.qk + s.rp, _p(weight), _p(state), _p(out), _p(seq.slots), _p(seq.start), _p(seq.count), B,
                                       s.vdim, s.vdp, _f(eps), code(dtype), _stream(u)), "gated_linear_step")
    _count()
    return out


# ------------------------------------------------------------------------------------ gated recurrence per channel
def gated_recurrence(u, w, ring, state, seq, s, scale, out) -> torch.Tensor:
    B, T, _ = u.shape
    _contiguous(*w, ring, state)
    g = ctypes.byref(_GatedRecurrence(*(t.data_ptr() for t in (w.conv, w.conv_bias, w.bias_r, w.bias_i, w.rate, w.gates)), s.blocks, s.pp, s.taps, scale))
    where = (_p(seq.slots), _p(seq.start), _p(seq.count), B)
    ld, ldo = _ll(_rows_of(u)), _ll(_rows_of(out))
    if T == 1:
        _check(lib().kvb_gated_recurrence_step(g, _p(u), ld, _p(ring), _p(state), _p(out), ldo, *where, code(u.dtype), _stream(u)), "gated_recurrence_step")
        _count()
        return out
    x = short_conv(u, s.channels, w.conv, w.conv_bias, ring, seq, False)
    z = bmm_fp32(x.view(B * T, s.blocks, s.pp).transpose(0, 1), w.gates)
    _check(lib().kvb_gated_recurrence_scan(g, _p(x), _p(z), _p(u), ld, _p(state), _p(out), ldo, *where, T, code(u.dtype), _p(status_word(u.device)),
                                           _stream(u)), "gated_recurrence_scan")
    _count()
    return out


def bmm_fp32(a, b) -> torch.Tensor:
    """Batched library product with an fp32 result."""
    return torch.bmm(a, b) if a.dtype == torch.float32 else torch.bmm(a, b, out_dtype=torch.float32)


# --------------------------------------------------------------------------------------- state-space recurrence
def short_conv(u, col, w, bias, ring, seq, silu=True, out=None) -> torch.Tensor:
    B, T, _ = u.shape
    taps, channels = w.shape
    if out is None:
        out = torch.empty((B, T, channels), dtype=u.dtype, device=u.device)
    _contiguous(w, bias, ring, out)
    if ring.dtype != u.dtype:
        raise NativeError(f"inputs of type {u.dtype} are kept as {ring.dtype}")
    _check(lib().kvb_short_conv(_p(u), _ll(_rows_of(u)), col, _p(w), _p(bias), _p(out), _p(ring), _p(seq.slots), _p(seq.start), _p(seq.count), B, T,
                                channels, taps, int(silu), code(u.dtype), _stream(u)), "short_conv")
    _count()
    return out


def state_scan(u, xbc, dt_bias, a_log, skip, state, seq, s) -> torch.Tensor:
    B, T, ld = u.shape
    y = torch.empty((B, T, s.inner), dtype=u.dtype, device=u.device)
    _contiguous(u, xbc, state)
    if u.dtype == torch.bfloat16 and not FORCE_SIMPLE and lib().kvb_state_scan_tc_supported(s.heads, s.groups, s.vdp, s.np):
        nbytes = int(lib().kvb_state_scan_tc_scratch_bytes(B, T, s.heads, s.groups, s.vdp, s.np))
        scratch = torch.empty(nbytes, dtype=torch.uint8, device=u.device) if nbytes else None
        _check(lib().kvb_state_scan_tc(_p(u), _ll(ld), s.dt_col, _p(xbc), _p(dt_bias), _p(a_log), _p(skip), _p(state), _p(y), _p(scratch),
                                       _p(seq.slots), _p(seq.start), _p(seq.count), B, T, s.heads, s.groups, s.vdp, s.np,
                                       _p(status_word(u.device)), _stream(u)), "state_scan_tc")
        _count(3 if nbytes else 1)
        return y
    _check(lib().kvb_state_scan(_p(u), _ll(ld), s.dt_col, _p(xbc), _p(dt_bias), _p(a_log), _p(skip), _p(state), _p(y), _p(seq.slots),
                                _p(seq.start), _p(seq.count), B, T, s.heads, s.groups, s.vdp, s.np, code(u.dtype), _stream(u)), "state_scan")
    _count()
    return y


def state_step(u, w, bias, dt_bias, a_log, skip, ring, state, seq, s) -> torch.Tensor:
    B, _, ld = u.shape
    y = torch.empty((B, 1, s.inner), dtype=u.dtype, device=u.device)
    _contiguous(u, w, bias, ring, state)
    _check(lib().kvb_state_step(_p(u), _ll(ld), s.inner, s.dt_col, _p(w), _p(bias), _p(dt_bias), _p(a_log), _p(skip), _p(ring), _p(state),
                                _p(y), _p(seq.slots), _p(seq.start), _p(seq.count), B, s.heads, s.groups, s.vdp, s.np, s.taps,
                                code(u.dtype), _stream(u)), "state_step")
    _count()
    return y


def gated_group_norm(y, u, weight, s, eps) -> torch.Tensor:
    out = torch.empty_like(y)
    _contiguous(y, u, weight)
    _check(lib().kvb_gated_group_norm(_p(y), _p(u), _ll(u.shape[-1]), _p(weight), _p(out), _ll(y.numel() // s.inner), s.heads, s.vdim, s.vdp,
                                      s.norm_groups, _f(eps), code(y.dtype), _stream(y)), "gated_group_norm")
    _count()
    return out


def glu(x, ff, limit=None) -> torch.Tensor:
    half = x.shape[-1] // 2
    out = torch.empty((*x.shape[:-1], half), dtype=x.dtype, device=x.device)
    _contiguous(x)
    _check(lib().kvb_glu(_p(x), _p(out), _ll(x.numel() // (2 * half)), _ll(2 * half), half, ff, half, _f(limit or 0.0), code(x.dtype), _stream(x)), "glu")
    _count()
    return out


# ---------------------------------------------------------------------------------------------- routed experts
def moe_tile(n_choices: int, n_expert: int, dtype: torch.dtype) -> int:
    """Rows per tile of the grouped products: the expected number of tokens per expert, 16 … 256."""
    if dtype != torch.bfloat16 or FORCE_SIMPLE:
        return 32
    per = n_choices / n_expert
    tile = 16
    while tile < 256 and tile < per:
        tile *= 2
    return tile


def moe_forward(h, logits, up, down, top: int, act: int, rule, n_up: int, n_down: int, correction=None):
    """``h (n, width)``, fp32 router ``logits (n, E)``, ``up (E, ff, ldw)`` (gated: ``(E, 2 ff, ldw)``, rows of gate and up in turns),
    ``down (E, width, ldf)`` (rows padded to multiples of 8). Returns ``(expert_out, row (n, top), weight (n, top))``: row of every choice in ``expert_out``."""
    n, width = h.shape
    E = logits.shape[1]
    dev, dt = h.device, h.dtype
    _contiguous(h, logits, up, down, correction)
    router = _Router(int(rule.score == "sigmoid"), rule.groups, rule.keep, int(rule.renormalize), rule.eps,
                     None if correction is None else correction.data_ptr())
    tile = moe_tile(n * top, E, dt)
    max_tiles = n * top // tile + min(E, n * top)
    ints = torch.empty(E + 2 * n * top + 1 + 2 * max_tiles, dtype=torch.int32, device=dev)
    counters, expert, row, plan, tile_expert, tile_row = torch.split(ints, [E, n * top, n * top, 1, max_tiles, max_tiles])
    weight = torch.empty((n, top), dtype=torch.float32, device=dev)
    _check(lib().kvb_moe_route(_p(logits), _p(expert), _p(weight), _p(row), _p(counters), _p(plan), _p(tile_expert), _p(tile_row), _ll(n), E,
                               top, tile, max_tiles, ctypes.byref(router), _stream(h)), "moe_route")
    ldw, ldf = up.shape[2], down.shape[2]
    ldo = (n_down + 7) // 8 * 8
    sorted_h = torch.empty((max_tiles * tile, ldw), dtype=dt, device=dev)
    _check(lib().kvb_moe_gather(_p(h), _p(row), _p(sorted_h), _ll(n), top, width, _ll(ldw), code(dt), _stream(h)), "moe_gather")
    hidden = torch.empty((max_tiles * tile, ldf), dtype=dt, device=dev)
    st = _p(status_word(dev))
    _check(lib().kvb_moe_gemm(_p(sorted_h), _p(up), _p(hidden), _p(plan), _p(tile_expert), _p(tile_row), tile, max_tiles, E, up.shape[1], width,
                              _ll(ldw), _ll(ldf), act, code(dt), int(FORCE_SIMPLE), st, _stream(h)), "moe_gemm (up)")
    out = torch.empty((max_tiles * tile, ldo), dtype=dt, device=dev)
    _check(lib().kvb_moe_gemm(_p(hidden), _p(down), _p(out), _p(plan), _p(tile_expert), _p(tile_row), tile, max_tiles, E, n_down, n_up,
                              _ll(ldf), _ll(ldo), 0, code(dt), int(FORCE_SIMPLE), st, _stream(h)), "moe_gemm (down)")
    _count(6)
    return out, row.view(n, top), weight
