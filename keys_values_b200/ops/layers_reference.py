"""PyTorch restatement of :mod:`keys_values_b200.ops.layers` for CPU tensors (same layouts, same padding)."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def _norm_and_shift(x, gain, shift, state, h, hs, seq, eps) -> None:
    if gain is None:
        return
    hf = x * (gain / torch.sqrt(x.square().mean(-1, keepdim=True) + eps))
    h.copy_(hf)
    if shift is None:
        return
    slots = seq.slots.long()
    first = torch.where(seq.start[:, None] > 0, state[slots], torch.zeros_like(state[slots]))
    before = torch.cat((first[:, None], hf[:, :-1]), dim=1)
    hs.copy_(hf + (before - hf) * shift)
    for b, n in enumerate(seq.count.tolist()):
        if n > 0:
            state[slots[b]] = hf[b, n - 1]


def embed_edge(idx, prev_token, embed, bigram, buckets, mul_prev, mul_cur, hist, gain, shift, state, h, hs, seq, eps) -> None:
    if int(idx.min()) < 0 or int(idx.max()) >= embed.shape[0]:
        raise IndexError("token id outside of the vocabulary")
    x = embed[idx].float()
    if bigram is not None:
        prev = torch.cat((prev_token[seq.slots.long()].long()[:, None], idx[:, :-1]), dim=1)
        row = (prev * mul_prev + idx * mul_cur) % buckets
        row[:, 0] = torch.where(seq.start > 0, row[:, 0], torch.full_like(row[:, 0], buckets))
        x = x + bigram[row].float()
    hist.copy_(x)
    _norm_and_shift(x, gain, shift, state, h, hs, seq, eps)


def layer_edge(x_in, mix, expert_out, expert_row, expert_w, hist, n_hist, coef, x_out, gain, shift, state, h, hs, seq, eps) -> None:
    sub = mix.float()
    if expert_out is not None:
        width = sub.shape[-1]
        sub = sub + (expert_w[:, :, None] * expert_out[expert_row.long()][:, :, :width].float()).sum(1).view_as(sub)
    new = x_in + sub
    if coef is None:
        x_out.copy_(new)
    else:
        hist[n_hist] = new
        x_out.copy_((coef.view(-1, 1, 1, 1) * hist[: n_hist + 1]).sum(0))
    _norm_and_shift(x_out, gain, shift, state, h, hs, seq, eps)


def scalar_rmsnorm(x, rows, gain, eps, dtype):
    x = x if rows is None else x[rows]
    return (x * (gain / torch.sqrt(x.square().mean(-1, keepdim=True) + eps))).to(dtype)


def sequence_advance(idx, pos, prev_token, seq) -> None:
    for b, (slot, n) in enumerate(zip(seq.slots.tolist(), seq.count.tolist())):
        if n > 0:
            pos[slot] += n
            prev_token[slot] = int(idx[b, n - 1])


def _rotate(x, cos, sin, dims):
    half = dims // 2
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, rest), dim=-1)


def latent_prep(qkv, norm_w, freq, latent, ring, seq, P, s, eps):
    B, T, _ = qkv.shape
    nq = s.heads * (s.dim + s.rot)
    qf = qkv[..., :nq].float().view(B, T, s.heads, s.dim + s.rot)
    c, kr = qkv[..., nq : nq + s.kv_rank].float(), qkv[..., nq + s.kv_rank :].float()
    pos = seq.start[:, None] + torch.arange(T)
    angle = pos.float()[..., None] * freq
    cos, sin = angle.cos(), angle.sin()
    q = torch.zeros(B, T, s.heads, s.dimp + s.rp, dtype=qkv.dtype)
    q[..., : s.dim] = qf[..., : s.dim]
    q[..., s.dimp : s.dimp + s.rot] = _rotate(qf[..., s.dim :], cos[:, :, None], sin[:, :, None], s.rot_dims)
    row = torch.zeros(B, T, s.row, dtype=qkv.dtype)
    row[..., : s.kv_rank] = c / torch.sqrt(c.square().mean(-1, keepdim=True) + eps) * norm_w
    row[..., s.kvp : s.kvp + s.rot] = _rotate(kr, cos, sin, s.rot_dims)
    if latent is not None:
        latent[:, P:] = row
    if ring is not None:
        C = ring.shape[1]
        for b, (slot, n) in enumerate(zip(seq.slots.tolist(), seq.count.tolist())):
            for t in range(max(0, n - C), n):
                ring[slot, int(pos[b, t]) % C] = row[b, t]
    return q


def ring_gather(ring, latent, seq, P) -> None:
    C = ring.shape[1]
    latent[:, :P] = 0
    for b, (slot, start) in enumerate(zip(seq.slots.tolist(), seq.start.tolist())):
        for j in range(P):
            p = start - P + j
            if p >= max(0, start - C):
                latent[b, j] = ring[slot, p % C]


def latent_attend(q, kv, latent, seq, P, s, window, scale):
    B, T = q.shape[:2]
    N = P + T
    kv = kv.view(B, N, s.heads, s.dimp + s.vdp).float()
    qf = q.float()
    score = torch.einsum("bthd,bjhd->bhtj", qf[..., : s.dimp], kv[..., : s.dimp])
    score = (score + torch.einsum("bthr,bjr->bhtj", qf[..., s.dimp :], latent[..., s.kvp :].float())) * scale
    j = torch.arange(N)
    back = P + torch.arange(T)[:, None] - j
    seen = (back >= 0) & ((back < window) if window > 0 else torch.ones_like(back, dtype=torch.bool))
    seen = seen[None] & (j[None, None] >= P - seq.start[:, None, None])
    w = score.masked_fill(~seen[:, None], float("-inf")).softmax(-1)
    return torch.einsum("bhtj,bjhv->bthv", w, kv[..., s.dimp :]).reshape(B, T, s.heads * s.vdp).to(q.dtype)


def latent_decode(q_abs, q, ring, seq, s, scale):
    out = torch.empty_like(q_abs)
    for b, (slot, start) in enumerate(zip(seq.slots.tolist(), seq.start.tolist())):
        rows = ring[slot, : min(start + 1, ring.shape[1])].float()
        qc = torch.cat((q_abs[:, b].float(), q[b, 0, :, s.dimp :].float()), dim=-1)
        w = (qc @ rows.t() * scale).softmax(-1)
        out[:, b] = (w @ rows[:, : s.kvp]).to(out.dtype)
    return out


def _choose(score, correction, top, rule):
    choice = score if correction is None else score + correction
    if rule.groups > 1:
        n, E = choice.shape
        parts = choice.view(n, rule.groups, -1)
        group = parts.topk(min(2, parts.shape[-1]), dim=-1).values.sum(-1)
        best = torch.sort(group, dim=-1, descending=True, stable=True)[1][:, : rule.keep]
        seen = torch.zeros_like(group, dtype=torch.bool).scatter_(1, best, True)
        choice = parts.masked_fill(~seen[..., None], float("-inf")).reshape(n, E)
    return torch.sort(choice, dim=-1, descending=True, stable=True)[1][:, :top]  # ties: lower index


def moe_forward(h, logits, up, down, top, act, rule, n_up, n_down, correction=None):
    n, width = h.shape
    scores = logits.softmax(-1) if rule.score == "softmax" else torch.sigmoid(logits)
    expert = _choose(scores, correction, top, rule)
    weight = scores.gather(1, expert)
    if rule.renormalize:
        weight = weight / (weight.sum(-1, keepdim=True) + rule.eps)
    out = torch.zeros(n * top, (n_down + 7) // 8 * 8, dtype=h.dtype)
    for e in range(logits.shape[1]):
        t, k = torch.where(expert == e)
        if t.numel():
            z = h[t].float() @ up[e, : 2 * n_up if act == 2 else n_up, :width].float().t()
            if act == 1:
                z = z.relu().square()
            elif act == 2:
                z = F.silu(z[:, ::2]) * z[:, 1::2]
            out[t * top + k, :n_down] = (z.to(h.dtype).float() @ down[e, :n_down, :n_up].float().t()).to(h.dtype)
    return out, torch.arange(n * top, dtype=torch.int32).view(n, top), weight


def glu(x, ff, limit=None):
    n = x.shape[-1] // 2
    g, u = x[..., :n].float(), x[..., n:].float()
    if limit is None:
        y = F.silu(g) * u
    else:
        g = g.clamp(max=limit)
        y = g * torch.sigmoid(1.702 * g) * (u.clamp(-limit, limit) + 1)
    y[..., ff:] = 0
    return y.to(x.dtype)


# ---- sequential layers
def _norm(x, weight, eps, center):
    if center:
        x = x - x.mean(-1, keepdim=True)
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps) * weight


def norm_edge(x_in, sub, after, x_out, before, h, idx, embed, step, eps, center, experts=None, tokens=None) -> None:
    x = torch.zeros_like(x_out) if x_in is None else x_in
    s = None if sub is None else sub.float()
    if experts is not None:
        out, row, weight = experts
        width = x_out.shape[-1]
        add = (weight[:, :, None] * out[row.long()][:, :, :width].float()).sum(1).view_as(x_out)
        s = add if s is None else s + add
    if s is not None:
        x = x + (s if after is None else _norm(s, after, eps, center))
    if embed is not None:
        if int(idx.min()) < 0 or int(idx.max()) >= embed.shape[0]:
            raise IndexError("token id outside of the vocabulary")
        x = x + embed[idx].float()
    if tokens is not None and tokens.table is not None:
        at = (tokens.seq.start[:, None] + torch.arange(x_out.shape[1])).clamp(max=tokens.table.shape[0] - 1)  # padding may lie beyond
        x = x + tokens.table[at.long()].float()
    if step is not None:
        x = x + step
    x_out.copy_(x)
    if h is not None:
        h.copy_(x if before is None else _norm(x, before, eps, center))
        if tokens is not None and tokens.conv is not None:
            short_conv(h.clone(), 0, tokens.conv, None, tokens.ring, tokens.seq, False, h)


def row_norm(x, weight, eps, center, dtype):
    return _norm(x, weight, eps, center).to(dtype)


def activate(x, act):
    return x.relu_().square_() if act == 1 else x


# ---- grouped-query attention
def _places(s, plan, positions):
    p = torch.as_tensor(positions)
    if s.pool:
        return plan.head + p % plan.ring
    return p if plan.ring == 0 else torch.where(p < plan.head, p, plan.head + (p - plan.head) % plan.ring)


def grouped_prep(qkv, norm_q, norm_k, freq, rows, seq, s, eps, plan, q_scale=None):
    B, T, _ = qkv.shape
    H, G = s.heads * s.maps, 0 if s.borrowed else s.kv_heads * s.maps
    nq, nk = H * s.dimp, G * s.dimp
    q, k = qkv[..., :nq].float(), qkv[..., nq : nq + nk].float()
    if norm_q is not None and s.head_norm:
        q, k = (x.view(B, T, -1, s.dimp) for x in (q, k))
        q, k = (x / torch.sqrt(x.square().sum(-1, keepdim=True) / s.dim + eps) * w for x, w in ((q, norm_q), (k, norm_k)))
    elif norm_q is not None:  # padding adds nothing to the sums of squares
        q = q / torch.sqrt(q.square().sum(-1, keepdim=True) / (H * s.dim) + eps) * norm_q
        k = k / torch.sqrt(k.square().sum(-1, keepdim=True) / (G * s.dim) + eps) * norm_k
    angle = (seq.start[:, None] + torch.arange(T)).float()[..., None] * freq
    cos, sin = angle.cos()[:, :, None], angle.sin()[:, :, None]
    q = _rotate(q.reshape(B, T, H, s.dimp), cos, sin, s.rot_dims)
    if q_scale is not None:
        q = q * q_scale.repeat_interleave(s.maps)[:, None]
    q = q.to(qkv.dtype)
    if s.borrowed:
        return q
    k = _rotate(k.reshape(B, T, G, s.dimp), cos, sin, s.rot_dims).to(qkv.dtype).reshape(B, T, s.kv_heads, s.maps * s.dimp)
    v = qkv[..., s.value_col : s.value_col + s.kv_heads * s.vdp].view(B, T, s.kv_heads, s.vdp)
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        at = _places(s, plan, torch.arange(start, start + n))
        rows[slot, at] = torch.cat((k[b, :n], v[b, :n]), -1)
        if s.pool:
            for block in range(start // s.pool, (start + n) // s.pool):
                held = _places(s, plan, torch.arange(block * s.pool, (block + 1) * s.pool))
                rows[slot, block] = rows[slot, held].float().mean(0).to(rows.dtype)
    return q


def _seen(s, query, key):
    """Which of the positions ``key (N,)`` each of ``query (T,)`` sees."""
    i, j = query[:, None], key[None]
    seen = j <= i
    if s.chunk:
        return seen & (i // s.chunk == j // s.chunk)
    return seen & ((i - j < s.window) | (j < s.keep)) if s.window else seen


def grouped_attend(q, qkv, rows, seq, s, sink, plan, into=None):
    B, T = q.shape[:2]
    out = torch.zeros(B, T, s.heads, s.vdp)
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        if n == 0:
            continue
        key = torch.arange(start + n)
        if plan.ring:  # positions that are seen no more have lost their rows
            key = key[((key < plan.head) & (s.pool == 0)) | (key > start - s.span)]
        places, hidden = _places(s, plan, key), ~_seen(s, start + torch.arange(n), key)
        if s.pool:
            block = torch.arange((start + n) // s.pool)
            places = torch.cat((block, places))
            hidden = torch.cat(((block[None] + 1) * s.pool - 1 > start + torch.arange(n)[:, None] - s.window, hidden), 1)
        kv = rows[slot, places].float().repeat_interleave(s.heads // s.kv_heads, dim=1)
        maps = []
        for u in range(s.maps):
            score = torch.einsum("thd,jhd->htj", q[b, :n, u :: s.maps].float(), kv[..., u * s.dimp : (u + 1) * s.dimp]) * s.scale
            if s.softcap:
                score = s.softcap * torch.tanh(score / s.softcap)
            score = score.masked_fill(hidden, float("-inf"))
            if s.sink:
                add = torch.zeros(s.heads) if sink is None else sink
                score = torch.cat((score, add.view(-1, 1, 1).expand(-1, n, 1)), dim=-1)
            maps.append(torch.einsum("htj,jhv->thv", score.softmax(-1)[..., : len(places)], kv[..., s.maps * s.dimp :]))
        if s.maps == 2:
            d = maps[0] - s.lam * maps[1]
            maps[0] = d / torch.sqrt(d.square().sum(-1, keepdim=True) / s.vdim + s.eps)
        out[b, :n] = maps[0] * s.post
    if s.gate:
        gate = torch.sigmoid(qkv[..., s.gate_col : s.gate_col + s.heads * s.gate_cols].float())
        out = out * gate.view(B, T, s.heads, s.gate_cols)
    out = out.view(B, T, -1).to(q.dtype)
    return out if into is None else into.copy_(out)


# ---- retention
def retention_prep(qk, freq, seq, s, dtype):
    B, T, _ = qk.shape
    x = qk[..., : s.qk].view(B, T, 2 * s.heads, s.np)
    angle = (seq.start[:, None] + torch.arange(T)).float()[..., None] * freq
    x = _rotate(x, angle.cos()[:, :, None], angle.sin()[:, :, None], s.rot_dims).clone()
    x[:, :, s.heads :] *= s.key_scale
    return x.reshape(B, T, s.qk).to(dtype)


def retention_scan(qk, v, decay, log2_decay, state, seq, s):
    B, T = qk.shape[:2]
    q, k = qk.float().view(B, T, 2, s.heads, s.np).unbind(2)
    v = v[..., : s.inner].float().reshape(B, T, s.heads, s.vdp)
    y = torch.zeros(B, T, s.heads, s.vdp)
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
        for t in range(n):
            S = decay[:, None, None] * S + k[b, t, :, :, None] * v[b, t, :, None]
            y[b, t] = torch.einsum("hnp,hn->hp", S, q[b, t])
        if n > 0:
            state[slot] = S
    return y.view(B, T, -1).to(qk.dtype)


def head_norm_gate(y, gate, s, eps, weight=None):
    x = y.float().view(*y.shape[:-1], s.heads, s.vdp)
    x = x / torch.sqrt(x.square().sum(-1, keepdim=True) / s.vdim + eps)
    if weight is not None:
        x = x * weight
    return (x.view(y.shape) * F.silu(gate[..., : s.inner].float())).to(y.dtype)


def retention_step(u, freq, decay, state, seq, s, eps, dtype):
    qk = retention_prep(u, freq, seq, s, torch.float32)
    y = retention_scan(qk, u[..., s.qk :], decay, None, state, seq, s)
    return head_norm_gate(y, u[..., s.qk + s.inner :], s, eps).to(dtype)


# ---- gated linear attention
def _log_decay(a, decay, s):
    """Logarithms of the decays ``(B, T, heads, np)``."""
    z = a.float()[..., : s.rank] @ decay.weight + decay.bias
    return (F.logsigmoid(z) / s.tau).view(*a.shape[:-1], s.heads, s.np)


def gated_linear_scan(qka, v, decay, state, seq, s):
    B, T = qka.shape[:2]
    q, k = qka[..., : s.qk].view(B, T, 2, s.heads, s.np).unbind(2)
    alpha = torch.exp(_log_decay(qka[..., s.qk :], decay, s))
    dtype, v = v.dtype, v[..., : s.inner].float().reshape(B, T, s.heads, s.vdp)
    y = torch.zeros(B, T, s.heads, s.vdp)
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
        for t in range(n):
            S = alpha[b, t, :, :, None] * S + k[b, t, :, :, None] * v[b, t, :, None]
            y[b, t] = torch.einsum("hnp,hn->hp", S, q[b, t] * s.query_scale)
        if n > 0:
            state[slot] = S
    return y.view(B, T, -1).to(dtype)


def gated_linear_step(u, decay, weight, state, seq, s, eps, dtype):
    y = gated_linear_scan(u[..., : s.qk + s.rp], u[..., s.qk + s.rp :], decay, state, seq, s)
    return head_norm_gate(y, u[..., s.qk + s.rp + s.inner :], s, eps, weight).to(dtype)


# ---- gated recurrence per channel
def gated_recurrence(u, w, ring, state, seq, s, scale, out):
    B, T, _ = u.shape
    x = short_conv(u, s.channels, w.conv, w.conv_bias, ring, seq, False)
    z = torch.einsum("btpk,pkn->btpn", x.float().view(B, T, s.blocks, s.pp), w.gates.float())
    r, i = (torch.sigmoid(g.reshape(B, T, -1) + b) for g, b in zip(z.split(s.pp, dim=-1), (w.bias_r, w.bias_i)))
    log_a = r * w.rate * math.log(2.0)
    a, add = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * x.float()
    y = F.gelu(u[..., : s.channels].float(), approximate="tanh") * scale
    out.zero_()
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
        for t in range(n):
            S = a[b, t] * S + add[b, t]
            out[b, t] = (S * y[b, t]).to(out.dtype)
        if n > 0:
            state[slot] = S
    return out


# ---- state-space recurrence
def short_conv(u, col, w, bias, ring, seq, silu=True, out=None):
    B, T, _ = u.shape
    taps, channels = w.shape
    x = u[..., col : col + channels].float()
    out = torch.empty(B, T, channels, dtype=u.dtype) if out is None else out
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        before = [ring[slot, p % taps].float() if p >= 0 else torch.zeros(channels) for p in range(start - taps + 1, start)]
        rows = torch.cat((torch.stack(before), x[b])) if before else x[b]
        y = sum(w[k] * rows[k : k + T] for k in range(taps)) + (0 if bias is None else bias)
        out[b] = F.silu(y) if silu else y
        for t in range(max(0, n - taps), n):
            ring[slot, (start + t) % taps] = u[b, t, col : col + channels]
    return out


def state_scan(u, xbc, dt_bias, a_log, skip, state, seq, s):
    B, T, _ = u.shape
    y = torch.zeros(B, T, s.heads, s.vdp)
    x = xbc[..., : s.inner].float().view(B, T, s.heads, s.vdp)
    bc = xbc[..., s.inner :].float().view(B, T, 2, s.groups, s.np).repeat_interleave(s.heads // s.groups, dim=3)
    dt = F.softplus(u[..., s.dt_col : s.dt_col + s.heads].float() + dt_bias, threshold=1e9)
    decay = torch.exp(-torch.exp(a_log) * dt)
    for b, (slot, start, n) in enumerate(zip(seq.slots.tolist(), seq.start.tolist(), seq.count.tolist())):
        S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
        for t in range(n):
            S = decay[b, t, :, None, None] * S + (dt[b, t, :, None] * bc[b, t, 0])[..., None] * x[b, t, :, None]
            y[b, t] = torch.einsum("hnp,hn->hp", S, bc[b, t, 1]) + skip[:, None] * x[b, t]
        if n > 0:
            state[slot] = S
    return y.view(B, T, -1).to(u.dtype)


def state_step(u, w, bias, dt_bias, a_log, skip, ring, state, seq, s):
    return state_scan(u, short_conv(u, s.inner, w, bias, ring, seq), dt_bias, a_log, skip, state, seq, s)


def gated_group_norm(y, u, weight, s, eps):
    g = y.float() * F.silu(u[..., : s.inner].float())
    lead = g.shape[:-1]
    plain = g.view(*lead, s.heads, s.vdp)[..., : s.vdim].reshape(*lead, s.norm_groups, -1)
    plain = plain / torch.sqrt(plain.square().mean(-1, keepdim=True) + eps)
    out = torch.zeros_like(g).view(*lead, s.heads, s.vdp)
    out[..., : s.vdim] = plain.reshape(*lead, s.heads, s.vdim)
    return (out.view(g.shape) * weight).to(y.dtype)
