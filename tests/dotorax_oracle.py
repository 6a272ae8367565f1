"""Plain, slow restatement of the Dotorax design in float64, written from its equations: one function per mechanism, no code
shared with the package. Works on tensors under the design's own names and on the content of its ``config.json``; also
makes random models. The writer of model folders is the one of ``pazenex_oracle``."""
import math

import torch

from pazenex_oracle import sigmoid, silu, write_model  # noqa: F401 (plain float64 functions)


# ------------------------------------------------------------------------------------------------- mechanisms
def over_rms(v, eps):
    """A vector divided by its root mean square."""
    return v / math.sqrt(float((v * v).mean()) + eps)


def norm_rows(x, w, eps):
    """Norm of every row; the weight is stored around zero."""
    return torch.stack([over_rms(r, eps) * (1 + w) for r in x])


def causal_conv(x, w, bias=None):
    """``x (T, C)``, ``w (C, taps)``, the last column meets the token itself; zeros before the start."""
    T, taps = len(x), w.shape[1]
    out = []
    for t in range(T):
        y = torch.zeros_like(x[0]) if bias is None else bias.clone()
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y = y + w[:, j] * x[s]
        out.append(y)
    return torch.stack(out)


def input_conv(h, w):
    return h + causal_conv(h, w)


def rotate_rows(x, rot, interleaved):
    """``x (T, heads, dim)``, position = row."""
    T, _, dim = x.shape
    half = rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        u, v = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        a = torch.arange(T, dtype=torch.float64)[:, None] * float(rot["base"]) ** (-2.0 * i / rot["dims"])
        out[..., u] = x[..., u] * a.cos() - x[..., v] * a.sin()
        out[..., v] = x[..., v] * a.cos() + x[..., u] * a.sin()
    return out


def softmax_sum(scores, values):
    e = torch.exp(scores - scores.max())
    return (e @ values) / e.sum()


def attend(q, k, v, scale):
    """One head, causal: ``q, k (T, D)``, ``v (T, V)``."""
    return torch.stack([softmax_sum(k[: i + 1] @ q[i] * scale, v[: i + 1]) for i in range(len(q))])


def blocks_seen(i, size, pool):
    """Blocks of ``pool`` positions that end before the window of position ``i``."""
    n = 0
    while n * pool + pool - 1 <= i - size:
        n += 1
    return n


def pooled_row(i, q, k, v, scale, size, pool):
    """Result of one query at position ``i`` over a window of tokens and the means of the blocks that lie before it, in one softmax."""
    n, first = blocks_seen(i, size, pool), max(0, i - size + 1)
    keys, values = list(k[first : i + 1]), list(v[first : i + 1])
    for b in range(n):
        keys.append(k[b * pool : (b + 1) * pool].mean(0))
        values.append(v[b * pool : (b + 1) * pool].mean(0))
    return softmax_sum(torch.stack(keys) @ q * scale, torch.stack(values))


def attend_pooled(q, k, v, scale, size, pool):
    """One head."""
    return torch.stack([pooled_row(i, q[i], k, v, scale, size, pool) for i in range(len(q))])


def keys_values(h, w, m):
    G = m["kv_heads"]
    return rotate_rows((h @ w["k"].T).view(len(h), G, m["dim"]), m["rot"], False), (h @ w["v"].T).view(len(h), G, m["vdim"])


def attention(h, w, m, kv):
    """``kv``: keys and values of the layer they are taken from. Returns ``(T, width)``."""
    H, G = m["heads"], m["kv_heads"]
    k, v = kv
    q = rotate_rows((h @ w["q"].T).view(len(h), H, m["dim"]), m["rot"], False)
    gate = sigmoid(h @ w["g"].T)
    heads = [attend(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], m["scale"]) * gate[:, n : n + 1] for n in range(H)]
    return torch.cat(heads, 1) @ w["o"].T


def pooled_attention(h, w, m, eps):
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], len(h)

    def unit(x):
        return torch.stack([over_rms(r, eps) for r in x.reshape(-1, d)]).view(x.shape)

    q = unit(rotate_rows((h @ w["q"].T).view(T, H, d), m["rot"], True))
    k = unit(rotate_rows((h @ w["k"].T).view(T, G, d), m["rot"], True))
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    size, pool = m["mask"]["size"], m["mask"]["pool"]
    heads = [attend_pooled(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], m["scale"] * float(w["temp"][n]), size, pool) for n in range(H)]
    return torch.cat(heads, 1) @ w["o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z**3)))


def gated_lru(u, r, i, lam):
    """``u, r, i (T, C)``: inputs and gates. Returns the states ``(T, C)``."""
    S = torch.zeros_like(lam)
    out = []
    for t in range(len(u)):
        log_a = -8 * r[t] * torch.log1p(torch.exp(lam))
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def block_product(u, w, b):
    """``u (T, C)`` in equal parts, each with a matrix ``w[part]`` and a bias ``b[part]`` of its own."""
    n = len(w)
    return torch.cat([x @ w[p].T + b[p] for p, x in enumerate(u.chunk(n, dim=1))], 1)


def griffin(h, w, m):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    S = gated_lru(u, sigmoid(block_product(u, w["ra"], w["ra.b"])), sigmoid(block_product(u, w["ri"], w["ri.b"])), w["lam"])
    return (S * y) @ w["o"].T


def side_by_side(h, w, m, eps):
    left = pooled_attention(h, part(w, "left."), m["left"], eps)
    return m["left_scale"] * left + m["right_scale"] * griffin(h, part(w, "right."), m["right"])


def gla_recurrence(q, k, v, alpha):
    """One head, token by token: ``q, k, alpha (T, D)``, ``v (T, V)``. Returns ``o (T, V)`` and the last state ``(D, V)``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64)
    out = []
    for t in range(len(q)):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def gla(h, w, m, eps):
    H, d, P, T = m["heads"], m["dim"], m["vdim"], len(h)
    q, k, v = (h @ w["q"].T).view(T, H, d) * d**-0.5, (h @ w["k"].T).view(T, H, d), (h @ w["v"].T).view(T, H, P)
    alpha = (sigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]) ** (1.0 / m["tau"])).view(T, H, d)
    o = [torch.stack([over_rms(r, eps) * w["norm"] for r in gla_recurrence(q[:, n], k[:, n], v[:, n], alpha[:, n])[0]]) for n in range(H)]
    return (torch.cat(o, 1) * silu(h @ w["g"].T)) @ w["o"].T


def clamped_unit(gate, up, limit):
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def feed_forward(h, w, f):
    return clamped_unit(h @ w["gate"].T, h @ w["up"].T, f["limit"]) @ w["down"].T


# -------------------------------------------------------------------------------------------------- the model
def part(w, prefix):
    return {k[len(prefix) :]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens, w, content):
    """Logits ``(T, vocab)`` and the stream after every layer, float64."""
    w = {k: v.double() for k, v in w.items()}
    eps, mult = content["norm"]["eps"], content["residual_mult"]
    x = torch.stack([w["embed"][t] + w["pos"][p] for p, t in enumerate(tokens)])
    after, held = [], {}
    for i, layer in enumerate(content["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        mix = part(w, p + "mix.")
        h = input_conv(norm_rows(x, w[p + "norm1"], eps), w[p + "canon1"])
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                held[i] = keys_values(h, mix, m)
            y = attention(h, mix, m, held[i if src is None else src])
        else:
            y = gla(h, mix, m, eps) if layer["type"] == "gla" else side_by_side(h, mix, m, eps)
        x = x + mult * norm_rows(y, w[p + "norm1b"], eps)
        if f is not None:
            h = input_conv(norm_rows(x, w[p + "norm2"], eps), w[p + "canon2"])
            x = x + mult * norm_rows(feed_forward(h, part(w, p + "mlp."), f), w[p + "norm2b"], eps)
        after.append(x)
    return norm_rows(x, w["final.norm"], eps) @ w["head"].T, after


def greedy(prompt, n_new, w, content):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(tokens, w, content)[0][-1].argmax()))
    return tokens[len(prompt) :]


# ---------------------------------------------------------------------------------------------- random models
def dense(ff=28, limit=1.1):
    return {"kind": "dense", "ff": ff, "limit": limit}


def attention_layer(heads=6, kv_heads=2, dim=20, vdim=12, dims=12, base=900.0, scale=0.4, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def parallel_layer(heads=4, kv_heads=2, dim=12, vdim=20, dims=8, base=300.0, scale=0.7, size=9, pool=4, left_scale=0.8, right_scale=1.3, width=36,
                   blocks=3, conv=3, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims},
            "mask": {"size": size, "pool": pool}}
    m = {"left": left, "left_scale": left_scale, "right": {"width": width, "blocks": blocks, "conv": conv}, "right_scale": right_scale}
    return {"type": "parallel", "mlp": mlp, "mixer": m}


def gla_layer(heads=3, dim=16, vdim=24, tau=8.0, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def content(layers, width=40, vocab=61, eps=2e-2, taps=3, mult=0.5, positions=400):
    return {"architecture": "Dotorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "residual_mult": mult,
            "max_positions": positions, "layers": layers}


def tensors(c, seed=0, rank=5):
    """Random bf16 tensors. Norm weights, biases, scales and decays differ from what would hide them; decays keep some channels for long."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, gain=1.0):
        return torch.randn(*shape, generator=g) * (gain / math.sqrt(shape[-1]))

    def near(value, *shape, spread=0.2):
        return value + spread * torch.randn(shape, generator=g)

    W, taps = c["width"], c["canon"]["taps"]
    w = {"embed": torch.randn(c["vocab"], W, generator=g), "pos": 0.5 * torch.randn(c["max_positions"], W, generator=g),
         "final.norm": near(0.2, W), "head": mat(c["vocab"], W, gain=2.0)}
    for i, la in enumerate(c["layers"]):
        p, m, f = f"l{i}.", la["mixer"], la["mlp"]
        x = p + "mix."
        w.update({p + "norm1": near(0.1, W), p + "norm1b": near(-0.2, W), p + "norm2": near(0.1, W), p + "norm2b": near(-0.3, W),
                  p + "canon1": near(0.0, W, taps, spread=0.4), p + "canon2": near(0.0, W, taps, spread=0.4)})
        if la["type"] == "gla":
            H, d, P = m["heads"], m["dim"], m["vdim"]
            w.update({x + "q": mat(H * d, W), x + "k": mat(H * d, W), x + "v": mat(H * P, W), x + "g": mat(H * P, W), x + "o": mat(W, H * P),
                      x + "norm": near(1.2, P, spread=0.4), x + "a1": mat(rank, W), x + "a2": mat(H * d, rank, gain=1.5),
                      x + "a2.b": near(1.5, H * d, spread=2.0)})
        elif la["type"] == "attention":
            H, G, d, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({x + "q": mat(H * d, W, gain=1.5), x + "g": mat(H, W, gain=1.5), x + "o": mat(W, H * P)})
            if m.get("kv_from") is None:
                w.update({x + "k": mat(G * d, W), x + "v": mat(G * P, W)})
        else:
            s, r = m["left"], m["right"]
            H, G, d, P, C, n = s["heads"], s["kv_heads"], s["dim"], s["vdim"], r["width"], r["blocks"]
            w.update({x + "left.q": mat(H * d, W), x + "left.k": mat(G * d, W), x + "left.v": mat(G * P, W), x + "left.o": mat(W, H * P),
                      x + "left.temp": near(0.9, H, spread=0.6)})
            w.update({x + "right.y": mat(C, W), x + "right.y.b": near(0.3, C), x + "right.x": mat(C, W), x + "right.x.b": near(-0.2, C),
                      x + "right.conv": mat(C, r["conv"], gain=1.2), x + "right.conv.b": near(0.1, C), x + "right.ra": mat(n, C // n, C // n, gain=1.5),
                      x + "right.ra.b": near(-0.5, n, C // n), x + "right.ri": mat(n, C // n, C // n), x + "right.ri.b": near(0.3, n, C // n),
                      x + "right.lam": near(-3.0, C, spread=1.5), x + "right.o": mat(W, C)})
        if f is not None:
            w.update({p + "mlp.gate": mat(f["ff"], W), p + "mlp.up": mat(f["ff"], W), p + "mlp.down": mat(W, f["ff"])})
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
