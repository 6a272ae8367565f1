"""Plain, slow restatement of the Ladadra design in float64, written from its equations: one function per mechanism, no code
shared with the package. Works on tensors under the design's own names and on the content of its ``config.json``; also
makes random models. The writer of model folders is the one of ``pazenex_oracle``."""
import math

import torch

from pazenex_oracle import rms_norm, sigmoid, silu, write_model  # noqa: F401 (plain float64 functions of one vector)


# ------------------------------------------------------------------------------------------------- mechanisms
def frequencies(rot):
    """Angle per position of every rotated pair. With scaling: wavelengths above original / low are stretched by the factor, those
    below original / high stay, those between are blended."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wavelength = 2 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wavelength >= sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(vec, pos, rot):
    out, half = vec.clone(), rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        c, s = math.cos(pos * f), math.sin(pos * f)
        u, v = float(vec[i]), float(vec[half + i])
        out[i], out[half + i] = u * c - v * s, v * c + u * s
    return out


def rotate_rows(x, rot):
    """``x (T, heads, dim)``, position = row."""
    f = torch.tensor(frequencies(rot), dtype=torch.float64)
    a = torch.arange(len(x), dtype=torch.float64)[:, None, None] * f
    half = rot["dims"] // 2
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[..., 2 * half :]), -1)


def sees_chunked(i, j, size):
    return j <= i and (size is None or i // size == j // size)


def sees_window(i, j, size, keep_first):
    return j <= i and (size is None or i - j < size or j < keep_first)


def soft_cap(score, cap):
    return score if not cap else cap * math.tanh(score / cap)


def attend(q, k, v, scale, sees, cap=None, sink=None):
    """One head: ``q, k (T, D)``, ``v (T, V)``; ``sees(i, j)``; a sink adds exp(sink) to the denominator."""
    out = []
    for i in range(len(q)):
        js = [j for j in range(i + 1) if sees(i, j)]
        s = [soft_cap(x * scale, cap) for x in (k[js] @ q[i]).tolist()]
        top = max(s + ([] if sink is None else [sink]))
        e = torch.tensor([math.exp(x - top) for x in s], dtype=torch.float64)
        out.append((e @ v[js]) / (float(e.sum()) + (0.0 if sink is None else math.exp(sink - top))))
    return torch.stack(out)


def attention(h, w, m, eps):
    """``w``: tensors of one mixer by their last name. Returns ``(T, width)``."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = h @ w["q"].T + w["q.b"]
    k = h @ w["k"].T + w["k.b"]
    v = (h @ w["v"].T + w["v.b"]).view(len(h), G, m["vdim"])
    q = torch.stack([rms_norm(r, w["q.norm"], eps) for r in q]).view(len(h), H, d)
    k = torch.stack([rms_norm(r, w["k.norm"], eps) for r in k]).view(len(h), G, d)
    q, k = rotate_rows(q, m["rot"]), rotate_rows(k, m["rot"])
    size = (m.get("mask") or {}).get("size")
    gate = sigmoid(h @ w["g"].T)
    heads = []
    for n in range(H):
        y = attend(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], m["scale"], lambda i, j: sees_chunked(i, j, size), m.get("softcap"),
                   float(w["sink"][n]))
        heads.append(y * gate[:, n : n + 1])
    return torch.cat(heads, 1) @ w["o"].T


def difference(a1, a2, lam, diff, eps):
    o = a1 - lam * a2
    return torch.stack([r / math.sqrt(float((r * r).mean()) + eps) for r in o]) * (1 - diff)


def differential_attention(h, w, m, eps):
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], len(h)
    norm = lambda x, wt: torch.stack([rms_norm(r, wt, eps) for r in x.reshape(-1, d)])
    q = norm(h @ w["q"].T, w["q.norm"]).view(T, H, 2, d)
    k = norm(h @ w["k"].T, w["k.norm"]).view(T, G, 2, d)
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    mask = m.get("mask") or {}
    sees = lambda i, j: sees_window(i, j, mask.get("size"), mask.get("keep_first", 0))
    lam = math.exp(float((w["lq1"] * w["lk1"]).sum())) - math.exp(float((w["lq2"] * w["lk2"]).sum())) + m["diff"]
    heads = []
    for n in range(H):
        a = [attend(q[:, n, i], k[:, n // (H // G), i], v[:, n // (H // G)], m["scale"], sees) for i in range(2)]
        heads.append(difference(a[0], a[1], lam, m["diff"], eps))
    return torch.cat(heads, 1) @ w["o"].T


def retain(q, k, v, decay):
    """One head, token by token. Returns ``o (T, V)`` and the last state ``(D, V)``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64)
    out = []
    for t in range(len(q)):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def retention(h, w, m, eps):
    H, d, P, T = m["heads"], m["dim"], m["vdim"], len(h)
    q = rotate_rows((h @ w["q"].T).view(T, H, d), m["rot"])
    k = rotate_rows((h @ w["k"].T).view(T, H, d), m["rot"]) * d**-0.5
    v = (h @ w["v"].T).view(T, H, P)
    ones = torch.ones(P, dtype=torch.float64)
    o = [torch.stack([rms_norm(r, ones, eps) for r in retain(q[:, n], k[:, n], v[:, n], m["decay"][n])[0]]) for n in range(H)]
    return (torch.cat(o, 1) * silu(h @ w["g"].T)) @ w["o"].T


def swiglu(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose(scores, correction, top, groups):
    """Experts of one token: the largest corrected scores, out of the groups whose two largest sum to most."""
    E = len(scores)
    c = [float(scores[e]) + float(correction[e]) for e in range(E)]
    count, keep = (groups["count"], groups["keep"]) if groups else (1, 1)
    size = E // count
    rank = sorted(range(count), key=lambda g: -sum(sorted(c[g * size : (g + 1) * size], reverse=True)[:2]))
    allowed = [e for g in rank[:keep] for e in range(g * size, (g + 1) * size)]
    return sorted(allowed, key=lambda e: -c[e])[:top]


def experts(h, w, f):
    r = f["router"]
    out = []
    for x in h:
        s = sigmoid(w["router"] @ x)
        chosen = choose(s, w["correction"], r["top"], r.get("groups"))
        total = sum(float(s[e]) for e in chosen) + 1e-20
        y = torch.zeros_like(x)
        for e in chosen:
            y = y + float(s[e]) / total * swiglu(x, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
        if f.get("shared"):
            y = y + swiglu(x, w["shared.gate"], w["shared.up"], w["shared.down"])
        out.append(y)
    return torch.stack(out)


def feed_forward(h, w, f):
    return experts(h, w, f) if f["kind"] == "moe" else swiglu(h, w["gate"], w["up"], w["down"])


MIXERS = {"attention": attention, "attention_2": differential_attention, "retention": retention}


# -------------------------------------------------------------------------------------------------- the model
def part(w, prefix):
    return {k[len(prefix) :]: v for k, v in w.items() if k.startswith(prefix)}


def add_normed(x, y, weight, eps):
    return x + torch.stack([rms_norm(r, weight, eps) for r in y])


def forward(tokens, w, content):
    """Logits ``(T, vocab)`` and the stream after every layer, float64."""
    w = {k: v.double() for k, v in w.items()}
    eps = content["norm"]["eps"]
    x, after = torch.stack([w["embed"][t] for t in tokens]), []
    for i, layer in enumerate(content["layers"]):
        p = f"l{i}."
        x = add_normed(x, MIXERS[layer["type"]](x, part(w, p + "mix."), layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = add_normed(x, feed_forward(x, part(w, p + "mlp."), layer["mlp"]), w[p + "norm2"], eps)
        after.append(x)
    return torch.stack([rms_norm(r, w["final.norm"], eps) for r in x]) @ w["embed"].T, after


def greedy(prompt, n_new, w, content):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(tokens, w, content)[0][-1].argmax()))
    return tokens[len(prompt) :]


# ---------------------------------------------------------------------------------------------- random models
def dense(ff=28):
    return {"kind": "dense", "ff": ff}


def moe(n=10, top=3, groups=(5, 2), ff=12, shared=20):
    r = {"experts": n, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def attention_layer(heads=6, kv_heads=2, dim=20, vdim=12, dims=12, base=900.0, scaling=(3.0, 1.5, 5.0, 60), scale=0.4, cap=4.0, size=24,
                    mlp=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if cap:
        m["softcap"] = cap
    if size:
        m["mask"] = {"size": size}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def differential_layer(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.4, size=9, keep_first=3, diff=0.35, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if size:
        m["mask"] = {"size": size, "keep_first": keep_first}
    return {"type": "attention_2", "mlp": mlp, "mixer": m}


def retention_layer(heads=3, dim=16, vdim=24, dims=12, base=500.0, decay=(0.7, 0.96, 0.995), mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": base, "dims": dims}}
    return {"type": "retention", "mlp": mlp, "mixer": m}


def content(layers, width=40, vocab=61, eps=1e-4):
    return {"architecture": "Ladadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def tensors(c, seed=0, decided=False):
    """Random bf16 tensors. Norm weights, sinks, biases and corrections differ from what would hide them. ``decided``: corrections so far
    apart that rounding changes no choice of experts."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, gain=1.0):
        return torch.randn(*shape, generator=g) * (gain / math.sqrt(shape[-1]))

    def near(value, *shape, spread=0.2):
        return value + spread * torch.randn(shape, generator=g)

    W = c["width"]
    w = {"embed": torch.randn(c["vocab"], W, generator=g), "final.norm": near(1.2, W)}

    def glu(prefix, ff):
        w.update({prefix + "gate": mat(ff, W), prefix + "up": mat(ff, W), prefix + "down": mat(W, ff)})

    for i, la in enumerate(c["layers"]):
        p, m, f = f"l{i}.", la["mixer"], la["mlp"]
        H, P, d = m["heads"], m["vdim"], m["dim"]
        w.update({p + "norm1": near(0.6, W), p + "norm2": near(0.5, W), p + "mix.o": mat(W, H * P)})
        if la["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * P)):
                w.update({f"{p}mix.{n}": mat(rows, W), f"{p}mix.{n}.b": near(0.2, rows, spread=0.5)})
            w.update({p + "mix.q.norm": near(1.2, H * d, spread=0.4), p + "mix.k.norm": near(1.2, G * d, spread=0.4),
                      p + "mix.g": mat(H, W, gain=1.5), p + "mix.sink": near(0.5, H, spread=1.5)})
        elif la["type"] == "attention_2":
            G = m["kv_heads"]
            w.update({p + "mix.q": mat(2 * H * d, W), p + "mix.k": mat(2 * G * d, W), p + "mix.v": mat(G * P, W),
                      p + "mix.q.norm": near(1.2, d, spread=0.4), p + "mix.k.norm": near(1.2, d, spread=0.4)})
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + "mix." + n] = near(0.1, d, spread=0.3)
        else:
            w.update({p + "mix.q": mat(H * d, W), p + "mix.k": mat(H * d, W), p + "mix.v": mat(H * P, W), p + "mix.g": mat(H * P, W)})
        if f is None:
            continue
        if f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
            continue
        E = f["router"]["experts"]
        for e in range(E):
            glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
        w.update({p + "mlp.router": mat(E, W, gain=2.0), p + "mlp.correction": near(-0.4, E, spread=0.5)})
        if decided:
            w[p + "mlp.correction"] = 3 * 1.8 ** torch.randperm(E, generator=g).float()
        if f.get("shared"):
            glu(p + "mlp.shared.", f["shared"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
