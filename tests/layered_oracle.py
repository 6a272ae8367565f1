"""Plain, slow restatement of the Mezilix design in float64, written from its equations: one function per mechanism,
token by token where that is the clearest form, no code shared with the package. Works on tensors under the design's own
names and on the content of its ``config.json``; also makes random models and writes them to disk."""
import json
import math
import struct

import torch


# ------------------------------------------------------------------------------------------------- mechanisms
def unit_rms(x, eps):
    return x / math.sqrt(float((x * x).mean()) + eps)


def scalar_norm(x, gain, eps):
    return torch.stack([unit_rms(row, eps) * gain for row in x])


def bigram_rows(tokens, spec):
    rows = [spec["buckets"]]
    for before, now in zip(tokens[:-1], tokens[1:]):
        rows.append((before * spec["mul_prev"] + now * spec["mul_cur"]) % spec["buckets"])
    return rows


def embedding(tokens, w, content):
    rows = bigram_rows(tokens, content["embedding"]["bigram"])
    return torch.stack([w["embed"][t] + w["bigram"][r] for t, r in zip(tokens, rows)])


def token_shift(h, blend):
    out = []
    for t in range(len(h)):
        before = h[t - 1] if t > 0 else torch.zeros_like(h[0])
        out.append(h[t] + (before - h[t]) * blend)
    return torch.stack(out)


def rotate(vec, pos, base, dims):
    out = vec.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = float(vec[i]), float(vec[i + dims // 2])
        out[i] = u * math.cos(a) - v * math.sin(a)
        out[i + dims // 2] = v * math.cos(a) + u * math.sin(a)
    return out


def latent_rows(h, w, m, eps):
    """Latents ``(T, kv_rank)`` and rotated key parts ``(T, rot_dim)``."""
    kv = h @ w["dkv"].T
    c = torch.stack([unit_rms(r[: m["kv_rank"]], eps) * w["dkv.norm"] for r in kv])
    rot = torch.stack([rotate(r[m["kv_rank"] :], t, m["rot"]["base"], m["rot"]["dims"]) for t, r in enumerate(kv)])
    return c, rot


def window_softmax_attention(q, k, v, scale, size):
    """``q, k (T, D)``, ``v (T, V)`` of one head; position i sees ``i - size < j <= i``."""
    out = []
    for i in range(len(q)):
        lo = max(0, i - size + 1)
        s = (k[lo : i + 1] @ q[i]) * scale
        p = torch.exp(s - s.max())
        out.append((p / p.sum()) @ v[lo : i + 1])
    return torch.stack(out)


def latent_attention(h, w, m, eps):
    """``w``: tensors of one mixer by their last name."""
    H, d, r, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = latent_rows(h, w, m, eps)
    q = (h @ w["q"].T).view(len(h), H, d + r)
    k_plain, v = (c @ w["uk"].T).view(len(h), H, d), (c @ w["uv"].T).view(len(h), H, dv)
    heads = []
    for n in range(H):
        q_rot = torch.stack([rotate(q[t, n, d:], t, m["rot"]["base"], m["rot"]["dims"]) for t in range(len(h))])
        heads.append(window_softmax_attention(torch.cat((q[:, n, :d], q_rot), 1), torch.cat((k_plain[:, n], k_rot), 1), v[:, n],
                                              m["scale"], m["mask"]["size"]))
    return torch.cat(heads, 1) @ w["o"].T


def routed_experts(h, w, f):
    """``w``: tensors of one feed-forward by name."""
    out = torch.zeros_like(h)
    for t, x in enumerate(h):
        z = w["router"] @ x
        s = torch.exp(z - z.max())
        s = s / s.sum()
        for e in sorted(range(len(s)), key=lambda i: -float(s[i]))[: f["router"]["top"]]:
            out[t] += s[e] * (w[f"e{e}.down"] @ torch.clamp(w[f"e{e}.up"] @ x, min=0) ** 2)
    return out


def depth_average(streams, coef):
    return sum(c * x for c, x in zip(coef, streams))


# -------------------------------------------------------------------------------------------------- the model
def _part(w, prefix):
    return {k[len(prefix) :]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens, w, content):
    """Logits ``(T, vocab)`` and the stream after every layer, float64."""
    w = {k: v.double() for k, v in w.items()}
    eps = content["norm"]["eps"]
    x = embedding(tokens, w, content)
    streams, after = [x], []
    for i, layer in enumerate(content["layers"]):
        p = f"l{i}."
        h = scalar_norm(x, w[p + "norm1"], eps)
        y = latent_attention(token_shift(h, w[p + "shift"]), _part(w, p + "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + routed_experts(h, _part(w, p + "mlp."), layer["mlp"])
        streams.append(x + y)
        x = depth_average(streams, w[p + "dwa"])
        after.append(x)
    return scalar_norm(x, w["final.norm"], eps) @ w["head"].T, after


def greedy(prompt, n_new, w, content):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(tokens, w, content)[0][-1].argmax()))
    return tokens[len(prompt) :]


# ---------------------------------------------------------------------------------------------- random models
def layer(heads=3, dim=12, rot_dim=4, vdim=20, kv_rank=24, window=9, base=700.0, experts=5, top=2, ff=16, scale=None):
    return {
        "type": "latent_attention",
        "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                  "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale},
        "mlp": None if not experts else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}},
    }


def content(layers, width=40, vocab=61, eps=1e-4, buckets=37, mul_prev=11, mul_cur=3):
    return {"architecture": "Mezilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


def tensors(c, seed=0):
    """Random bf16 tensors. Queries and keys are strong enough that attention picks few keys, gains and averages differ
    from 1, the shift blends visibly."""
    g = torch.Generator().manual_seed(seed)

    def mat(*shape, gain=1.0):
        return torch.randn(*shape, generator=g) * (gain / math.sqrt(shape[-1]))

    def near(value, *shape, spread=0.2):
        return value + spread * torch.randn(shape, generator=g)

    W = c["width"]
    w = {"embed": torch.randn(c["vocab"], W, generator=g), "bigram": 0.7 * torch.randn(c["embedding"]["bigram"]["buckets"] + 1, W, generator=g),
         "final.norm": near(1.3), "head": mat(c["vocab"], W)}
    for i, la in enumerate(c["layers"]):
        p, m = f"l{i}.", la["mixer"]
        H, d, r, dv, kv = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        w.update({
            p + "norm1": near(0.9), p + "shift": torch.rand(W, generator=g), p + "dwa": near(0.4, i + 2),
            p + "mix.q": mat(H * (d + r), W, gain=2.0), p + "mix.dkv": mat(kv + r, W, gain=1.5), p + "mix.dkv.norm": near(1.0, kv),
            p + "mix.uk": mat(H * d, kv, gain=1.5), p + "mix.uv": mat(H * dv, kv), p + "mix.o": mat(W, H * dv),
        })
        f = la["mlp"]
        if f is not None:
            w[p + "mlp.router"] = mat(f["router"]["experts"], W, gain=2.0)
            for e in range(f["router"]["experts"]):
                w[f"{p}mlp.e{e}.up"] = mat(f["expert"]["ff"], W)
                w[f"{p}mlp.e{e}.down"] = mat(W, f["expert"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write_model(folder, c, w):
    """``config.json`` and ``model.safetensors`` (8-byte length, JSON header, data)."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(c))
    head, data = {}, b""
    for k, v in w.items():
        raw = v.contiguous().view(torch.int16).numpy().tobytes()
        head[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    blob = json.dumps(head).encode()
    blob += b" " * (-len(blob) % 8)
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(blob)) + blob + data)
