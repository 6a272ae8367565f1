"""Each mechanism of the sequential layers alone, against the plain oracle: norms between sublayers, rotation, grouped attention with
sink and gate, short convolution, state-space recurrence, gated norm. Attention inputs are made so that one key stands out:
seen, it decides the output; hidden, it leaves no trace. CPU restatement and, marked ``gpu``, the kernels in both precisions
and both variants."""
import math

import pytest
import torch

import pazenex_oracle as oracle
from keys_values_b200.kvcache.sequences import SequenceTable
from keys_values_b200.ops import layers as L

# (device, dtype, CUDA-core kernels forced)
VARIANTS = [
    ("cpu", torch.float32, False),
    pytest.param(("cuda", torch.float32, False), marks=pytest.mark.gpu),
    pytest.param(("cuda", torch.bfloat16, False), marks=pytest.mark.gpu),
    pytest.param(("cuda", torch.bfloat16, True), marks=pytest.mark.gpu),
]
variant_param = pytest.mark.parametrize("variant", VARIANTS)


@pytest.fixture
def env(variant, monkeypatch):
    device, dtype, simple = variant
    if device == "cuda":
        from keys_values_b200.ops import layers_cuda

        monkeypatch.setattr(layers_cuda, "FORCE_SIMPLE", simple)
    return torch.device(device), dtype


def close(got, want, dtype, scale=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-6)
    assert err < scale * (2e-5 if dtype == torch.float32 else 1.2e-2), err


def table(device, start, n_slots=None, slots=None):
    B = len(start)
    t = SequenceTable(n_slots or B, device)
    got = [t.acquire() for _ in range(t.n_slots)]
    t.set_batch(slots if slots is not None else got[:B])
    for s, n in zip(t.batch, start):
        t.pos[s] = n
        t.pos_host[s] = n
    return t


def move(tab, seq):
    """The pass is over: positions move on."""
    for s, n in zip(seq.slots_host, seq.count_host):
        tab.pos[s] += n
        tab.pos_host[s] += n


def padded(x, groups, n):
    """Last dimension as ``groups`` parts, each padded to ``n``."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    out = torch.zeros(*parts.shape[:-1], n)
    out[..., : parts.shape[-1]] = parts
    return out.reshape(*x.shape[:-1], groups * n)


def check(device):
    from keys_values_b200 import ops

    ops.check_status(device)


# ----------------------------------------------------------------------------------------------------- norms
@variant_param
@pytest.mark.parametrize("center", [True, False])
@pytest.mark.parametrize("width", [1, 7, 64, 250, 1028, 3072, 8200])
def test_norm_edge(env, width, center):
    """Every combination of what may be left out, with a mean far from zero and outputs that a norm scales up."""
    dev, dtype = env
    g = torch.Generator().manual_seed(width)
    n, vocab, eps = 5, 11, 1e-3
    x = (3 + torch.randn(n, width, generator=g)).double()
    sub = (0.05 * torch.randn(n, width, generator=g) + 0.2).to(dtype).double()
    after, before, step = (torch.randn(width, generator=g).double() for _ in range(3))
    embed = torch.randn(vocab, width, generator=g).to(dtype).double()
    idx = torch.randint(0, vocab, (n,), generator=g)

    def norm(rows, w):
        return torch.stack([(oracle.layer_norm if center else oracle.rms_norm)(r, w, eps) for r in rows])

    for use in ("x_in sub after before", "x_in sub after before embed step", "x_in sub", "embed step before", "embed", "x_in sub after", "x_in step before"):
        use = use.split()
        new = torch.zeros(n, width).double()
        if "x_in" in use:
            new = new + x
        if "sub" in use:
            new = new + (norm(sub, after) if "after" in use else sub)
        if "embed" in use:
            new = new + embed[idx]
        if "step" in use:
            new = new + step
        f32 = lambda t: t.float().to(dev)  # noqa: E731
        x_out = f32(x) if "x_in" in use else torch.empty(n, width, device=dev)
        h = torch.zeros(n, width, dtype=dtype, device=dev)
        L.norm_edge(x_out if "x_in" in use else None, sub.to(dev, dtype) if "sub" in use else None, f32(after) if "after" in use else None,
                    x_out, f32(before) if "before" in use else None, h, idx.to(dev) if "embed" in use else None,
                    embed.to(dev, dtype) if "embed" in use else None, f32(step) if "step" in use else None, eps, center)
        close(x_out, new, torch.float32)
        if "before" in use:
            close(h, norm(new, before), dtype)
    close(L.row_norm(f32(x), f32(after), eps, center, dtype), norm(x, after), dtype)
    check(dev)


@variant_param
def test_token_ids_are_checked(env):
    dev, dtype = env
    embed, x = torch.ones(4, 8, dtype=dtype, device=dev), torch.zeros(2, 8, device=dev)
    with pytest.raises((IndexError, RuntimeError)):
        L.norm_edge(None, None, None, x, None, None, torch.tensor([1, 4], device=dev), embed, None, 1e-5, True)
        check(dev)
    if dev.type == "cuda":  # the kernel took row 0 instead and the report is cleared
        check(dev)


@variant_param
def test_squared_relu(env):
    dev, dtype = env
    x = torch.linspace(-3, 3, 1003).to(dtype)
    close(L.activate(x.clone().to(dev), "relu_squared"), torch.clamp(x.double(), min=0) ** 2, dtype)
    assert L.activate(x, "none") is x


# ------------------------------------------------------------------------------------------ grouped attention
def shape_of(m, **kw):
    args = dict(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], rot_dims=m["rot"]["dims"], shared_value=True, gate=True,
                sink=True, scale=m["scale"])
    args.update(kw)
    return L.GroupedShape(**args)


def freqs(m):
    d = m["rot"]["dims"]
    return (m["rot"]["base"] ** (torch.arange(d // 2).double() * (-2.0 / max(d, 1))) / m["rot"].get("scaling", {}).get("factor", 1.0)).float()


ATTENTIONS = {
    "plain": oracle.attention_layer(heads=4, kv_heads=2, dim=32, dims=32, base=10000.0)["mixer"],
    "part": oracle.attention_layer(heads=6, kv_heads=3, dim=40, dims=16, base=77.0, factor=None)["mixer"],
    "odd": oracle.attention_layer(heads=3, kv_heads=1, dim=7, dims=4, factor=2.5)["mixer"],
    "wide": oracle.attention_layer(heads=20, kv_heads=1, dim=128, dims=128, scale=0.09)["mixer"],
    "deep": oracle.attention_layer(heads=2, kv_heads=1, dim=200, dims=100, scale=0.06)["mixer"],
    "unrotated": oracle.attention_layer(heads=2, kv_heads=2, dim=24, dims=0)["mixer"],
}


@variant_param
@pytest.mark.parametrize("name", list(ATTENTIONS))
def test_grouped_attention_matches_oracle(env, name):
    """The whole of prep and attention, in passes of several sizes and single tokens, two sequences in slots 2 and 0."""
    dev, dtype = env
    m, eps = ATTENTIONS[name], 1e-4
    s = shape_of(m)
    H, G, d = s.heads, s.kv_heads, s.dim
    g = torch.Generator().manual_seed(5)
    T, width = 140, 16
    h = torch.randn(2, T, width, generator=g)
    w = {"q": torch.randn(H * d, width, generator=g), "k": torch.randn(G * d, width, generator=g), "g": torch.randn(H * d, width, generator=g),
         "q.norm": 1 + 0.3 * torch.randn(H * d, generator=g), "k.norm": 1 + 0.3 * torch.randn(G * d, generator=g)}
    parts = [(h @ w[n].T).to(dtype) for n in ("q", "k", "g")]
    # the oracle starts from the same rounded projections
    eye = {"q": torch.eye(H * d), "k": torch.eye(G * d)}
    want = []
    for b in range(2):
        q = torch.stack([oracle.rms_norm(r, w["q.norm"].double(), eps) for r in parts[0][b].double()]).view(T, H, d)
        k, v = oracle.keys_and_values(parts[1][b].double(), {"k": eye["k"].double(), "k.norm": w["k.norm"].double()}, m, eps)
        heads = [oracle.sink_attention(torch.stack([oracle.rotate(q[t, n], t, m["rot"]) for t in range(T)]), k[:, n // (H // G)], v[:, n // (H // G)],
                                       m["scale"]) for n in range(H)]
        want.append(padded((torch.cat(heads, 1) * oracle.sigmoid(parts[2][b].double())).float(), H, s.vdp))
    want = torch.stack(want)
    qkv = torch.cat((padded(parts[0].float(), H, s.dimp), padded(parts[1].float(), G, s.dimp), padded(parts[2].float(), H, s.vdp)), -1).to(dev, dtype)
    nq, nk, fr = padded(w["q.norm"], H, s.dimp).to(dev), padded(w["k.norm"], G, s.dimp).to(dev), freqs(m).to(dev)
    tab = table(dev, [0, 0], 3, [2, 0])
    rows = torch.full((3, T + 3, G, s.dimp + s.vdp), 9.0, dtype=dtype, device=dev)  # what an earlier owner left
    at = [0, 0]
    for n, counts in ((37, [37, 20]), (1, [1, 1]), (1, [1, 1]), (95, [95, 64]), (2, [2, 2]), (1, [0, 1]), (4, [4, 4])):
        part = torch.zeros(2, n, qkv.shape[-1], dtype=dtype, device=dev)
        for b in range(2):
            part[b, : counts[b]] = qkv[b, at[b] : at[b] + counts[b]]
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        q = L.grouped_prep(part, nq, nk, fr, rows, seq, s, eps)
        out = L.grouped_attend(q, part, rows, seq, s)
        assert torch.isfinite(out).all()
        for b in range(2):
            if counts[b]:
                close(out[b, : counts[b]], want[b, at[b] : at[b] + counts[b]], dtype)
            at[b] += counts[b]
        move(tab, seq)
    assert torch.all(rows[1] == 9) and torch.all(rows[2, at[0] :] == 9)  # another sequence's slot, rows not reached
    check(dev)


@variant_param
@pytest.mark.parametrize("shared", [True, False])
def test_prep_without_norm_and_with_values_of_their_own(env, shared):
    dev, dtype = env
    m = ATTENTIONS["part"]
    s = shape_of(m, shared_value=shared, gate=False, vdim=m["vdim"] if shared else 24)
    g = torch.Generator().manual_seed(1)
    T = 5
    q, k = (torch.randn(1, T, n * s.dim, generator=g).to(dtype) for n in (s.heads, s.kv_heads))
    v = torch.randn(1, T, s.kv_heads * s.vdim, generator=g).to(dtype)
    cols = [padded(q.float(), s.heads, s.dimp), padded(k.float(), s.kv_heads, s.dimp)] + ([] if shared else [padded(v.float(), s.kv_heads, s.vdp)])
    tab = table(dev, [1000])
    rows = torch.zeros(1, 1010, s.kv_heads, s.dimp + s.vdp, dtype=dtype, device=dev)
    seq = tab.begin(1, T)
    got = L.grouped_prep(torch.cat(cols, -1).to(dev, dtype), None, None, freqs(m).to(dev), rows, seq, s, 1e-5)
    for t in range(T):
        for n in range(s.heads):
            close(got[0, t, n, : s.dim], oracle.rotate(q[0, t].double().view(s.heads, -1)[n], 1000 + t, m["rot"]), dtype, 10)
        for n in range(s.kv_heads):
            close(rows[0, 1000 + t, n, : s.dim], oracle.rotate(k[0, t].double().view(s.kv_heads, -1)[n], 1000 + t, m["rot"]), dtype, 10)
    want = (k if shared else v).float().view(T, s.kv_heads, s.vdim)
    assert torch.equal(rows[0, 1000:1005, :, s.dimp : s.dimp + s.vdim].float().cpu(), want)


@variant_param
@pytest.mark.parametrize("n_keys", [1, 15, 16, 17, 63, 64, 65, 127, 128, 129, 1023, 1025])
def test_one_key_stands_out(env, n_keys):
    """Keys at the borders of tiles and splits: the first, the last visible one and the first hidden one, for a single token and
    for the first and last query of a pass; scores far below the sink, too."""
    dev, dtype = env
    s = L.GroupedShape(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=0, shared_value=True, gate=False, sink=True, scale=0.5)
    pos = n_keys - 1
    length = n_keys + 9
    for T in (1, 2, 9):
        for marked in sorted({0, n_keys // 2, pos, pos + 1, pos + T - 1, pos + T}):
            if marked >= length:
                continue
            rows = torch.zeros(1, length, 1, 32, dtype=dtype, device=dev)
            rows[..., :16] = -1.0           # scores of −8 · 4: they leave almost everything to the sink
            rows[..., 16:] = 100.0
            rows[0, marked, 0, :16] = 1.0
            rows[0, marked, 0, 16:] = torch.arange(16.0)
            q = torch.full((1, T, 2, 16), 4.0, dtype=dtype, device=dev)
            seq = table(dev, [pos]).begin(1, T)
            out = L.grouped_attend(q, torch.zeros(1, T, 8, dtype=dtype, device=dev), rows, seq, s).view(T, 2, 16)
            for t in range(T):
                want = torch.arange(16.0) if marked <= pos + t else torch.zeros(16)
                assert torch.allclose(out[t].float().cpu(), want.expand(2, 16), atol=0.02, rtol=0.01), (T, marked, t)
    check(dev)


@variant_param
@pytest.mark.parametrize("sink", [True, False])
def test_sink_takes_its_share(env, sink):
    """All scores equal: with the sink every key has 1 / (n + e^-s), whatever the sign and size of s."""
    dev, dtype = env
    s = L.GroupedShape(heads=4, kv_heads=2, dim=8, vdim=8, rot_dims=0, shared_value=True, gate=False, sink=sink, scale=1.0)
    for score in (-60.0, -3.0, 0.0, 2.5, 40.0):
        for n, T in ((1, 1), (5, 1), (200, 1), (5, 3), (300, 130)):
            rows = torch.zeros(1, n, 2, 16, dtype=dtype, device=dev)
            rows[..., 0], rows[..., 8:] = 1.0, 1.0
            q = torch.zeros(1, T, 4, 8, dtype=dtype, device=dev)
            q[..., 0] = score
            seq = table(dev, [n - T]).begin(1, T)
            out = L.grouped_attend(q, torch.zeros(1, T, 8, dtype=dtype, device=dev), rows, seq, s).view(T, 32).float().cpu()
            for t in range(T):
                seen = n - T + t + 1
                want = 1.0 if not sink else seen / (seen + math.exp(-score))
                assert torch.allclose(out[t], torch.full((32,), want), rtol=1e-2, atol=1e-30), (score, n, T, t)
    check(dev)


# --------------------------------------------------------------------------------------- state-space recurrence
MIXERS = {
    "plain": L.StateShape(heads=4, vdim=24, state=16, groups=2, norm_groups=4, taps=4),
    "odd": L.StateShape(heads=3, vdim=5, state=11, groups=3, norm_groups=5, taps=6),
    "one": L.StateShape(heads=1, vdim=8, state=1, groups=1, norm_groups=1, taps=1),
    "usual": L.StateShape(heads=4, vdim=64, state=128, groups=2, norm_groups=2, taps=4),
    "uneven": L.StateShape(heads=3, vdim=48, state=72, groups=1, norm_groups=2, taps=2),
    "wide": L.StateShape(heads=2, vdim=128, state=96, groups=1, norm_groups=1, taps=4),
    "large": L.StateShape(heads=2, vdim=160, state=200, groups=1, norm_groups=16, taps=3),
}
PASSES = [(33, [33, 20]), (1, [1, 1]), (2, [2, 2]), (1, [0, 1]), (130, [100, 130]), (1, [1, 1]), (257, [257, 250])]


def projection(s, T, seed, dtype, dt_mean=-1.0):
    """Random columns ``z | x | B | C | dt`` (unpadded, rounded) of two sequences."""
    g = torch.Generator().manual_seed(seed)
    inner, bc = s.heads * s.vdim, s.groups * s.state
    z, x = torch.randn(2, T, inner, generator=g), torch.randn(2, T, inner, generator=g)
    b, c = (torch.randn(2, T, bc, generator=g) for _ in range(2))
    dt = dt_mean + torch.randn(2, T, s.heads, generator=g)
    return [t.to(dtype).float() for t in (z, x, b, c, dt)]


def joint(s, cols, dtype, device):
    z, x, b, c, dt = cols
    u = torch.cat((padded(z, s.heads, s.vdp), padded(x, s.heads, s.vdp), padded(b, s.groups, s.np), padded(c, s.groups, s.np), dt), -1)
    return torch.nn.functional.pad(u, (0, s.ld - u.shape[-1])).to(device, dtype)


def channels(s, x, b, c):
    return torch.cat((padded(x, s.heads, s.vdp), padded(b, s.groups, s.np), padded(c, s.groups, s.np)), -1)


def part_of(u, at, n, counts):
    out = torch.zeros(2, n, u.shape[-1], dtype=u.dtype, device=u.device)
    for b in range(2):
        out[b, : counts[b]] = u[b, at[b] : at[b] + counts[b]]
    return out


@variant_param
@pytest.mark.parametrize("name", list(MIXERS))
def test_short_conv(env, name):
    dev, dtype = env
    s = MIXERS[name]
    T = max(sum(c[b] for _, c in PASSES) for b in range(2))
    z, x, b, c, dt = cols = projection(s, T, 3, dtype)
    g = torch.Generator().manual_seed(4)
    n_ch = s.heads * s.vdim + 2 * s.groups * s.state
    w, bias = torch.randn(n_ch, s.taps, generator=g), torch.randn(n_ch, generator=g)
    inner, bc = s.heads * s.vdim, s.groups * s.state
    want = [oracle.short_conv(torch.cat((x, b, c), -1)[i].double(), w.double(), bias.double()).float() for i in range(2)]
    want = [channels(s, *torch.split(t, [inner, bc, bc], -1)) for t in want]
    wp = channels(s, *torch.split(w.t(), [inner, bc, bc], -1)).contiguous().to(dev)
    bp = channels(s, *torch.split(bias, [inner, bc, bc], -1)).contiguous().to(dev)
    u = joint(s, cols, dtype, dev)
    ring = torch.full((3, s.taps, s.channels), 5.0, dtype=dtype, device=dev)
    tab, at = table(dev, [0, 0], 3, [2, 0]), [0, 0]
    for n, counts in PASSES + [(2, [2, 2])] * 3:
        counts = [min(k, T - a) for k, a in zip(counts, at)]
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        out = L.short_conv(part_of(u, at, n, counts), s.inner, wp, bp, ring, seq)
        for i in range(2):
            if counts[i]:
                close(out[i, : counts[i]], want[i][at[i] : at[i] + counts[i]], dtype)
            at[i] += counts[i]
        move(tab, seq)
    assert torch.all(ring[1] == 5)
    check(dev)


def scan_truth(s, x, b, c, dt, dt_bias, a_log, skip):
    """``y (2, T, inner)`` and states after every token asked for, in float64."""
    ys, states = [], []
    for i in range(2):
        heads, last = [], []
        for n in range(s.heads):
            k = n // (s.heads // s.groups)
            y, S = oracle.state_space(x[i, :, n * s.vdim : (n + 1) * s.vdim].double(), b[i, :, k * s.state : (k + 1) * s.state].double(),
                                      c[i, :, k * s.state : (k + 1) * s.state].double(), oracle.softplus(dt[i, :, n].double() + float(dt_bias[n])),
                                      float(a_log[n]), float(skip[n]))
            heads.append(y)
            last.append(S)
        ys.append(padded(torch.cat(heads, 1).float(), s.heads, s.vdp))
        states.append(torch.stack(last))
    return ys, states


@variant_param
@pytest.mark.parametrize("rates", ["mixed", "slow", "fast"])
@pytest.mark.parametrize("name", list(MIXERS))
def test_state_scan(env, name, rates):
    """Passes of several sizes with the state carried between them. Slow decays keep the first token for hundreds; fast ones
    underflow within a chunk."""
    dev, dtype = env
    s = MIXERS[name]
    passes = PASSES + [(2, [2, 2])]
    T = [sum(c[b] for _, c in passes) for b in range(2)]
    z, x, b, c, dt = cols = projection(s, max(T), 6, dtype)
    if rates == "slow":
        x[:, 0], b[:, 0] = 40.0, 1.0
    g = torch.Generator().manual_seed(7)
    dt_bias, skip = 0.5 * torch.randn(s.heads, generator=g), torch.randn(s.heads, generator=g)
    a_log = {"mixed": -1.0, "slow": -7.0, "fast": 4.0}[rates] + torch.randn(s.heads, generator=g)
    want, last = [], []
    for i in range(2):
        cut = [t[:, : T[i]] for t in (x, b, c, dt)]
        y, S = scan_truth(s, *cut, dt_bias, a_log, skip)
        want.append(y[i])
        last.append(S[i])
    u, xbc = joint(s, cols, dtype, dev), channels(s, x, b, c).to(dev, dtype)
    state = torch.full((3, s.heads, s.np, s.vdp), 50.0, device=dev)  # what an earlier owner left
    tab, at = table(dev, [0, 0], 3, [2, 0]), [0, 0]
    for n, counts in passes:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        y = L.state_scan(part_of(u, at, n, counts), part_of(xbc, at, n, counts), dt_bias.to(dev), a_log.to(dev), skip.to(dev), state, seq, s)
        for i in range(2):
            if counts[i]:
                got, ref = y[i, : counts[i]].double().cpu(), want[i][at[i] : at[i] + counts[i]].double()
                scale = float(want[i].abs().max())
                assert float((got - ref).abs().max()) < scale * (2e-5 if dtype == torch.float32 else 4e-3), (n, i)
            assert torch.all(y[i, counts[i] :] == 0)
            at[i] += counts[i]
        move(tab, seq)
    for slot, S in zip((2, 0), last):
        got = state[slot, :, : s.state, : s.vdim].double().cpu()
        # the state is fp32 in both precisions: products of rounded inputs, summed without further rounding to 16 bits
        assert float((got - S).abs().max()) < float(S.abs().max()) * 5e-5
        assert torch.all(state[slot, :, s.state :] == 0) and torch.all(state[slot, :, :, s.vdim :] == 0)
    assert torch.all(state[1] == 50)
    check(dev)


@variant_param
@pytest.mark.parametrize("name", list(MIXERS))
def test_state_step(env, name):
    """Token by token from the first on, then after a prompt, against convolution and recurrence over the whole; rows
    without a token keep everything."""
    dev, dtype = env
    s = MIXERS[name]
    T, first = 23, 9
    z, x, b, c, dt = cols = projection(s, T, 8, dtype)
    g = torch.Generator().manual_seed(9)
    inner, bc = s.heads * s.vdim, s.groups * s.state
    w, bias = torch.randn(inner + 2 * bc, s.taps, generator=g), torch.randn(inner + 2 * bc, generator=g)
    dt_bias, skip, a_log = 0.5 * torch.randn(s.heads, generator=g), torch.randn(s.heads, generator=g), -1 + torch.randn(s.heads, generator=g)
    conv = torch.stack([oracle.short_conv(torch.cat((x, b, c), -1)[i].double(), w.double(), bias.double()) for i in range(2)])
    want, _ = scan_truth(s, *torch.split(conv, [inner, bc, bc], -1), dt, dt_bias, a_log, skip)
    wp = channels(s, *torch.split(w.t(), [inner, bc, bc], -1)).contiguous().to(dev)
    bp = channels(s, *torch.split(bias, [inner, bc, bc], -1)).contiguous().to(dev)
    u = joint(s, cols, dtype, dev)
    vec = [t.to(dev) for t in (dt_bias, a_log, skip)]
    for prompt in (0, first):
        ring = torch.full((3, s.taps, s.channels), 5.0, dtype=dtype, device=dev)
        state = torch.full((3, s.heads, s.np, s.vdp), 50.0, device=dev)
        tab, at = table(dev, [0, 0], 3, [2, 0]), [0, 0]
        if prompt:
            seq = tab.begin(2, prompt, [prompt, prompt - 2])
            seq.start = seq.start.clone()
            part = part_of(u, at, prompt, seq.count_host)
            xbc = L.short_conv(part, s.inner, wp, bp, ring, seq)
            L.state_scan(part, xbc, *vec, state, seq, s)
            at = list(seq.count_host)
            move(tab, seq)
        while at[0] < T:
            counts = [1, 0 if at[0] in (4, 15) else 1]
            seq = tab.begin(2, 1, counts)
            seq.start = seq.start.clone()
            y = L.state_step(part_of(u, at, 1, counts), wp, bp, *vec, ring, state, seq, s)
            for i in range(2):
                if counts[i]:
                    scale = float(want[i].abs().max())
                    err = float((y[i, 0].double().cpu() - want[i][at[i]].double()).abs().max())
                    assert err < scale * (2e-5 if dtype == torch.float32 else 8e-3), (prompt, at, i, err / scale)
                else:
                    assert torch.all(y[i] == 0)
                at[i] += counts[i]
            move(tab, seq)
        assert torch.all(ring[1] == 5) and torch.all(state[1] == 50)
    check(dev)


@variant_param
@pytest.mark.parametrize("name", list(MIXERS))
def test_gated_group_norm(env, name):
    dev, dtype = env
    s, eps, T = MIXERS[name], 1e-3, 5
    z, x, b, c, dt = cols = projection(s, T, 11, dtype)
    y = (torch.randn(2, T, s.heads * s.vdim, generator=torch.Generator().manual_seed(12)) * torch.logspace(-2, 1, s.heads * s.vdim)).to(dtype).float()
    w = 1 + 0.3 * torch.randn(s.heads * s.vdim, generator=torch.Generator().manual_seed(13))
    want = torch.stack([oracle.gated_group_norm(y[i].double(), z[i].double(), w.double(), s.norm_groups, eps) for i in range(2)])
    got = L.gated_group_norm(padded(y, s.heads, s.vdp).to(dev, dtype), joint(s, cols, dtype, dev), padded(w, s.heads, s.vdp).to(dev), s, eps)
    close(got, padded(want.float(), s.heads, s.vdp), dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["usual", "uneven", "wide"])
def test_state_scan_in_segments(name):
    """Few heads and many tokens: the pass is cut into segments that run side by side. Against the token-by-token kernel."""
    from keys_values_b200.ops import layers_cuda as LC

    s = MIXERS[name]
    T, counts = 3100, [3100, 700]
    cols = projection(s, T, 21, torch.bfloat16)
    g = torch.Generator().manual_seed(22)
    vec = [t.cuda() for t in (0.5 * torch.randn(s.heads, generator=g), -4 + torch.randn(s.heads, generator=g), torch.randn(s.heads, generator=g))]
    u, xbc = joint(s, cols, torch.bfloat16, "cuda"), channels(s, *cols[1:4]).to("cuda", torch.bfloat16)
    assert LC.lib().kvb_state_scan_tc_scratch_bytes(2, T, s.heads, s.groups, s.vdp, s.np) > 0
    for start in (0, 5):
        ys, states = [], []
        for dtype in (torch.float32, torch.bfloat16):
            state = torch.linspace(-20, 20, s.heads * s.np * s.vdp, device="cuda").view(1, s.heads, s.np, s.vdp).repeat(2, 1, 1, 1)
            state[:, :, s.state :] = 0
            state[:, :, :, s.vdim :] = 0
            seq = table("cuda", [start, start]).begin(2, T, counts)
            seq.start = seq.start.clone()
            ys.append(L.state_scan(u.to(dtype), xbc.to(dtype), *vec, state, seq, s))
            states.append(state)
        for b, n in enumerate(counts):
            want = ys[0][b, :n].double()
            assert float((ys[1][b, :n].double() - want).abs().max()) < 4e-3 * float(want.abs().max())
            assert torch.all(ys[1][b, n:] == 0)
        assert float((states[1] - states[0]).abs().max()) < 5e-5 * float(states[0].abs().max())
    check("cuda")
