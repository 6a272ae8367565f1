"""Each mechanism of the Ladadra design alone, against the plain oracle: norms after the sublayers, gated units, routing in groups, banded
rotation, chunked and windowed attention with kept tokens, soft cap, learned sink, gate per head, differential maps, rows in a ring,
retention. Attention inputs are made so that one key stands out: seen, it decides the output; hidden, it leaves no trace. CPU
restatement and, marked ``gpu``, the kernels in both precisions and both variants."""
import math

import pytest
import torch

import ladadra_oracle as oracle
from keys_values_b200.models.grouped_attention import grouped_shape, rotation_frequencies
from keys_values_b200.ops import layers as L
from test_pazenex_mechanisms import check, close, env, move, padded, part_of, table, variant_param  # noqa: F401 (env is a fixture)


# ------------------------------------------------------------------------------------- norms, gated units, experts
@variant_param
@pytest.mark.parametrize("width", [1, 7, 64, 250, 2048])
def test_norm_of_sublayer_with_experts(env, width):
    """Weighted expert rows with and without a shared output, and the stream itself as the next input."""
    dev, dtype = env
    g = torch.Generator().manual_seed(width)
    n, top, eps = 6, 3, 1e-3
    ld = L.round8(width)
    x, sub = torch.randn(n, width, generator=g).double(), torch.randn(n, width, generator=g).to(dtype).double()
    out = torch.randn(n * top, ld, generator=g).to(dtype)
    row = torch.randperm(n * top, generator=g).int().view(n, top)
    weight = torch.rand(n, top, generator=g)
    after = torch.randn(width, generator=g).double()
    routed = (weight.double()[:, :, None] * out.double()[row.long()][:, :, :width]).sum(1)
    experts = (out.to(dev), row.to(dev), weight.to(dev))
    for shared in (True, False):
        for normed in (True, False):
            y = routed + (sub if shared else 0)
            want = x + (torch.stack([oracle.rms_norm(r, after, eps) for r in y]) if normed else y)
            stream, h = x.float().to(dev), torch.zeros(n, width, dtype=dtype, device=dev)
            L.norm_edge(stream, sub.to(dev, dtype) if shared else None, after.float().to(dev) if normed else None, stream, None, h, None, None, None,
                        eps, False, experts)
            close(stream, want, torch.float32)
            close(h, want, dtype)
    check(dev)


@variant_param
@pytest.mark.parametrize("ff", [1, 8, 13, 200])
def test_gated_unit(env, ff):
    dev, dtype = env
    g = torch.Generator().manual_seed(ff)
    gate, up = (3 * torch.randn(5, ff, generator=g)).to(dtype), torch.randn(5, ff, generator=g).to(dtype)
    n = L.round8(ff)
    x = torch.cat((padded(gate.float(), 1, n), padded(up.float(), 1, n)), -1).to(dev, dtype)
    got = L.glu(x, ff)
    assert got.shape == (5, n) and not got[:, ff:].any()
    close(got[:, :ff], oracle.silu(gate.double()) * up.double(), dtype)


ROUTERS = [(10, 3, (5, 2)), (12, 4, (4, 4)), (8, 1, (8, 1)), (9, 2, (3, 1)), (70, 8, (7, 3)), (6, 6, (2, 2)), (40, 5, None), (1, 1, None)]


@variant_param
@pytest.mark.parametrize("E,top,groups", ROUTERS)
def test_choice_of_experts(env, E, top, groups):
    """The chosen ones and their weights, with corrections that make most choice scores negative: those of other groups must stay out
    all the same, and the weights know nothing of the correction."""
    dev, dtype = env
    g = torch.Generator().manual_seed(E)
    n, width, ff = 33, 8, 8
    logits = 2 * torch.randn(n, E, generator=g)
    correction = -1.5 + 0.8 * torch.randn(E, generator=g)
    # expert e returns e in coordinate 0, whatever the token
    up, down = torch.zeros(E, 2 * ff, width), torch.zeros(E, width, ff)
    up[:, :2, 0] = 2.0
    down[:, 0, 0] = torch.arange(E).float()
    rule = L.RouterRule(score="sigmoid", groups=groups[0] if groups else 1, keep=groups[1] if groups else 1, renormalize=True, eps=1e-20)
    h = torch.ones(n, width)
    out, row, weight = L.routed_experts(h.to(dev, dtype), logits.to(dev), up.to(dev, dtype), down.to(dev, dtype), top, "silu_gated", rule, ff, width,
                                        correction.to(dev))
    unit = float(oracle.silu(torch.tensor(2.0, dtype=torch.float64))) * 2
    chosen = (out.float().cpu()[row.long().cpu()][:, :, 0] / unit).round().long()
    for t in range(n):
        s = oracle.sigmoid(logits[t].double())
        want = oracle.choose(s, correction.double(), top, None if not groups else dict(count=groups[0], keep=groups[1]))
        assert sorted(chosen[t].tolist()) == sorted(want)
        total = sum(float(s[e]) for e in want)
        close(weight[t], torch.tensor([float(s[e]) / total for e in chosen[t]]), torch.float32)
    check(dev)


@variant_param
@pytest.mark.parametrize("n,E,top,width,ff", [(1, 5, 2, 24, 20), (7, 4, 3, 33, 13), (90, 6, 2, 64, 65), (300, 3, 1, 40, 136)])
def test_gated_experts(env, n, E, top, width, ff):
    dev, dtype = env
    g = torch.Generator().manual_seed(n)
    w = {"router": torch.randn(E, width, generator=g).double(), "correction": 0.3 * torch.randn(E, generator=g).double()}
    for e in range(E):
        for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            w[f"e{e}.{name}"] = (torch.randn(*shape, generator=g) / shape[1] ** 0.5).to(dtype).double()
    h = torch.randn(n, width, generator=g).to(dtype)
    want = oracle.experts(h.double(), w, {"router": {"experts": E, "top": top}})
    logits = (h.double() @ w["router"].T).float()
    pairs = torch.stack([torch.stack((w[f"e{e}.gate"], w[f"e{e}.up"]), 1).reshape(2 * ff, width) for e in range(E)])
    up, down = padded(pairs.float(), 1, L.round8(width)), padded(torch.stack([w[f"e{e}.down"] for e in range(E)]).float(), 1, L.round8(ff))
    out, row, weight = L.routed_experts(h.to(dev), logits.to(dev), up.to(dev, dtype), down.to(dev, dtype), top, "silu_gated",
                                        L.RouterRule("sigmoid", renormalize=True, eps=1e-20), ff, width, w["correction"].float().to(dev))
    got = (weight.cpu().double()[:, :, None] * out.cpu().double()[row.cpu().long()][:, :, :width]).sum(1)
    close(got, want, dtype)
    check(dev)


# --------------------------------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 64), (8.0, 2.0, 3.0, 500), (1.0, 1.0, 2.0, 10), (3.0, 1.0, 1000.0, 100)])
def test_banded_frequencies(scaling):
    """Pairs of all three bands: kept, stretched, blended."""
    m = oracle.attention_layer(dim=48, dims=40, base=3000.0, scaling=scaling)["mixer"]
    spec = dict(rope_base=3000.0, rope_dims=40, rope_bands=None if not scaling else dict(zip(("factor", "low", "high", "original"), scaling)))
    want = torch.tensor(oracle.frequencies(m["rot"]), dtype=torch.float64)
    assert torch.allclose(rotation_frequencies(spec), want, rtol=1e-12)
    if scaling and scaling[0] == 4.0:
        plain = torch.tensor(oracle.frequencies({"base": 3000.0, "dims": 40}), dtype=torch.float64)
        ratio = want / plain
        assert ((ratio - 1).abs() < 1e-12).any() and ((ratio - 0.25).abs() < 1e-12).any() and ((ratio > 0.26) & (ratio < 0.99)).any()


# ------------------------------------------------------------------------------------------------- attention
def spec_of(m, **kw):
    """Description of a mixer of the oracle in the package's terms."""
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    spec = dict(n_head=m["heads"], n_kv_head=m["kv_heads"], dim=m["dim"], v_dim=m["vdim"], scale=m["scale"])
    if "diff" in m:
        spec.update(qk_norm="head", window=mask.get("size"), keep_first=mask.get("keep_first"), differential=m["diff"])
    else:
        spec.update(qk_norm=True, rope_base=rot["base"], rope_dims=rot["dims"], softcap=m.get("softcap"), chunk=mask.get("size"), sink="learned",
                    gate="head")
        if "scaling" in rot:
            spec["rope_bands"] = rot["scaling"]
    spec.update(kw)
    return spec


A, D = oracle.attention_layer, oracle.differential_layer
ATTENTIONS = {
    "chunked": A(heads=4, kv_heads=2, dim=32, vdim=24, dims=32, size=50)["mixer"],
    "small chunks": A(heads=6, kv_heads=3, dim=40, vdim=64, dims=16, base=77.0, scaling=None, size=7)["mixer"],
    "one chunk": A(heads=20, kv_heads=1, dim=128, vdim=72, dims=64, scale=0.09, size=None, cap=None)["mixer"],
    "chunk of a tile": A(heads=2, kv_heads=1, dim=72, vdim=136, dims=8, scale=0.1, size=64, cap=1.5)["mixer"],
    "odd": A(heads=3, kv_heads=1, dim=7, vdim=5, dims=4, size=33)["mixer"],
    "deep": A(heads=2, kv_heads=1, dim=200, vdim=160, dims=100, scale=0.06, size=100)["mixer"],
    "differential": D(heads=4, kv_heads=2, dim=24, vdim=48, size=30, keep_first=5)["mixer"],
    "differential, wide": D(heads=9, kv_heads=1, dim=64, vdim=128, scale=0.12, size=70, keep_first=66, diff=0.8)["mixer"],
    "differential, one key": D(heads=2, kv_heads=2, dim=128, vdim=40, scale=0.08, size=1, keep_first=1)["mixer"],
    "differential, odd": D(heads=3, kv_heads=3, dim=9, vdim=11, size=40, keep_first=0)["mixer"],
    "differential, open": D(heads=4, kv_heads=1, dim=72, vdim=100, scale=0.1, size=None, diff=0.2)["mixer"],
    "differential, deep": D(heads=2, kv_heads=1, dim=136, vdim=144, scale=0.08, size=60, keep_first=20)["mixer"],
}
PASSES = [(37, [37, 20]), (1, [1, 1]), (1, [1, 1]), (95, [95, 64]), (2, [2, 2]), (1, [0, 1]), (4, [4, 4])]


def attention_case(name, dtype, T=140):
    """Joint projection of two sequences, packed norms and the oracle's result per head (gated, before the output projection)."""
    m, eps = ATTENTIONS[name], 1e-4
    s = grouped_shape(spec_of(m))
    H, G, d, P = s.heads, s.kv_heads, s.dim, s.vdim
    g = torch.Generator().manual_seed(len(name))
    parts = [torch.randn(2, T, n, generator=g).to(dtype) for n in (H * s.maps * d, G * s.maps * d, G * P, H)]
    if s.maps == 2:
        nq, nk = (1 + 0.3 * torch.randn(d, generator=g) for _ in range(2))
        lam = 0.6
        s = L.GroupedShape(**{**s.__dict__, "lam": lam, "eps": eps})
    else:
        nq, nk = (1 + 0.3 * torch.randn(n * d, generator=g) for n in (H, G))
    sink = torch.linspace(-2, 3, H) if s.sink else None
    mask = m.get("mask") or {}
    want = []
    for b in range(2):
        q, k, v, gate = (p[b].double() for p in parts)
        v = v.view(T, G, P)
        norm = lambda x, w: torch.stack([oracle.rms_norm(r, w.double(), eps) for r in x])  # noqa: E731
        heads = []
        if s.maps == 1:
            q, k = norm(q, nq).view(T, H, d), norm(k, nk).view(T, G, d)
            q, k = oracle.rotate_rows(q, m["rot"]), oracle.rotate_rows(k, m["rot"])
            sees = lambda i, j: oracle.sees_chunked(i, j, mask.get("size"))  # noqa: E731
            for n in range(H):
                y = oracle.attend(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], m["scale"], sees, m.get("softcap"), float(sink[n]))
                heads.append(y * oracle.sigmoid(gate[:, n : n + 1]))
        else:
            q, k = norm(q.view(-1, d), nq).view(T, H, 2, d), norm(k.view(-1, d), nk).view(T, G, 2, d)
            sees = lambda i, j: oracle.sees_window(i, j, mask.get("size"), mask.get("keep_first", 0))  # noqa: E731
            for n in range(H):
                a = [oracle.attend(q[:, n, i], k[:, n // (H // G), i], v[:, n // (H // G)], m["scale"], sees) for i in range(2)]
                heads.append(oracle.difference(a[0], a[1], lam, m["diff"], eps))
        want.append(padded(torch.cat(heads, 1).float(), H, s.vdp))
    cols = [padded(parts[0].float(), H * s.maps, s.dimp), padded(parts[1].float(), G * s.maps, s.dimp), padded(parts[2].float(), G, s.vdp)]
    if s.gate:
        cols.append(parts[3].float())
    qkv = padded(torch.cat(cols, -1), 1, s.ld)
    pn = (lambda w, n: padded(w, 1, s.dimp)) if s.head_norm else (lambda w, n: padded(w, n, s.dimp))
    fr = torch.tensor(oracle.frequencies(m["rot"])).float() if "rot" in m else torch.empty(0)
    return s, qkv, pn(nq, H), pn(nk, G), fr, sink, torch.stack(want), eps


def run_passes(env, case, passes, plan=L.RowPlan(), length=None):
    """Outputs of two sequences in slots 2 and 0, pass by pass, and the rows they leave."""
    dev, dtype = env
    s, qkv, nq, nk, fr, sink, want, eps = case
    qkv, nq, nk, fr = qkv.to(dev, dtype), nq.to(dev), nk.to(dev), fr.to(dev)
    sink = None if sink is None else sink.to(dev)
    tab = table(dev, [0, 0], 3, [2, 0])
    rows = torch.full((3, length or qkv.shape[1] + 3, s.kv_heads, s.row), 9.0, dtype=dtype, device=dev)  # what an earlier owner left
    at, outs = [0, 0], [[], []]
    for n, counts in passes:
        part = part_of(qkv, at, n, counts)
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        q = L.grouped_prep(part, nq, nk, fr, rows, seq, s, eps, plan)
        out = L.grouped_attend(q, part, rows, seq, s, sink, plan)
        for b in range(2):
            outs[b].append(out[b, : counts[b]])
            at[b] += counts[b]
        move(tab, seq)
    check(dev)
    return [torch.cat(o) for o in outs], rows, at


@variant_param
@pytest.mark.parametrize("name", list(ATTENTIONS))
def test_attention_matches_oracle(env, name):
    """The whole of prep and attention, in passes of several sizes and single tokens."""
    case = attention_case(name, env[1])
    got, rows, at = run_passes(env, case, PASSES)
    for b in range(2):
        assert torch.isfinite(got[b]).all()
        close(got[b], case[6][b, : at[b]], env[1], 4.0 if case[0].maps == 2 else 1.5)
    assert torch.all(rows[1] == 9) and torch.all(rows[2, at[0] :] == 9)  # another sequence's slot, rows not reached


@variant_param
@pytest.mark.parametrize("name", ["chunked", "differential", "differential, wide"])
def test_rows_in_a_ring(env, name):
    """Bounded layers over far more positions than rows: the same results as with a row per position, while rows are used again in the
    middle of passes and by single tokens."""
    case = attention_case(name, env[1], T=140)
    s, qkv = case[0], case[1]
    long = qkv.repeat(1, 9, 1) * torch.linspace(0.6, 1.4, 9).repeat_interleave(140)[None, :, None]
    case = (s, long, *case[2:])
    passes = [(150, [150, 93]), (1, [1, 1]), (170, [170, 170]), (1, [1, 1]), (2, [2, 2])] + [(180, [180, 171])] * 4 + [(1, [1, 1])] * 5 + [(100, [100, 100])]
    plain, _, _ = run_passes(env, case, passes)
    plan = L.RowPlan(128 if s.keep else 0, 256)
    assert max(n for n, _ in passes) <= plan.ring - s.span
    ring, rows, _ = run_passes(env, case, passes, plan, sum(plan))
    for b in range(2):
        if env[0].type == "cuda":  # the same tiles in the same order
            assert torch.equal(plain[b], ring[b])
        else:
            close(ring[b], plain[b], torch.float32)


def standing(window=0, keep=0, chunk=0, **kw):
    return L.GroupedShape(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=0, shared_value=False, gate=False, sink=False, scale=0.5, window=window,
                          keep=keep, chunk=chunk, **kw)


EDGES = [dict(window=1), dict(window=2, keep=1), dict(window=63, keep=3), dict(window=64, keep=64), dict(window=65, keep=65), dict(window=128, keep=100),
         dict(window=129, keep=200), dict(window=30, keep=128), dict(window=200, keep=130), dict(chunk=1), dict(chunk=5), dict(chunk=64), dict(chunk=100),
         dict(chunk=128), dict(chunk=300)]


@variant_param
@pytest.mark.parametrize("edge", EDGES, ids=str)
def test_one_key_stands_out(env, edge):
    """Keys just inside and just outside every window, chunk and stretch of kept tokens, far ones and the last one: for single tokens
    and for the first, a middle and the last query of passes, at positions around the borders of tiles, windows and chunks."""
    dev, dtype = env
    s = standing(**edge)
    span, keep = s.span, s.keep
    sees = (lambda i, j: oracle.sees_chunked(i, j, s.chunk)) if s.chunk else (lambda i, j: oracle.sees_window(i, j, s.window, keep))
    base = (torch.arange(16.0) + 1).to(dtype).float()
    starts = sorted({0, span - 1, span, span + keep, 2 * span - 1, 2 * span, 127, 128, 200, 385} - {-1})
    # values are 0.5 everywhere; the marked key's score stands so far above the others' that it takes all weight
    for start in starts:
        for T in (1, 2, 140):
            if T == 140 and start not in (0, span, 200):
                continue
            length = start + T
            queries = sorted({0, T // 2, T - 1})
            marks = set()
            for t in queries:
                i = start + t
                marks |= {0, keep - 1, keep, i, i - 1, i - span, i - span + 1, i // span * span - 1, i // span * span}
            marks = sorted(j for j in marks if 0 <= j < length)
            # all marks of this case side by side, one sequence each
            B = len(marks)
            rows = torch.zeros(B, length + 2, 1, s.row, dtype=dtype, device=dev)
            rows[..., :16] = -1.0
            rows[..., 16:] = 0.5
            for b, j in enumerate(marks):
                rows[b, j, 0, :16] = 1.0
                rows[b, j, 0, 16:] = base.to(dtype)
            q = torch.full((B, T, 2, 16), 4.0, dtype=dtype, device=dev)
            seq = table(dev, [start] * B).begin(B, T)
            out = L.grouped_attend(q, torch.zeros(B, T, 8, dtype=dtype, device=dev), rows, seq, s).view(B, T, 2, 16).float().cpu()
            for b, j in enumerate(marks):
                for t in queries:
                    want = base if sees(start + t, j) else torch.full((16,), 0.5)
                    assert torch.allclose(out[b, t], want.expand(2, 16), atol=0.01, rtol=0.01), (edge, start, T, t, j)
    check(dev)


@variant_param
@pytest.mark.parametrize("n", [3, 150, 700])
def test_maps_see_their_own_keys(env, n):
    """Two heads whose maps each look for another key: the result is value 1 less lambda times value 2, normed; with lambda and the
    factor behind the norm changed."""
    dev, dtype = env
    j1, j2 = 1, n - 2
    values = torch.zeros(n, 32)
    values[j1, :16], values[j2, 8:] = 2.0, 3.0
    for lam, post in ((0.5, 1.0), (-0.4, 0.3), (1.7, 0.9)):
        s = L.GroupedShape(heads=2, kv_heads=1, dim=16, vdim=32, rot_dims=0, shared_value=False, gate=False, sink=False, scale=1.0, maps=2,
                           lam=lam, post=post, eps=1e-3)
        rows = torch.zeros(1, n, 1, s.row, dtype=dtype, device=dev)
        rows[0, j1, 0, 0] = rows[0, j2, 0, 16 + 1] = 4.0
        rows[0, :, 0, 32:] = values.to(dev, dtype)
        q = torch.zeros(1, 2, 4, 16, dtype=dtype, device=dev)
        q[:, :, 0::2, 0] = q[:, :, 1::2, 1] = 8.0
        for T in (1, 2):
            seq = table(dev, [n - T]).begin(1, T)
            out = L.grouped_attend(q[:, :T].contiguous(), torch.zeros(1, T, 8, dtype=dtype, device=dev), rows, seq, s).view(T, 2, 32)
            o = values[j1] - lam * values[j2]
            want = (o / torch.sqrt(o.square().mean() + 1e-3) * post).double()
            for h in range(2):
                close(out[-1, h], want, dtype)
    check(dev)


@variant_param
@pytest.mark.parametrize("cap", [0.5, 5.0, 50.0, 1e5])
def test_soft_cap(env, cap):
    """Scores from far below to far above the cap; the weights show every one of them."""
    dev, dtype = env
    s = standing(softcap=cap)
    n = 200
    scores = torch.linspace(-2, 2, n) * min(cap, 50.0)
    scores = torch.where(torch.arange(n) % 3 == 0, scores * 0.05, scores)
    k = (scores * 0.5).to(dtype)  # q 4, scale 0.5: score = 2 k
    rows = torch.zeros(1, n, 1, s.row, dtype=dtype, device=dev)
    rows[0, :, 0, 0] = k.to(dev)
    rows[0, :, 0, 16:] = torch.nn.functional.one_hot(torch.arange(n) % 16, 16).to(dev, dtype)
    for T in (1, 2, 130):
        q = torch.zeros(1, T, 2, 16, dtype=dtype, device=dev)
        q[..., 0] = 4.0
        seq = table(dev, [n - T]).begin(1, T)
        out = L.grouped_attend(q, torch.zeros(1, T, 8, dtype=dtype, device=dev), rows, seq, s).view(T, 2, 16)
        for t in (0, T - 1):
            seen = n - T + t + 1
            e = torch.tensor([math.exp(oracle.soft_cap(2 * float(x), cap)) for x in k[:seen].double()], dtype=torch.float64)
            want = torch.zeros(16, dtype=torch.float64).index_add(0, torch.arange(seen) % 16, e / e.sum())
            close(out[t], want.expand(2, 16), dtype)
    check(dev)


@variant_param
def test_sinks_of_their_own(env):
    """One key and a sink per head from far below to far above its score; not scaled, not capped, counted once."""
    dev, dtype = env
    sinks = torch.tensor([-80.0, -3.0, 0.0, 1.5, 30.0, 70.0])
    s = L.GroupedShape(heads=6, kv_heads=2, dim=8, vdim=8, rot_dims=0, shared_value=False, gate=False, sink=True, scale=0.5, softcap=20.0)
    for n, T in ((1, 1), (300, 1), (5, 3), (300, 130)):
        rows = torch.zeros(1, n, 2, 16, dtype=dtype, device=dev)
        rows[..., 0], rows[..., 8:] = 1.0, 1.0
        q = torch.zeros(1, T, 6, 8, dtype=dtype, device=dev)
        q[..., 0] = 4.0
        seq = table(dev, [n - T]).begin(1, T)
        out = L.grouped_attend(q, torch.zeros(1, T, 8, dtype=dtype, device=dev), rows, seq, s, sinks.to(dev)).view(T, 6, 8).float().cpu()
        score = oracle.soft_cap(2.0, 20.0)
        for t in (0, T - 1):
            seen = n - T + t + 1
            want = seen / (seen + torch.exp(sinks.double() - score))
            assert torch.allclose(out[t].double(), want[:, None].expand(6, 8), rtol=1e-2, atol=1e-30), (n, T, t)
    check(dev)


@variant_param
@pytest.mark.parametrize("per_head", [True, False])
def test_gate(env, per_head):
    dev, dtype = env
    s = L.GroupedShape(heads=3, kv_heads=1, dim=8, vdim=16, rot_dims=0, shared_value=False, gate=True, sink=False, scale=1.0, gate_per_head=per_head)
    g = torch.Generator().manual_seed(3)
    for T in (1, 5):
        qkv = torch.zeros(1, T, s.ld)
        gate = 2 * torch.randn(1, T, s.heads * s.gate_cols, generator=g).to(dtype).float()
        qkv[..., s.gate_col : s.gate_col + gate.shape[-1]] = gate
        rows = torch.ones(1, T, 1, s.row, dtype=dtype, device=dev)
        q = torch.ones(1, T, 3, 8, dtype=dtype, device=dev)
        out = L.grouped_attend(q, qkv.to(dev, dtype), rows, table(dev, [0]).begin(1, T), s).view(T, 3, 16)
        close(out, oracle.sigmoid(gate.double()).view(T, 3, -1).expand(T, 3, 16), dtype)


# ------------------------------------------------------------------------------------------------- retention
RETENTIONS = {
    "plain": (L.RetentionShape(heads=3, dim=16, vdim=24, rot_dims=12), [0.7, 0.96, 0.999]),
    "odd": (L.RetentionShape(heads=2, dim=7, vdim=5, rot_dims=4), [0.9, 0.5]),
    "extremes": (L.RetentionShape(heads=3, dim=64, vdim=64, rot_dims=64), [0.0, 1.0, 0.98]),
    "wide": (L.RetentionShape(heads=2, dim=128, vdim=128, rot_dims=128), [0.96875, 0.9995]),
    "uneven": (L.RetentionShape(heads=1, dim=40, vdim=104, rot_dims=0), [0.99]),
    "large": (L.RetentionShape(heads=1, dim=136, vdim=200, rot_dims=64), [0.97]),
    "single": (L.RetentionShape(heads=1, dim=1, vdim=1, rot_dims=0), [0.9]),
}
SCANS = [(33, [33, 20]), (1, [1, 1]), (2, [2, 2]), (1, [0, 1]), (130, [100, 130]), (1, [1, 1]), (257, [257, 250])]
ROT_BASE = 300.0


def retention_case(name, T, dtype, seed=7):
    """fp32 projections (values and gate rounded to ``dtype``) and the oracle's outputs before the norm and after norm and gate."""
    s, decay = RETENTIONS[name]
    g = torch.Generator().manual_seed(seed)
    q, k = (torch.randn(2, T, s.heads * s.dim, generator=g) for _ in range(2))
    v, z = (torch.randn(2, T, s.heads * s.vdim, generator=g).to(dtype).float() for _ in range(2))
    rot = {"base": ROT_BASE, "dims": s.rot_dims}
    raw, want = [], []
    for b in range(2):
        qh, kh = (oracle.rotate_rows(x[b].double().view(T, s.heads, s.dim), rot) for x in (q, k))
        vh = v[b].double().view(T, s.heads, s.vdim)
        o = [oracle.retain(qh[:, n], kh[:, n] * s.dim**-0.5, vh[:, n], decay[n])[0] for n in range(s.heads)]
        raw.append(torch.cat(o, 1))
        ones = torch.ones(s.vdim, dtype=torch.float64)
        normed = [torch.stack([oracle.rms_norm(r, ones, 1e-4) for r in x]) for x in o]
        want.append(torch.cat(normed, 1) * oracle.silu(z[b].double()))
    u = torch.cat((padded(q, s.heads, s.np), padded(k, s.heads, s.np), padded(v, s.heads, s.vdp), padded(z, s.heads, s.vdp)), -1)
    freq = torch.tensor(oracle.frequencies(rot)).float() if s.rot_dims else torch.empty(0)
    return s, torch.tensor(decay, dtype=torch.float64), u, freq, raw, want


def retain_pass(s, part, seq, state, decay, freq, dtype, eps=1e-4):
    """What the mixer does between its projections."""
    dev = part.device
    d, ld = decay.float().to(dev), decay.log2().clamp(min=-100.0).float().to(dev)
    if part.shape[1] == 1:
        return L.retention_step(part, freq, d, state, seq, s, eps, dtype)
    qk = L.retention_prep(part[..., : s.qk].contiguous(), freq, seq, s, dtype)
    vg = part[..., s.qk :].to(dtype).contiguous()
    return L.head_norm_gate(L.retention_scan(qk, vg, d, ld, state, seq, s), vg[..., s.inner :], s, eps)


@variant_param
@pytest.mark.parametrize("name", list(RETENTIONS))
def test_retention_matches_oracle(env, name):
    """Passes of several sizes and single tokens, two sequences in slots 2 and 0 whose states hold what an earlier owner left."""
    dev, dtype = env
    T = max(sum(c[b] for _, c in SCANS) for b in range(2))
    s, decay, u, freq, raw, want = retention_case(name, T, dtype)
    u, freq = u.to(dev), freq.to(dev)
    state = torch.full((3, s.heads, s.np, s.vdp), 7.0, device=dev)
    state[2, :, s.dim :] = state[2, :, :, s.vdim :] = state[0, :, s.dim :] = state[0, :, :, s.vdim :] = 0
    tab, at = table(dev, [0, 0], 3, [2, 0]), [0, 0]
    for n, counts in SCANS:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        out = retain_pass(s, part_of(u, at, n, counts), seq, state, decay, freq, dtype)
        assert torch.isfinite(out).all()
        for b in range(2):
            got = out[b, : counts[b]].view(counts[b], s.heads, s.vdp)
            assert not got[..., s.vdim :].any()
            if counts[b]:
                # a head whose products nearly cancel is scaled up by its norm, rounding included: compared in the scale before it
                here = slice(at[b], at[b] + counts[b])
                size = raw[b][here].view(counts[b], s.heads, s.vdim).square().mean(-1, keepdim=True).sqrt()
                close(got[..., : s.vdim].double().cpu() * size, want[b][here].view(counts[b], s.heads, s.vdim) * size, dtype, 2.0)
            at[b] += counts[b]
        move(tab, seq)
    assert torch.all(state[1] == 7)
    check(dev)


@variant_param
def test_state_goes_a_long_way(env):
    """One token far back is all there is: with a decay of one it stays whole, with others exactly its share is left, across chunks,
    passes and single tokens; rotation takes the distance into account."""
    dev, dtype = env
    s = L.RetentionShape(heads=4, dim=64, vdim=64, rot_dims=0)
    decay = torch.tensor([1.0, 0.995, 0.9, 0.0], dtype=torch.float64)
    T, mark = 700, 3
    u = torch.zeros(1, T, s.qk + 2 * s.inner)
    u[..., : s.heads * 64] = 1.0
    u[0, mark, s.heads * 64 : s.qk] = 1.0
    u[..., s.qk : s.qk + s.inner] = 1.0
    dd, ld = decay.float().to(dev), decay.log2().clamp(min=-100.0).float().to(dev)
    state, tab, at, got = torch.zeros(1, 4, 64, 64, device=dev), table(dev, [0]), 0, []
    freq = torch.empty(0, device=dev)
    for n in (2, 300, 127, 129, 142):
        seq = tab.begin(1, n)
        seq.start = seq.start.clone()
        part = u[:, at : at + n].to(dev)
        qk = L.retention_prep(part[..., : s.qk].contiguous(), freq, seq, s, dtype)
        got.append(L.retention_scan(qk, part[..., s.qk :].to(dtype).contiguous(), dd, ld, state, seq, s)[0].float().cpu())
        at += n
        move(tab, seq)
    got = torch.cat(got).view(T, 4, 64)
    power = (torch.arange(T) - mark).clamp(min=0)
    want = decay[None] ** power[:, None] * 8.0  # 64 products of 1 and 64^-1/2
    want[:mark] = 0
    close(got, want[..., None].expand(T, 4, 64).float(), dtype)
    assert float((got[-1, 1, 0] / want[-1, 1] - 1).abs()) < 1e-2
    close(state, (decay ** (T - 1 - mark) / 8).view(4, 1, 1).expand(1, 4, 64, 64).float(), torch.float32)
    check(dev)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["extremes", "wide", "uneven"])
def test_retention_in_segments(name):
    """Passes that the chunked kernel cuts into segments, against the kernel that goes token by token; unequal rows."""
    from keys_values_b200.ops import layers_cuda as LC

    dev = torch.device("cuda")
    s, decay = RETENTIONS[name]
    decay = torch.tensor(decay, dtype=torch.float64)
    T, counts = 2100, [2100, 1000]
    assert LC.lib().kvb_state_scan_tc_scratch_bytes(2, T, s.heads, s.heads, s.vdp, s.np) > 0
    g = torch.Generator().manual_seed(0)
    qk = torch.zeros(2, T, 2 * s.heads, s.np)
    qk[..., : s.dim] = torch.randn(2, T, 2 * s.heads, s.dim, generator=g) * s.dim**-0.5
    v = torch.zeros(2, T, s.heads, s.vdp)
    v[..., : s.vdim] = torch.randn(2, T, s.heads, s.vdim, generator=g)
    qk, v = qk.view(2, T, -1).to(dev, torch.bfloat16), v.view(2, T, -1).to(dev, torch.bfloat16)
    ys, states = [], []
    for dtype in (torch.bfloat16, torch.float32):
        state = torch.randn(2, s.heads, s.np, s.vdp, generator=torch.Generator().manual_seed(1)).to(dev)
        state[:, :, s.dim :] = state[..., s.vdim :] = 0
        tab = table(dev, [0, 5])  # the second one goes on
        seq = tab.begin(2, T, counts)
        ys.append(L.retention_scan(qk.to(dtype), v.to(dtype), decay.float().to(dev), decay.log2().clamp(min=-100.0).float().to(dev), state, seq, s))
        states.append(state)
    for b in range(2):
        close(ys[0][b, : counts[b]], ys[1][b, : counts[b]], torch.bfloat16)
    close(states[0], states[1], torch.float32, 10)
    assert not ys[0][1, 1000:].any()
    check(dev)
