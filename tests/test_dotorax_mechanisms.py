"""Each mechanism of the Dotorax design alone, against the plain oracle: the convolution in front of a sublayer, norms around zero, positions,
clamped units, windows with pooled blocks, keys and values of another layer, interleaved rotation, gated linear attention, the gated
recurrence, two mixers side by side. Inputs are made so that a fault shows: keys that stand out at every edge, decays that keep a mark for
thousands of tokens or drop it at once. CPU restatement and, marked ``gpu``, the kernels in both precisions and both variants."""
import math

import pytest
import torch

import dotorax_oracle as oracle
from keys_values_b200.kvcache.factory import KVCacheFactory
from keys_values_b200.models import dotorax
from keys_values_b200.models.registry import create_model
from keys_values_b200.ops import layers as L
from test_pazenex_mechanisms import check, close, env, move, padded, part_of, table, variant_param  # noqa: F401 (env is a fixture)


# ------------------------------------------------------------------------------------------------- between sublayers
def plus_identity(w):
    """h + conv(h) as one convolution ``(taps, width)``."""
    w = w.t().clone(memory_format=torch.contiguous_format)
    w[-1] += 1
    return w


EDGE_PASSES = [(9, [9, 6]), (1, [1, 1]), (2, [2, 2]), (1, [0, 1]), (40, [40, 33]), (1, [1, 1]), (3, [0, 3]), (5, [5, 1])]


@variant_param
@pytest.mark.parametrize("width,taps", [(1, 3), (7, 1), (64, 2), (250, 4), (1028, 5), (2048, 4), (3000, 9), (5120, 4), (1030, 3), (4096, 4), (3076, 3), (4096, 8),
                                        (1024, 4), (512, 7), (1022, 6)])
def test_edge_with_convolution(env, width, taps):
    """Residual sum of a normed result, norm, convolution, pass by pass: single tokens, runs that end anywhere, rows without tokens; a slot
    that is not part of the pass keeps what it holds."""
    dev, dtype = env
    g = torch.Generator().manual_seed(width)
    T, eps = 70, 1e-3
    x, sub = torch.randn(2, T, width, generator=g).double(), torch.randn(2, T, width, generator=g).to(dtype).double()
    after, before = (0.3 * torch.randn(width, generator=g).double() for _ in range(2))
    w = torch.randn(width, taps, generator=g).double()
    stream = torch.stack([x[b] + oracle.norm_rows(sub[b], after, eps) for b in range(2)])
    want = torch.stack([oracle.input_conv(oracle.norm_rows(s, before, eps), w) for s in stream])
    tab = table(dev, [0, 0], 3, [2, 0])
    ring = torch.full((3, taps, width), 9.0, dtype=dtype, device=dev)  # what an earlier owner left
    f32 = lambda t: t.float().to(dev)  # noqa: E731
    at, got = [0, 0], [([], []), ([], [])]
    for n, counts in EDGE_PASSES:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        xin, part = f32(part_of(x, at, n, counts)), part_of(sub, at, n, counts).to(dev, dtype)
        out, h = torch.empty_like(xin), torch.zeros(2, n, width, dtype=dtype, device=dev)
        L.norm_edge(xin, part, f32(1 + after), out, f32(1 + before), h, None, None, None, eps, False, None, L.EdgeTokens(seq, None, f32(plus_identity(w)), ring))
        for b in range(2):
            got[b][0].append(out[b, : counts[b]])
            got[b][1].append(h[b, : counts[b]])
            at[b] += counts[b]
        move(tab, seq)
    for b in range(2):
        close(torch.cat(got[b][0]), stream[b, : at[b]], torch.float32)
        close(torch.cat(got[b][1]), want[b, : at[b]], dtype, 1.0 if dtype != torch.float32 else 2.0)
    assert torch.all(ring[1] == 9)
    check(dev)


@variant_param
@pytest.mark.parametrize("T", [1, 2, 300])
def test_entry_with_positions(env, T):
    """Embedding and position vectors, norm and convolution of the first layer, rows at different places of the table and at its end."""
    dev, dtype = env
    g = torch.Generator().manual_seed(T)
    width, vocab, taps, eps = 36, 11, 3, 1e-3
    embed, pos = (torch.randn(n, width, generator=g).to(dtype) for n in (vocab, 700))
    w, before = torch.randn(width, taps, generator=g).double(), 0.2 * torch.randn(width, generator=g).double()
    start, counts = [0, 700 - T, 5], [T, T, max(1, T - 2)]
    tokens = torch.randint(0, vocab, (3, 700), generator=g)
    seq = table(dev, start).begin(3, T, counts)
    ring = torch.zeros(3, taps, width, dtype=dtype, device=dev)
    idx = torch.zeros(3, T, dtype=torch.int64)
    streams = []
    for b in range(3):
        x = embed[tokens[b]].double() + pos.double()
        h = oracle.norm_rows(x, before, eps)
        for p in range(max(0, start[b] - taps + 1), start[b]):
            ring[b, p % taps] = h[p].to(dtype)
        idx[b, : counts[b]] = tokens[b, start[b] : start[b] + counts[b]]
        streams.append((x, oracle.input_conv(h, w)))
    x, h = torch.empty(3, T, width, device=dev), torch.zeros(3, T, width, dtype=dtype, device=dev)
    L.norm_edge(None, None, None, x, (1 + before).float().to(dev), h, idx.to(dev), embed.to(dev), None, eps, False, None,
                L.EdgeTokens(seq, pos.to(dev), plus_identity(w).float().to(dev), ring))
    for b, (xs, hs) in enumerate(streams):
        at = slice(start[b], start[b] + counts[b])
        close(x[b, : counts[b]], xs[at], torch.float32)
        close(h[b, : counts[b]], hs[at], dtype)
    check(dev)


@variant_param
@pytest.mark.parametrize("ff,limit", [(1, 0.7), (8, 7.0), (13, 1.0), (200, 0.05)])
def test_clamped_unit(env, ff, limit):
    """Gates far above the limit are cut, far below it they are not; the other factor is cut on both sides."""
    dev, dtype = env
    g = torch.Generator().manual_seed(ff)
    gate, up = (4 * limit * torch.randn(6, ff, generator=g)).to(dtype), (4 * limit * torch.randn(6, ff, generator=g)).to(dtype)
    n = L.round8(ff)
    x = torch.cat((padded(gate.float(), 1, n), padded(up.float(), 1, n)), -1).to(dev, dtype)
    got = L.glu(x, ff, limit)
    assert got.shape == (6, n) and not got[:, ff:].any()
    close(got[:, :ff], oracle.clamped_unit(gate.double(), up.double(), limit), dtype)


@variant_param
def test_norm_weights_around_zero(env):
    from keys_values_b200.config import Config

    dev, dtype = env
    norm = Config(n_embd=40, n_head=1, norm_class_name="StreamOffsetRMSNorm").norm_class(40, eps=1e-2).to(dev, dtype)
    assert not norm.weight.any()
    with torch.no_grad():
        norm.weight.copy_(torch.linspace(-1.5, 1, 40))
        x = torch.randn(5, 40, generator=torch.Generator().manual_seed(1))
        close(norm(x.to(dev)), oracle.norm_rows(x.double(), norm.weight.double().cpu(), 1e-2), dtype)


# -------------------------------------------------------------------------------------------- mixers with their weights
def mixers(c, env, positions=None):
    """The layers' mixers of a random model, with caches, and the oracle's weights."""
    dev, dtype = env
    w = oracle.tensors(c, seed=3)
    model = create_model(dotorax.config_from_json(c, {k: tuple(v.shape) for k, v in w.items()})).to(dtype)
    model.load_state_dict(dotorax.state_dict(w, model.config))
    model = model.to(dev).eval()
    model.assign_kv_caches(KVCacheFactory.create(model, "layered-default", 3, positions or c["max_positions"], device=dev, dtype=dtype))
    return model, [b.attn for b in model.transformer.h], {k: v.double() for k, v in w.items()}


@torch.inference_mode()
def run_mixers(model, layers, h, env, passes):
    """Outputs of the layers' mixers, all on the input ``h (2, T, width)``, of two sequences in slots 2 and 0."""
    dev, dtype = env
    tab = model.sequences
    got = [tab.acquire() for _ in range(3)]
    tab.set_batch([got[2], got[0]])
    at, outs = [0, 0], [([], []) for _ in layers]
    for n, counts in passes:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        for layer, out in zip(layers, outs):
            y = layer(part_of(h, at, n, counts).to(dev, dtype), seq)
            for b in range(2):
                out[b].append(y[b, : counts[b]])
        at = [a + n for a, n in zip(at, counts)]
        move(tab, seq)
    check(dev)
    return [[torch.cat(o) for o in out] for out in outs], at


PASSES = [(37, [37, 20]), (1, [1, 1]), (1, [1, 1]), (95, [95, 64]), (2, [2, 2]), (1, [0, 1]), (4, [4, 4]), (1, [1, 1])]
A, P, R = oracle.attention_layer, oracle.parallel_layer, oracle.gla_layer
MIXERS = {
    "attention": [A()],
    "attention, one key head": [A(heads=20, kv_heads=1, dim=64, vdim=72, dims=32, scale=0.12)],
    "attention, odd": [A(heads=3, kv_heads=3, dim=7, vdim=5, dims=2)],
    "attention, deep": [A(heads=2, kv_heads=1, dim=200, vdim=160, dims=100, scale=0.06)],
    "shared": [A(heads=6, kv_heads=3, dim=16, vdim=24, dims=16), A(heads=6, kv_heads=3, dim=16, vdim=24, dims=16, scale=0.2, kv_from=0),
               A(heads=4, dim=24), A(heads=4, dim=24, scale=0.7, kv_from=2), A(heads=6, kv_heads=3, dim=16, vdim=24, dims=16, kv_from=0)],
    "parallel": [P()],
    "parallel, wide": [P(heads=8, kv_heads=1, dim=64, vdim=32, dims=64, scale=0.4, size=44, pool=16, width=128, blocks=2, conv=4)],
    "parallel, odd": [P(heads=3, kv_heads=1, dim=7, vdim=5, dims=4, size=3, pool=5, left_scale=-0.4, right_scale=2.5, width=33, blocks=11, conv=1)],
    "parallel, pool of one": [P(heads=2, kv_heads=2, dim=40, vdim=136, dims=8, scale=0.5, size=1, pool=1, width=8, blocks=1, conv=7)],
    "parallel, deep": [P(heads=2, kv_heads=1, dim=136, vdim=40, dims=136, scale=0.6, size=70, pool=3, width=300, blocks=3, conv=2)],
    "gla": [R()],
    "gla, wide": [R(heads=2, dim=128, vdim=128, tau=16.0)],
    "gla, odd": [R(heads=1, dim=11, vdim=13, tau=3.0)],
    "gla, large": [R(heads=2, dim=136, vdim=72, tau=16.0)],
}


def oracle_mixers(c, w, h):
    """Results of all layers' mixers on ``h (T, width)``."""
    eps, held, out = c["norm"]["eps"], {}, []
    for i, la in enumerate(c["layers"]):
        m, mix = la["mixer"], oracle.part(w, f"l{i}.mix.")
        if la["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                held[i] = oracle.keys_values(h, mix, m)
            out.append(oracle.attention(h, mix, m, held[i if src is None else src]))
        else:
            out.append(oracle.gla(h, mix, m, eps) if la["type"] == "gla" else oracle.side_by_side(h, mix, m, eps))
    return out


@variant_param
@pytest.mark.parametrize("name", list(MIXERS))
def test_mixers_match_oracle(env, name):
    """Passes of several sizes, single tokens, a row without tokens; a slot outside of the batch is not touched."""
    c = oracle.content(MIXERS[name], width=48)
    model, layers, w = mixers(c, env)
    h = torch.randn(2, 145, 48, generator=torch.Generator().manual_seed(7)).to(env[1])
    got, at = run_mixers(model, layers, h, env, PASSES)
    for b in range(2):
        for out, want in zip(got, oracle_mixers(c, w, h[b, : at[b]].double())):
            close(out[b], want, env[1], 4.0)
    for cache in model.get_kv_caches():
        for part in getattr(cache, "parts", (cache,)):
            for t in part.buffers_ or ():
                assert not t[:, 1].any()


@variant_param
@pytest.mark.parametrize("rot_dims", [2, 6, 20])
def test_interleaved_rotation(env, rot_dims):
    """Scores of a rotated window without pooled blocks in reach: far from position 0 the angles matter, and a wrong pairing shows."""
    c = oracle.content([P(heads=2, kv_heads=1, dim=20, vdim=8, dims=rot_dims, base=20.0, scale=3.0, size=300, pool=7, right_scale=0.0)], width=24)
    model, layers, w = mixers(c, env)
    h = torch.randn(2, 120, 24, generator=torch.Generator().manual_seed(5)).to(env[1])
    got, _ = run_mixers(model, layers, h, env, [(119, [119, 100]), (1, [1, 1])])
    for b, n in ((0, 120), (1, 101)):
        close(got[0][b], oracle_mixers(c, w, h[b, :n].double())[0], env[1], 6.0)


# ------------------------------------------------------------------------------------------------ windows with pooled blocks
POOLS = [(1, 1), (1, 3), (2, 2), (5, 3), (8, 8), (16, 5), (3, 40), (64, 8), (63, 16), (65, 1), (128, 32), (130, 7), (100, 130)]


@variant_param
@pytest.mark.parametrize("size,pool", POOLS)
def test_marked_tokens_and_blocks(env, size, pool):
    """A token, or a whole block, whose key stands out, at every edge: the last token inside a window and the first one outside of it, the
    tokens of a block that is just seen and of one that is not yet, the first block. Single tokens and passes; the blocks' means come
    from passes of several sizes."""
    dev, dtype = env
    s = L.GroupedShape(heads=2, kv_heads=1, dim=16, vdim=16, rot_dims=0, shared_value=False, gate=False, sink=False, scale=0.5, window=size, pool=pool)
    total = 2 * (size + pool) + 150
    base = (torch.arange(16.0) + 1) / 4
    ends = sorted({size + pool, size + 2 * pool - 1, size + 2 * pool, 127 + size, 128 + size, total - 3})
    cases = []  # marked positions
    for i in ends:
        edge = oracle.blocks_seen(i, size, pool) * pool
        for j in (i, i - size + 1, i - size, edge - 1, edge, edge + pool - 1, 0):
            cases.append((i, [j]))
            b = j // pool
            cases.append((i, list(range(b * pool, min((b + 1) * pool, i + 1)))))
    cases = [(i, [j for j in js if 0 <= j <= i]) for i, js in cases]
    cases = [(i, js) for i, js in cases if js]
    B = len(cases)
    k, v = -torch.ones(B, total, 16), torch.full((B, total, 16), 0.5)
    for b, (i, js) in enumerate(cases):
        k[b, js], v[b, js] = 1.0, base
    cols = torch.cat((torch.full((B, total, 32), 4.0), k, v), -1).to(dev, dtype)
    tiles = lambda n: -(-n // 128) * 128  # noqa: E731
    plan = L.RowPlan(tiles(total // pool), tiles(total))
    rows = torch.full((B, sum(plan), 1, 32), 9.0, dtype=dtype, device=dev)
    tab = table(dev, [0] * B)
    empty = torch.empty(0, device=dev)
    wanted = {i: [b for b, (e, _) in enumerate(cases) if e == i] for i in ends}
    at = 0
    for i in ends:
        # up to the query in two passes and itself alone, then the same query as the last of a pass
        first = at + (i - at) // 2
        for lo, hi in ((at, first), (first, i), (i, i + 1), (i - 1, i + 1)):
            if lo < 0 or hi <= lo:
                continue
            for sl in tab.batch:
                tab.pos[sl], tab.pos_host[sl] = lo, lo
            seq = tab.begin(B, hi - lo)
            seq.start = seq.start.clone()
            part = cols[:, lo:hi].contiguous()
            q = L.grouped_prep(part, None, None, empty, rows, seq, s, 0.0, plan)
            out = L.grouped_attend(q, part, rows, seq, s, None, plan)[:, -1].float().cpu().view(B, 2, 16)
            if hi != i + 1:
                continue
            for b in wanted[i]:
                want = oracle.pooled_row(i, torch.full((16,), 4.0).double(), k[b].double(), v[b].double(), 0.5, size, pool)
                assert torch.allclose(out[b].double(), want.expand(2, 16), atol=0.02, rtol=0.02), (size, pool, cases[b], hi - lo)
        at = i + 1
    check(dev)


@variant_param
@pytest.mark.parametrize("size,pool,ring", [(30, 4, 256), (5, 60, 256), (64, 64, 384)])
def test_pooled_rows_in_a_ring(env, size, pool, ring):
    """Far more positions than the tokens have rows: the same results as with a row per position."""
    dev, dtype = env
    g = torch.Generator().manual_seed(pool)
    s = L.GroupedShape(heads=4, kv_heads=2, dim=24, vdim=40, rot_dims=8, shared_value=False, gate=False, sink=False, scale=0.4, window=size, pool=pool,
                       head_norm=True)
    total = 1300
    qkv = torch.randn(2, total, s.ld, generator=g).to(dev, dtype)
    ones, freq, temp = torch.ones(s.dimp, device=dev), torch.tensor([1.0, 0.3, 0.1, 0.01], device=dev), torch.tensor([1.5, -0.7, 0.2, 3.0], device=dev)
    passes = [(150, [150, 93]), (1, [1, 1]), (120, [120, 120]), (1, [1, 1]), (2, [2, 2])] + [(130, [130, 121])] * 5 + [(1, [1, 1])] * 5 + [(100, [100, 100])]
    results = []
    for length in (ring, 1408):
        plan = L.RowPlan(-(-(total // pool) // 128) * 128, length)
        tab = table(dev, [0, 0], 3, [2, 0])
        rows = torch.full((3, sum(plan), s.kv_heads, s.row), 9.0, dtype=dtype, device=dev)
        at, outs = [0, 0], []
        for n, counts in passes:
            part = part_of(qkv, at, n, counts)
            seq = tab.begin(2, n, counts)
            seq.start = seq.start.clone()
            q = L.grouped_prep(part, ones, ones, freq, rows, seq, s, 1e-5, plan, temp)
            out = L.grouped_attend(q, part, rows, seq, s, None, plan)
            outs += [out[b, : counts[b]] for b in range(2)]
            at = [a + c for a, c in zip(at, counts)]
            move(tab, seq)
        assert torch.all(rows[1] == 9)
        results.append(torch.cat(outs))
    if dev.type == "cuda":  # the same tiles in the same order
        assert torch.equal(*results)
    else:
        close(*results, torch.float32)
    check(dev)


# ---------------------------------------------------------------------------------------------------- gated linear attention
def gla_case(heads, dim, vdim, rank, tau, T, seed, bias=(1.0, 2.0), dtype=torch.float32):
    """Shape, fp32 columns ``[q | k | a]``, values, decays' weights, and per sequence the oracle's outputs and states."""
    g = torch.Generator().manual_seed(seed)
    s = L.GatedLinearShape(heads=heads, dim=dim, vdim=vdim, rank=rank, tau=tau)
    q, k, v = (torch.randn(2, T, heads, n, generator=g) for n in (dim, dim, vdim))
    v = v.to(dtype).float()
    a, w = torch.randn(2, T, rank, generator=g), torch.randn(heads * dim, rank, generator=g) / rank**0.5
    b = bias[0] + bias[1] * torch.randn(heads * dim, generator=g)
    flat = lambda t, n: padded(t.reshape(2, T, -1), heads, n)  # noqa: E731
    qka = torch.cat((flat(q, s.np), flat(k, s.np), padded(a, 1, s.rp)), -1)
    decay = L.DecayWeights(padded(w.t().contiguous(), heads, s.np).contiguous(), padded(b[None], heads, s.np)[0].contiguous())
    want, states = [], []
    for i in range(2):
        alpha = (oracle.sigmoid(a[i].double() @ w.double().T + b.double()) ** (1 / tau)).view(T, heads, dim)
        both = [oracle.gla_recurrence(q[i, :, h].double() * dim**-0.5, k[i, :, h].double(), v[i, :, h].double(), alpha[:, h]) for h in range(heads)]
        want.append(torch.stack([o for o, _ in both], 1))
        states.append(torch.stack([S for _, S in both]))
    return s, qka, flat(v, s.vdp), decay, want, states


def run_gla(env, case, passes):
    dev, dtype = env
    s, qka, v, decay, want, _ = case
    decay = L.DecayWeights(*(t.to(dev) for t in decay))
    state = torch.full((3, s.heads, s.np, s.vdp), 9.0, device=dev)
    tab = table(dev, [0, 0], 3, [2, 0])
    at, outs = [0, 0], [[], []]
    for n, counts in passes:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        vg = torch.cat((part_of(v, at, n, counts), torch.zeros(2, n, 8)), -1).to(dev, dtype)  # values are columns of something wider
        y = L.gated_linear_scan(part_of(qka, at, n, counts).to(dev), vg, decay, state, seq, s)
        for b in range(2):
            assert not y[b, counts[b] :].any()
            outs[b].append(y[b, : counts[b]].view(-1, s.heads, s.vdp)[..., : s.vdim])
            at[b] += counts[b]
        move(tab, seq)
    assert torch.all(state[1] == 9)
    check(dev)
    return [torch.cat(o) for o in outs], state, at


GLA = {
    "plain": (3, 16, 24, 5, 8.0), "full": (2, 128, 128, 16, 16.0), "narrow": (4, 64, 40, 1, 16.0), "odd": (1, 7, 9, 3, 2.0), "large": (2, 200, 24, 20, 16.0),
    "wide": (1, 24, 200, 33, 4.0), "one": (1, 1, 1, 1, 2.0),
}


@variant_param
@pytest.mark.parametrize("name", list(GLA))
def test_gated_linear_scan(env, name):
    """Passes that end beside the borders of chunks, unequal rows, single tokens as passes."""
    case = gla_case(*GLA[name], T=420, seed=len(name), dtype=env[1])
    got, state, at = run_gla(env, case, [(129, [129, 127]), (2, [2, 1]), (1, [1, 0]), (128, [100, 128]), (150, [150, 140])])
    s, _, _, _, want, _ = case
    for b in range(2):
        close(got[b], want[b][: at[b]], env[1], 1.5)


@variant_param
def test_gated_linear_state_after_a_pass(env):
    case = gla_case(2, 40, 24, 4, 16.0, T=300, seed=1, dtype=env[1])
    s = case[0]
    _, state, _ = run_gla(env, case, [(300, [300, 300])])
    for b, slot in ((0, 2), (1, 0)):
        close(state[slot, :, : s.dim, : s.vdim], case[5][b], env[1])
        assert not state[slot, :, s.dim :].any() and not state[slot, :, :, s.vdim :].any()


@variant_param
@pytest.mark.parametrize("bias,tau", [((-9.0, 6.0), 1.0), ((-3.0, 6.0), 0.3), ((8.0, 8.0), 1.0)])
def test_gated_linear_decays_of_any_size(env, bias, tau):
    """Channels that drop everything from one token to the next beside such that keep it: within a chunk the products of the chunked
    kernel would leave the range of the numbers; and heads with harmless decays beside them."""
    case = gla_case(3, 24, 16, 4, tau, T=300, seed=2, bias=bias, dtype=env[1])
    s, qka, v, decay, _, _ = case
    decay.bias[: s.np] = 6.0  # the first head: close to 1
    a = qka[..., s.qk : s.qk + s.rank].double()
    want = []
    for b in range(2):
        alpha = (oracle.sigmoid(a[b] @ decay.weight.double() + decay.bias.double()) ** (1 / tau)).view(300, 3, s.np)
        q, k = qka[b, :, : s.qk].double().view(300, 2, 3, s.np).unbind(1)
        want.append(torch.stack([oracle.gla_recurrence(q[:, h] * s.query_scale, k[:, h], v[b].double().view(300, 3, -1)[:, h], alpha[:, h])[0] for h in range(3)], 1))
    got, _, at = run_gla(env, case, [(200, [200, 131]), (100, [100, 100])])
    for b in range(2):
        assert torch.isfinite(got[b]).all()
        for h in range(3):
            close(got[b][:, h], want[b][: at[b], h], env[1], 1.5)


@variant_param
@pytest.mark.parametrize("T", [1300, 2500])
def test_gated_linear_remembers(env, T):
    """One marked token, then tokens without keys: what is left of it after thousands, over segments that are worked on side by side."""
    dev, dtype = env
    s = L.GatedLinearShape(heads=1, dim=8, vdim=8, rank=1, tau=16.0)
    z = torch.tensor([9.0, 8.0, 7.0, 6.0, 5.0, 4.0, 3.0, 1.0])
    qka, v = torch.zeros(1, T, s.qk + s.rp), torch.zeros(1, T, 8)
    qka[..., :8] = 1.0
    qka[0, 3, 8:16] = 1.0
    v[0, 3] = 1 + torch.arange(8.0)
    state = torch.zeros(1, 1, 8, 8, device=dev)
    seq = table(dev, [0]).begin(1, T)
    y = L.gated_linear_scan(qka.to(dev), v.to(dev, dtype), L.DecayWeights(torch.zeros(1, 8, device=dev), z.to(dev)), state, seq, s)[0]
    alpha = torch.sigmoid(z.double()) ** (1 / 16)
    for t in (3, 4, 63, 64, 127, 128, 640, T - 1):
        want = (alpha ** (t - 3)).sum() * 8**-0.5 * (1 + torch.arange(8.0).double())
        close(y[t], want, dtype)
    assert not y[:3].any()
    close(state[0, 0], (alpha ** (T - 4))[:, None] * (1 + torch.arange(8.0).double()), torch.float32, 5.0 if dtype == torch.float32 else 200.0)  # bf16: the key is rounded once
    check(dev)


@variant_param
@pytest.mark.parametrize("name", list(GLA))
def test_gated_linear_step(env, name):
    """Single tokens from the first one on: state, norm with a weight, gate."""
    dev, dtype = env
    s, qka, v, decay, want, _ = gla_case(*GLA[name], T=12, seed=4)
    eps = 1e-3
    g = torch.Generator().manual_seed(9)
    gate, weight = torch.randn(2, 12, s.heads, s.vdim, generator=g), 1 + 0.5 * torch.randn(s.vdim, generator=g)
    u = torch.cat((qka, v, padded(gate.reshape(2, 12, -1), s.heads, s.vdp)), -1).to(dev)
    decay, wt = L.DecayWeights(*(t.to(dev) for t in decay)), padded(weight, 1, s.vdp).to(dev)
    state = torch.full((3, s.heads, s.np, s.vdp), 9.0, device=dev)
    tab = table(dev, [0, 0], 3, [2, 0])
    at, n = [0, 0], 0
    for t in range(12):
        counts = [1, 0 if t == 5 else 1]
        seq = tab.begin(2, 1, counts)
        seq.start = seq.start.clone()
        y = L.gated_linear_step(torch.stack([u[b, at[b] : at[b] + 1] for b in range(2)]), decay, wt, state, seq, s, eps, dtype)
        for b in range(2):
            if counts[b]:
                o = torch.cat([oracle.over_rms(want[b][at[b], h], eps) * weight.double() * oracle.silu(gate[b, at[b], h].double()) for h in range(s.heads)])
                close(y[b, 0].view(s.heads, s.vdp)[:, : s.vdim].reshape(-1), o, dtype)
            else:
                assert not y[b].any()
            at[b] += counts[b]
        move(tab, seq)
    check(dev)


@variant_param
@pytest.mark.parametrize("heads,vdim", [(3, 24), (1, 9), (5, 128), (2, 200)])
def test_head_norm_with_weight(env, heads, vdim):
    dev, dtype = env
    g = torch.Generator().manual_seed(vdim)
    s = L.GatedLinearShape(heads=heads, dim=8, vdim=vdim, rank=1, tau=1.0)
    y, gate = (torch.randn(2, 7, heads, vdim, generator=g).to(dtype) for _ in range(2))
    weight = 1 + 0.5 * torch.randn(vdim, generator=g)
    flat = lambda t: padded(t.float().reshape(2, 7, -1), heads, s.vdp)  # noqa: E731
    got = L.head_norm_gate(flat(y).to(dev, dtype), flat(gate).to(dev, dtype), s, 1e-3, padded(weight, 1, s.vdp).to(dev)).view(2, 7, heads, s.vdp)
    want = torch.stack([oracle.over_rms(r, 1e-3) for r in y.double().view(-1, vdim)]).view(y.shape) * weight.double() * oracle.silu(gate.double())
    close(got[..., :vdim], want, dtype)
    assert not got[..., vdim:].any()


# ------------------------------------------------------------------------------------------------------- gated recurrence
def recurrence_case(width, blocks, taps, T, dtype, seed=0, lam=(-3.0, 1.5)):
    """Shape, weights, columns ``[y | x]`` and the oracle's results; everything the oracle starts from is rounded as the kernels get it."""
    g = torch.Generator().manual_seed(seed)
    s = L.RecurrenceShape(width=width, blocks=blocks, taps=taps)
    n = s.part
    conv, cb = torch.randn(width, taps, generator=g), 0.2 * torch.randn(width, generator=g)
    ra, ri = ((torch.randn(blocks, n, n, generator=g) / n**0.5).to(dtype).float() for _ in range(2))
    br, bi = (0.5 * torch.randn(width, generator=g) for _ in range(2))
    la = lam[0] + lam[1] * torch.randn(width, generator=g)
    y, x = (torch.randn(2, T, width, generator=g).to(dtype).float() for _ in range(2))
    ch = lambda t: padded(t, blocks, s.pp).contiguous()  # noqa: E731
    gates = torch.zeros(blocks, s.pp, 2 * s.pp)
    gates[:, :n, :n], gates[:, :n, s.pp : s.pp + n] = ra.transpose(1, 2), ri.transpose(1, 2)
    rate = -8 * torch.nn.functional.softplus(la.double()) / math.log(2)
    w = L.RecurrenceWeights(ch(conv.t()), ch(cb), gates.to(dtype), ch(br), ch(bi), ch(rate.float()))
    want = []
    for b in range(2):
        u = oracle.causal_conv(x[b].double(), conv.double(), cb.double()).to(dtype).double()
        r, i = (oracle.sigmoid(oracle.block_product(u, m.double(), v.double().view(blocks, n))) for m, v in ((ra, br), (ri, bi)))
        want.append(oracle.gated_lru(u, r, i, la.double()) * oracle.gelu_tanh(y[b].double()))
    return s, w, torch.cat((ch(y), ch(x)), -1), want


@variant_param
@pytest.mark.parametrize("width,blocks,taps", [(36, 3, 3), (64, 1, 4), (33, 11, 1), (320, 5, 4), (80, 2, 7), (1, 1, 2)])
def test_gated_recurrence(env, width, blocks, taps):
    """Convolution, gates, recurrence and output over passes of several sizes and single tokens; columns of wider rows; a factor."""
    dev, dtype = env
    s, w, u, want = recurrence_case(width, blocks, taps, 320, dtype)
    w = L.RecurrenceWeights(*(t.to(dev) for t in w))
    state, ring = torch.full((3, s.channels), 9.0, device=dev), torch.full((3, taps, s.channels), 9.0, dtype=dtype, device=dev)
    tab = table(dev, [0, 0], 3, [2, 0])
    at, outs = [0, 0], [[], []]
    for n, counts in [(129, [129, 60]), (1, [1, 1]), (2, [1, 2]), (1, [0, 1]), (128, [128, 128]), (3, [0, 3]), (1, [1, 1]), (17, [17, 16])]:
        seq = tab.begin(2, n, counts)
        seq.start = seq.start.clone()
        wide = torch.cat((torch.ones(2, n, 8), part_of(u, at, n, counts)), -1).to(dev, dtype)
        y = torch.full((2, n, s.channels + 16), 5.0, dtype=dtype, device=dev)
        L.gated_recurrence(wide[..., 8:], w, ring, state, seq, s, 1.75, y[..., 8:-8])
        assert torch.all(y[..., :8] == 5) and torch.all(y[..., -8:] == 5)
        for b in range(2):
            assert not y[b, counts[b] :, 8:-8].any()
            outs[b].append(y[b, : counts[b], 8:-8].reshape(-1, s.blocks, s.pp)[..., : s.part].reshape(counts[b], width))
            at[b] += counts[b]
        move(tab, seq)
    for b in range(2):
        close(torch.cat(outs[b]), 1.75 * want[b][: at[b]], dtype, 1.5)
    assert torch.all(state[1] == 9) and torch.all(ring[1] == 9)
    check(dev)


@variant_param
@pytest.mark.parametrize("lam", [-14.0, 4.0])
def test_gated_recurrence_at_both_ends(env, lam):
    """Decays so close to one that a state holds for thousands of tokens (and 1 − a² is tiny), and such that nothing is left."""
    dev, dtype = env
    s, w, u, want = recurrence_case(24, 1, 2, 1500, dtype, seed=3, lam=(lam, 0.1))
    w = L.RecurrenceWeights(*(t.to(dev) for t in w))
    state, ring = torch.zeros(2, s.channels, device=dev), torch.zeros(2, 2, s.channels, dtype=dtype, device=dev)
    seq = table(dev, [0, 0]).begin(2, 1500)
    y = torch.empty(2, 1500, s.channels, dtype=dtype, device=dev)
    L.gated_recurrence(u.to(dev, dtype), w, ring, state, seq, s, 1.0, y)
    for b in range(2):
        close(y[b], want[b], dtype, 1.5)
    check(dev)
