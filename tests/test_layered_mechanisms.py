"""Each mechanism of the layered models alone, against the plain oracle: layer edges, rotation, latent attention at the edges of
windows, tiles, splits and rings, routed experts. Attention inputs are made so that one key stands out: seen, it decides the
output; hidden, it leaves no trace. CPU restatement and, marked ``gpu``, the kernels in both precisions and both variants."""
import math

import pytest
import torch

import layered_oracle as oracle
from keys_values_b200.kvcache.sequences import SequenceTable
from keys_values_b200.ops import layers as L

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
device_param = pytest.mark.parametrize("device", DEVICES)
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


def tol(dtype):
    return 1e-4 if dtype == torch.float32 else 2e-2


def close(got, want, dtype, scale=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-6)
    assert err < scale * tol(dtype), err


def table(device, B, start, shift_layers=0, width=0, slots=None):
    t = SequenceTable(max(B, 1 + max(slots or [0])), device, shift_layers, width)
    got = [t.acquire() for _ in range(t.n_slots)]
    t.set_batch(slots if slots is not None else got[:B])
    for s, n in zip(t.batch, start):
        t.pos[s] = n
        t.pos_host[s] = n
    return t


def check(device):
    from keys_values_b200 import ops

    ops.check_status(device)


# ------------------------------------------------------------------------------------------------ layer edges
@variant_param
@pytest.mark.parametrize("width", [5, 64, 250, 1028, 3072])
def test_layer_edge(env, width):
    """Residual sum with expert outputs, depth average, norm and shift over two passes and a single token."""
    dev, dtype = env
    torch.manual_seed(width)
    B, n_hist, top, eps = 2, 3, 2, 1e-3
    T = 40 if width < 1000 else 9
    tab = table(dev, B, [0, 0], 1, width)
    tab.shift.fill_(7.0)  # what an earlier owner left
    gain, blend = torch.tensor(1.7), torch.rand(width)
    coef = torch.randn(n_hist + 1)
    counts = [T, T - 4]
    total = [T + 4, T - 3]
    x_in = torch.randn(B, T + 4, width)
    mix = torch.randn(B, T + 4, width).to(dtype).float()
    ex = torch.randn(B, T + 4, top, width).to(dtype).float()
    ew = torch.rand(B, T + 4, top)
    hist = torch.randn(n_hist, B, T + 4, width)
    new = x_in + mix + (ew[..., None] * ex).sum(2)
    want_x = oracle.depth_average([*hist, new], coef)
    want_h = torch.stack([oracle.scalar_norm(want_x[b].double(), float(gain), eps) for b in range(B)])
    want_hs = torch.stack([oracle.token_shift(want_h[b], blend.double()) for b in range(B)])
    at = [0, 0]
    for n, cs in ((T, counts), (1, [1, 1]), (3, [3, 0])):
        seq = tab.begin(B, n, cs)
        # rows beyond a row's count are padding: anything finite
        def part(t):
            out = torch.zeros(B, n, *t.shape[2:])
            for b in range(B):
                out[b, : cs[b]] = t[b, at[b] : at[b] + cs[b]]
            return out
        h_ = torch.zeros(n_hist + 2, B, n, width, device=dev)
        for j in range(n_hist):
            h_[j] = part(hist[j]).to(dev)
        expert_out = part(ex).reshape(-1, width).to(dev, dtype)
        perm = torch.randperm(expert_out.shape[0])
        rows = torch.empty_like(perm)
        rows[perm] = torch.arange(len(perm))
        out = torch.empty(B, n, width, device=dev)
        h = torch.empty(B, n, width, device=dev, dtype=dtype)
        hs = torch.empty_like(h)
        L.layer_edge(part(x_in).to(dev), part(mix).to(dev, dtype), (expert_out[perm.to(dev)].contiguous(), rows.view(-1, top).int().to(dev),
                     part(ew).reshape(-1, top).to(dev)), h_, n_hist, coef.to(dev), out, gain.to(dev), blend.to(dev), tab.shift[0], h, hs, seq, eps)
        for b in range(B):
            span = slice(at[b], at[b] + cs[b])
            close(h_[n_hist, b, : cs[b]], new[b, span], torch.float32) if cs[b] else None
            if cs[b]:
                close(out[b, : cs[b]], want_x[b, span], torch.float32)
                close(h[b, : cs[b]], want_h[b, span], dtype)
                close(hs[b, : cs[b]], want_hs[b, span], dtype)
                close(tab.shift[0, b], want_h[b, at[b] + cs[b] - 1], torch.float32)
        tab.finish(seq, torch.zeros(B, n, dtype=torch.int64, device=dev))
        at = [a + c for a, c in zip(at, cs)]
    assert at == total
    # without history, experts, shift
    out = torch.empty(B, 2, width, device=dev)
    h = torch.empty(B, 2, width, device=dev, dtype=dtype)
    L.layer_edge(x_in[:, :2].to(dev).contiguous(), mix[:, :2].to(dev, dtype).contiguous(), None, None, 0, None, out, gain.to(dev), None, None, h,
                 None, tab.begin(B, 2), eps)
    close(out, (x_in + mix)[:, :2], torch.float32)
    close(h[0], oracle.scalar_norm((x_in + mix)[0, :2].double(), float(gain), eps), dtype)
    rows = torch.tensor([3, 0], device=dev)
    y = L.scalar_rmsnorm(x_in[0].to(dev).contiguous(), gain.to(dev), eps, dtype, rows)
    close(y, oracle.scalar_norm(x_in[0, [3, 0]].double(), float(gain), eps), dtype)
    if dev.type == "cuda":
        check(dev)


@variant_param
def test_bigram_embedding_across_passes(env):
    dev, dtype = env
    vocab, width, eps = 50, 36, 1e-4
    bg = dict(buckets=23, mul_prev=1000003, mul_cur=7)  # products beyond 31 bits
    g = torch.Generator().manual_seed(0)
    embed, big = torch.randn(vocab, width, generator=g).to(dtype), torch.randn(24, width, generator=g).to(dtype)
    toks = [torch.randint(0, vocab, (n,), generator=g).tolist() for n in (30, 17)]
    want = [oracle.embedding(t, dict(embed=embed.double(), bigram=big.double()), dict(embedding=dict(bigram=bg))) for t in toks]
    tab = table(dev, 2, [0, 0], slots=[3, 1])
    tab.prev_token.fill_(11)
    at = [0, 0]
    for n, cs in ((9, [9, 4]), (1, [1, 1]), (2, [2, 2]), (12, [12, 10]), (6, [6, 0])):
        idx = torch.zeros(2, n, dtype=torch.int64)
        for b in range(2):
            idx[b, : cs[b]] = torch.tensor(toks[b][at[b] : at[b] + cs[b]], dtype=torch.int64)
        idx = idx.to(dev)
        seq = tab.begin(2, n, cs)
        x = torch.empty(2, n, width, device=dev)
        h = torch.empty(2, n, width, device=dev, dtype=dtype)
        L.embed_edge(idx, tab.prev_token, embed.to(dev), big.to(dev), bg["buckets"], bg["mul_prev"], bg["mul_cur"], x,
                     torch.tensor(0.5, device=dev), None, None, h, None, seq, eps)
        for b in range(2):
            if cs[b]:
                close(x[b, : cs[b]], want[b][at[b] : at[b] + cs[b]], torch.float32)
                close(h[b, : cs[b]], oracle.scalar_norm(want[b][at[b] : at[b] + cs[b]], 0.5, eps), dtype)
        tab.finish(seq, idx)
        at = [a + c for a, c in zip(at, cs)]
    assert tab.pos.tolist()[3] == 30 and tab.pos.tolist()[1] == 17


@pytest.mark.gpu
def test_token_outside_of_the_vocabulary_is_reported():
    from keys_values_b200.ops.cuda import NativeError

    dev = torch.device("cuda")
    tab = table(dev, 1, [0])
    x = torch.empty(1, 2, 8, device=dev)
    L.embed_edge(torch.tensor([[1, 9]], device=dev), tab.prev_token, torch.ones(9, 8, device=dev), None, 0, 0, 0, x, None, None, None, None, None,
                 tab.begin(1, 2), 1e-5)
    with pytest.raises(NativeError, match="index out of range"):
        check(dev)


# ------------------------------------------------------------------------------------------- latent attention
SHAPES = {
    "small": L.LatentShape(heads=3, dim=24, rot=8, vdim=40, kv_rank=48, rot_dims=8),
    "odd": L.LatentShape(heads=2, dim=5, rot=2, vdim=3, kv_rank=7, rot_dims=2),
    "partly rotated": L.LatentShape(heads=2, dim=16, rot=24, vdim=16, kv_rank=40, rot_dims=10),
    "two tiles of heads": L.LatentShape(heads=21, dim=128, rot=64, vdim=128, kv_rank=512, rot_dims=64),
    "one query tile per CTA": L.LatentShape(heads=2, dim=136, rot=32, vdim=200, kv_rank=264, rot_dims=32),
    "wide rotary part": L.LatentShape(heads=1, dim=40, rot=96, vdim=72, kv_rank=120, rot_dims=96),
}


@variant_param
@pytest.mark.parametrize("name", list(SHAPES))
def test_latent_prep(env, name):
    """Split, latent norm, rotation at near and far positions; rows into a buffer and straight into the ring."""
    dev, dtype = env
    s, eps, base = SHAPES[name], 1e-3, 500.0
    g = torch.Generator().manual_seed(1)
    B, T, P, C = 2, 3, 2, 5
    start = [0, 70001]
    tab = table(dev, B, start, slots=[2, 0])
    qkv = torch.randn(B, T, s.heads * (s.dim + s.rot) + s.kv_rank + s.rot, generator=g).to(dtype)
    norm = torch.randn(s.kv_rank, generator=g)
    freq = (base ** (torch.arange(s.rot_dims // 2, dtype=torch.float64) * (-2.0 / s.rot_dims))).float()
    nq = s.heads * (s.dim + s.rot)
    want_q = torch.zeros(B, T, s.heads, s.dimp + s.rp, dtype=torch.float64)
    want_l = torch.zeros(B, T, s.row, dtype=torch.float64)
    for b in range(B):
        for t in range(T):
            x, pos = qkv[b, t].double(), start[b] + t
            for h in range(s.heads):
                q = x[h * (s.dim + s.rot) : (h + 1) * (s.dim + s.rot)]
                want_q[b, t, h, : s.dim] = q[: s.dim]
                want_q[b, t, h, s.dimp : s.dimp + s.rot] = oracle.rotate(q[s.dim :], pos, base, s.rot_dims)
            want_l[b, t, : s.kv_rank] = oracle.unit_rms(x[nq : nq + s.kv_rank], eps) * norm.double()
            want_l[b, t, s.kvp : s.kvp + s.rot] = oracle.rotate(x[nq + s.kv_rank :], pos, base, s.rot_dims)
    latent = torch.zeros(B, P + T, s.row, dtype=dtype, device=dev)
    args = (norm.to(dev), freq.to(dev))
    q = L.latent_prep(qkv.to(dev), *args, latent, None, tab.begin(B, T), P, s, eps)
    # an angle of 7e4 radians has an fp32 spacing of 8e-3
    close(q, want_q, dtype, scale=100 if dtype == torch.float32 else 2)
    close(latent[:, P:], want_l, dtype, scale=100 if dtype == torch.float32 else 2)
    close(q[0], want_q[0], dtype)
    assert float(latent[:, :P].abs().max()) == 0
    ring = torch.full((3, C, s.row), 9.0, dtype=dtype, device=dev)
    one = qkv[:, :1].contiguous().to(dev)
    q1 = L.latent_prep(one, *args, None, ring, tab.begin(B, 1, [1, 0]), 0, s, eps)
    close(q1[0], want_q[0, :1], dtype)
    close(ring[2, 0], want_l[0, 0], dtype)
    ring[2, 0] = 9.0
    assert float((ring - 9.0).abs().max()) == 0  # the row without a token wrote nothing
    L.latent_prep(one, *args, None, ring, tab.begin(B, 1), 0, s, eps)
    close(ring[0, 70001 % C], want_l[1, 0], dtype, scale=100 if dtype == torch.float32 else 2)


@device_param
def test_rows_into_the_ring_and_back(device):
    """Several passes of unequal rows: the ring holds the newest positions, a pass finds those before it in order."""
    dev = torch.device(device)
    s = L.LatentShape(heads=1, dim=8, rot=8, vdim=8, kv_rank=8, rot_dims=8)
    B, C = 3, 7
    slots = [4, 0, 2]
    ring = torch.zeros(5, C, s.row, device=dev)
    tab = table(dev, B, [0, 0, 0], slots=slots)
    g = torch.Generator().manual_seed(0)
    qkv = torch.randn(B, 40, 16 + 8 + 8, generator=g)
    rows = torch.zeros(B, 40, s.row)
    for b in range(B):
        for p in range(40):
            rows[b, p, :8] = oracle.unit_rms(qkv[b, p, 16:24].double(), 0.1)
            rows[b, p, 8:] = oracle.rotate(qkv[b, p, 24:].double(), p, 100.0, 8)
    norm, freq = torch.ones(8, device=dev), (100.0 ** (torch.arange(4, dtype=torch.float64) * -0.25)).float().to(dev)
    at = [0, 0, 0]
    for n, cs in ((5, [5, 2, 0]), (9, [9, 1, 9]), (1, [1, 0, 1]), (2, [2, 2, 2]), (20, [3, 20, 0])):
        seq = tab.begin(B, n, cs)
        P = min(seq.max_start, C)
        latent = torch.full((B, P + n, s.row), -1.0, device=dev)
        L.ring_gather(ring, latent, seq, P)
        part = torch.zeros(B, n, qkv.shape[2])
        for b in range(B):
            part[b, : cs[b]] = qkv[b, at[b] : at[b] + cs[b]]
        L.latent_prep(part.to(dev), norm, freq, latent, ring, seq, P, s, 0.1)
        for b in range(B):
            want = torch.zeros(P + cs[b], s.row)
            for j in range(P + cs[b]):
                if at[b] - P + j >= 0:
                    want[j] = rows[b, at[b] - P + j]
            if len(want):
                close(latent[b, : P + cs[b]], want, torch.float32)
        tab.finish(seq, torch.zeros(B, n, dtype=torch.int64, device=dev))
        at = [a + c for a, c in zip(at, cs)]
        for b, slot in enumerate(slots):
            for p in range(max(0, at[b] - C), at[b]):
                close(ring[slot, p % C], rows[b, p], torch.float32)
    assert float(ring[1].abs().max()) == 0 and float(ring[3].abs().max()) == 0


def attend_inputs(s, B, T, P, dtype, seed, sharp=1.0):
    g = torch.Generator().manual_seed(seed)
    q = torch.zeros(B, T, s.heads, s.dimp + s.rp)
    q[..., : s.dim] = sharp * torch.randn(B, T, s.heads, s.dim, generator=g)
    q[..., s.dimp : s.dimp + s.rot] = sharp * torch.randn(B, T, s.heads, s.rot, generator=g)
    kv = torch.zeros(B, P + T, s.heads, s.dimp + s.vdp)
    kv[..., : s.dim] = torch.randn(B, P + T, s.heads, s.dim, generator=g)
    kv[..., s.dimp : s.dimp + s.vdim] = torch.randn(B, P + T, s.heads, s.vdim, generator=g)
    lat = torch.zeros(B, P + T, s.row)
    lat[..., s.kvp : s.kvp + s.rot] = torch.randn(B, P + T, s.rot, generator=g)
    return q.to(dtype), kv.to(dtype), lat.to(dtype)


@variant_param
@pytest.mark.parametrize("name", list(SHAPES))
@pytest.mark.parametrize("T,P,start,window", [(2, 0, [0, 0], 1), (70, 5, [5, 3], 6), (300, 0, [0, 0], 129), (260, 127, [127, 40], 128), (150, 200, [900, 0], 201),
                                              (130, 60, [60, 7], 0)])
def test_latent_attend(env, name, T, P, start, window):
    dev, dtype = env
    s, B = SHAPES[name], 2
    q, kv, lat = attend_inputs(s, B, T, P, dtype, seed=T)
    scale = 1.3 / math.sqrt(s.dim + s.rot)
    out = L.latent_attend(q.to(dev), kv.to(dev), lat.to(dev), table(dev, B, start).begin(B, T), P, s, window, scale)
    out = out.view(B, T, s.heads, s.vdp)
    for b in range(B):
        for h in range(s.heads) if s.heads < 8 else (0, 17, s.heads - 1):
            k = torch.cat((kv[b, :, h, : s.dimp], lat[b, :, s.kvp :]), -1).double()
            first = max(0, P - start[b])  # rows before that hold no token
            qa = torch.zeros(P + T, s.dimp + s.rp, dtype=torch.float64)
            qa[P:] = q[b, :, h].double()
            want = oracle.window_softmax_attention(qa[first:], k[first:], kv[b, first:, h, s.dimp :].double(), scale, window or P + T)[P - first :]
            close(out[b, :, h], want, dtype)
    if dev.type == "cuda":
        check(dev)


@variant_param
@pytest.mark.parametrize("window", [1, 2, 64, 127, 128, 129, 200, 256])
def test_window_edge_in_prompts(env, window):
    """One key outweighs all others: the last query that sees it and the first that does not, for keys at tile borders."""
    dev, dtype = env
    s = SHAPES["small"]
    T, P = 420, 130
    start = 500
    for key in (0, 1, 127, 128, 129, 130, 131, 255, 256, 257, 383, 384):
        q, kv, lat = attend_inputs(s, 1, T, P, dtype, seed=key)
        q[..., : s.dim] = 1.0
        q[..., s.dimp :] = 0.0
        kv[..., : s.dim] = 0.0
        kv[0, key, :, : s.dim] = 4.0  # score 96 · scale, all others 0
        kv[..., s.dimp : s.dimp + s.vdim] = 0.25
        kv[0, key, :, s.dimp : s.dimp + s.vdim] = -3.0
        out = L.latent_attend(q.to(dev), kv.to(dev), lat.to(dev), table(dev, 1, [start]).begin(1, T), P, s, window, 0.5)
        seen = out.view(T, s.heads, s.vdp)[:, :, : s.vdim].float().cpu() < -2.5
        want = torch.tensor([0 <= P + t - key < window for t in range(T)])
        assert torch.equal(seen.all(-1).all(-1), want) and torch.equal(seen.any(-1).any(-1), want), key
        assert torch.allclose(out.view(T, s.heads, s.vdp)[~want.to(dev)][..., : s.vdim].float(), torch.tensor(0.25, device=dev))


@variant_param
@pytest.mark.parametrize("name", list(SHAPES))
@pytest.mark.parametrize("C,positions", [(1, [0, 5]), (5, [0, 3, 4, 5, 12]), (64, [63, 64, 1000]), (300, [127, 299, 64, 5000, 0]), (1500, [1499, 700, 9999])])
def test_latent_decode(env, name, C, positions):
    """Sequences at different positions, full rings and partly filled ones, against every visible row."""
    dev, dtype = env
    s, B = SHAPES[name], len(positions)
    g = torch.Generator().manual_seed(C)
    slots = list(range(B))[::-1]
    ring = torch.zeros(B, C, s.row)
    ring[..., : s.kv_rank] = torch.randn(B, C, s.kv_rank, generator=g)
    ring[..., s.kvp : s.kvp + s.rot] = torch.randn(B, C, s.rot, generator=g)
    qa, q = torch.zeros(s.heads, B, s.kvp), torch.zeros(B, 1, s.heads, s.dimp + s.rp)
    qa[..., : s.kv_rank] = torch.randn(s.heads, B, s.kv_rank, generator=g)
    q[..., s.dimp : s.dimp + s.rot] = torch.randn(B, 1, s.heads, s.rot, generator=g)
    q[..., : s.dim] = 50.0  # not part of the score here
    ring, qa, q = ring.to(dtype), qa.to(dtype), q.to(dtype)
    scale = 1.5 / math.sqrt(s.kv_rank + s.rot)
    out = L.latent_decode(qa.to(dev), q.to(dev), ring.to(dev), table(dev, B, positions, slots=slots).begin(B, 1), s, scale)
    for b in range(B):
        rows = ring[slots[b], : min(positions[b] + 1, C)].double()
        for h in range(s.heads) if s.heads < 8 else (0, 16, s.heads - 1):
            qc = torch.cat((qa[h, b], q[b, 0, h, s.dimp :])).double()
            p = torch.softmax(rows @ qc * scale, 0)
            close(out[h, b], p @ rows[:, : s.kvp], dtype)
    # one row outweighs all others, wherever it lies
    for r in {0, C // 2, C - 1, min(63, C - 1), min(64, C - 1)}:
        ring[:] = 0
        ring[..., 0] = 0.25
        ring[:, r, : s.kv_rank] = -4.0
        qa[:] = 0
        qa[..., : s.kv_rank] = -2.0
        out = L.latent_decode(qa.to(dev), (q * 0).to(dev), ring.to(dev), table(dev, B, positions, slots=slots).begin(B, 1), s, 3.0)
        for b in range(B):
            seen = bool((out[:, b, 0].float() < -3.5).all())
            assert seen == (r < min(positions[b] + 1, C)), (r, positions[b])


# --------------------------------------------------------------------------------------------- routed experts
def experts(env, n, E, top, width, ff, seed, renormalize=False, spread=2.0):
    dev, dtype = env
    g = torch.Generator().manual_seed(seed)
    h = torch.randn(n, width, generator=g).to(dtype)
    w = {"router": (spread / math.sqrt(width) * torch.randn(E, width, generator=g)).to(dtype)}
    for e in range(E):
        w[f"e{e}.up"] = (torch.randn(ff, width, generator=g) / math.sqrt(width)).to(dtype)
        w[f"e{e}.down"] = (torch.randn(width, ff, generator=g) / math.sqrt(ff)).to(dtype)
    pad = lambda t, k: torch.nn.functional.pad(t, (0, k - t.shape[-1])).contiguous()  # noqa: E731
    up = pad(torch.stack([w[f"e{e}.up"] for e in range(E)]), L.round8(width)).to(dev)
    down = pad(torch.stack([w[f"e{e}.down"] for e in range(E)]), L.round8(ff)).to(dev)
    logits = L.linear_fp32(h.to(dev), w["router"].to(dev))
    assert logits.dtype == torch.float32
    out, row, weight = L.routed_experts(h.to(dev), logits, up, down, top, "relu_squared", L.RouterRule(renormalize=renormalize), ff, width)
    y = (weight[..., None] * out[row.long()][..., :width].float()).sum(1)
    return h.double(), {k: v.double() for k, v in w.items()}, y, weight, logits


@variant_param
@pytest.mark.parametrize("n,E,top,width,ff", [(1, 1, 1, 8, 8), (3, 5, 5, 31, 9), (40, 3, 1, 64, 72), (70, 70, 4, 40, 24), (600, 4, 2, 136, 200), (33, 6, 2, 520, 264)])
def test_routed_experts(env, n, E, top, width, ff):
    dev, dtype = env
    h, w, y, weight, logits = experts(env, n, E, top, width, ff, seed=n)
    want = oracle.routed_experts(h, w, {"router": {"top": top}})
    if dtype == torch.float32:
        close(y, want, dtype)
    else:  # the choice of a token may be a close call: compare the tokens that are not
        z = torch.sort(h @ w["router"].T, dim=-1, descending=True)[0]
        clear = torch.ones(n, dtype=torch.bool) if top == E else (z[:, top - 1] - z[:, top]) > 1e-2
        assert clear.float().mean() > 0.6
        close(y.cpu()[clear], want[clear], dtype)
    if dev.type == "cuda":
        check(dev)


@variant_param
def test_routing_weights_ties_and_unused_experts(env):
    """Every token to the same experts (the others get no row); equal scores go to the lower index; weights are the scores."""
    dev, dtype = env
    n, E, width, ff = 300, 9, 16, 16
    up = torch.zeros(E, ff, width, dtype=dtype)
    down = torch.zeros(E, width, ff, dtype=dtype)
    for e in range(E):
        up[e] = torch.eye(ff)
        down[e] = (e + 1) * torch.eye(width)
    h = (torch.arange(n)[:, None] % 7 - 3).float().expand(n, width).contiguous().to(dtype)
    logits = torch.full((n, E), -1.0)
    logits[:, 4] = 2.0
    logits[:, 6] = 2.0
    logits[:, 2] = 0.5
    out, row, weight = L.routed_experts(h.to(dev), logits.to(dev), up.to(dev), down.to(dev), 3, "relu_squared", L.RouterRule(), ff, width)
    s = torch.softmax(logits.double(), -1)
    close(weight, s[:, [4, 6, 2]], torch.float32)
    relu2 = h.double().clamp(min=0) ** 2
    for k, e in enumerate((4, 6, 2)):
        close(out[row[:, k].long()][:, :width], (e + 1) * relu2, dtype)
    assert len(set(row.view(-1).tolist())) == 3 * n
    _, _, weight = L.routed_experts(h.to(dev), logits.to(dev), up.to(dev), down.to(dev), 3, "relu_squared", L.RouterRule(renormalize=True), ff, width)
    close(weight.sum(-1), torch.ones(n), torch.float32)
    # all scores equal
    _, _, weight = L.routed_experts(h.to(dev), torch.zeros(n, E, device=dev), up.to(dev), down.to(dev), 2, "none", L.RouterRule(), ff, width)
    close(weight, torch.full((n, 2), 1 / 9), torch.float32)
