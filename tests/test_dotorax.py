"""Dotorax models against the plain oracle (``dotorax_oracle.py``): whole prompts, decoding, portions, batches of unequal requests, slots
that are used again, rows in a ring, keys and values of another layer, generation, loading. Every case runs on the CPU restatement and,
marked ``gpu``, on the kernels."""
import functools
import io
import json

import pytest
import torch

import dotorax_oracle as oracle
from keys_values_b200.config import Config
from keys_values_b200.generate.base import batched_generate_fn, generate
from keys_values_b200.generate.decode_graph import Decoder
from keys_values_b200.kvcache.factory import KVCacheFactory
from keys_values_b200.kvcache.grouped import BorrowedKVCache, GroupedKVCache
from keys_values_b200.kvcache.layer_cache import SideBySideCache
from keys_values_b200.kvcache.recurrent import GatedLinearCache
from keys_values_b200.long_context import LongContextInferenceModel
from keys_values_b200.models.head_model import CrossEntropyOnLogits
from keys_values_b200.models.layered import LayeredGPT
from keys_values_b200.models.registry import create_model, default_cache_name
from keys_values_b200.ops.layers import RowPlan
from keys_values_b200.tools.trace_run import TraceRunner, load_model, run

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
device_param = pytest.mark.parametrize("device", DEVICES)
dtype_param = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])

# rms error of logits relative to their rms. In bf16 a few positions may be over it, none three times: norms of heads whose products
# nearly cancel scale their rounding up
TOLERANCE = {torch.float32: 2e-4, torch.bfloat16: 5e-2}

A, P, R, dense = oracle.attention_layer, oracle.parallel_layer, oracle.gla_layer, oracle.dense
MODELS = {
    # all kinds of mixers, one layer without a feed-forward, two layers over the first one's keys
    "mixed": oracle.content([A(mlp=dense()), R(mlp=dense(ff=20, limit=0.4)), A(kv_from=0, scale=0.3, mlp=dense()), P(mlp=dense(limit=3.0)),
                             R(heads=2, dim=24, vdim=32, tau=16.0), A(kv_from=0, mlp=dense()),
                             P(heads=6, kv_heads=3, dim=16, vdim=24, dims=16, size=5, pool=7, width=64, blocks=2, conv=4, mlp=dense(ff=36))], positions=700),
    # sizes that no vector width divides
    "odd": oracle.content([P(heads=3, kv_heads=1, dim=7, vdim=9, dims=4, size=4, pool=3, width=21, blocks=7, conv=2, mlp=dense(ff=13)),
                           R(heads=1, dim=11, vdim=13, tau=1.0, mlp=dense(ff=15)), A(heads=3, kv_heads=1, dim=7, vdim=5, dims=4),
                           A(heads=3, kv_heads=1, dim=7, vdim=5, dims=4, kv_from=2, mlp=dense(ff=7))], width=31, vocab=43, taps=2, mult=1.3),
    # one of everything
    "one": oracle.content([R(heads=1, dim=8, vdim=8, tau=2.0, mlp=dense(ff=1)), A(heads=1, kv_heads=1, dim=8, vdim=8, dims=2),
                           P(heads=1, kv_heads=1, dim=8, vdim=16, dims=2, size=1, pool=1, width=8, blocks=1, conv=1, mlp=dense(ff=8))], width=24, taps=1, mult=1.0),
    # sizes of the kernels' tiles
    "tiles": oracle.content([A(heads=24, kv_heads=1, dim=16, vdim=16, dims=16, mlp=dense(ff=64)), R(heads=2, dim=64, vdim=128, tau=16.0),
                             P(heads=8, kv_heads=8, dim=16, vdim=32, dims=8, size=64, pool=16, width=128, blocks=4, conv=4)], width=64, taps=4),
}


@functools.lru_cache(maxsize=None)
def weights(name, seed=0):
    return oracle.tensors(MODELS[name], seed)


@functools.lru_cache(maxsize=None)
def truth(name, tokens):
    """Oracle logits and streams, once per model and prompt."""
    return oracle.forward(list(tokens), weights(name), MODELS[name])


def build(tmp_path, name, device, dtype):
    """The model and a function from tokens to the oracle's logits."""
    c, w = MODELS[name], weights(name)
    oracle.write_model(tmp_path / "m", c, w)
    return c, w, load_model(tmp_path / "m", dtype, torch.device(device)), lambda t: truth(name, tuple(t))[0]


def give_caches(model, batch, length=512):
    p = model.lm_head.weight
    model.assign_kv_caches(KVCacheFactory.create(model, default_cache_name(model.config), batch, length, device=p.device, dtype=p.dtype))
    return model


def tokens_of(n, c, seed=1):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).square().mean().sqrt() / want.square().mean().sqrt())


def assert_close(got, want, dtype):
    """Every position."""
    errors = [rel(g, w) for g, w in zip(got, want)]
    tol = TOLERANCE[dtype]
    assert len(got) == len(want) and max(errors) < (tol if dtype == torch.float32 else 3 * tol), errors
    assert sum(e > tol for e in errors) <= 1 + (0.0 if dtype == torch.float32 else 0.05) * len(errors), errors


def check(device):
    from keys_values_b200 import ops

    ops.check_status(torch.device(device))


@torch.inference_mode()
def feed(model, tokens, sizes):
    """Logits of every position, the tokens fed in portions of ``sizes`` (the last one repeats)."""
    model.reset()
    out, at, i = [], 0, 0
    dev = model.lm_head.weight.device
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(model(torch.tensor([tokens[at : at + n]], device=dev))[0])
        at, i = at + n, i + 1
    return torch.cat(out)


# ------------------------------------------------------------------------------------------ whole model against the oracle
@device_param
@dtype_param
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_matches_oracle(tmp_path, name, dtype, device):
    c, w, model, want = build(tmp_path, name, device, dtype)
    give_caches(model, 1)
    toks = tokens_of(45, c)
    streams = []
    model.set_start_of_layer_hook(lambda x, i: streams.append(x.clone()))
    got = feed(model, toks, [len(toks)])
    after = truth(name, tuple(toks))[1]
    assert len(streams) == len(after) + 1 == model.n_runs + 1
    for s, a in zip(streams[1:], after):
        assert s.dtype == torch.float32
        assert_close(s[0], a, dtype)
    assert got.dtype == torch.float32
    assert_close(got, want(toks), dtype)
    check(device)


@device_param
@pytest.mark.parametrize("name", list(MODELS))
@pytest.mark.parametrize("sizes", [[1], [2], [3], [1, 7], [20, 1], [17, 2, 1, 5, 1, 1, 11]])
def test_portions_and_single_tokens_match_oracle(tmp_path, name, sizes, device):
    c, w, model, want = build(tmp_path, name, device, torch.float32)
    give_caches(model, 1)
    toks = tokens_of(41, c, seed=2)
    assert_close(feed(model, toks, sizes), want(toks), torch.float32)


@device_param
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_long_prompt_across_tiles_and_chunks(tmp_path, name, device):
    """Prompts over several tiles of keys and chunks of the recurrence, whole, in portions that end beside the borders, and
    with the last tokens decoded."""
    dtype = torch.bfloat16 if device == "cuda" else torch.float32
    c, w, model, want = build(tmp_path, name, device, dtype)
    give_caches(model, 1)
    toks = tokens_of(280, c, seed=4)
    for sizes in ([280], [127, 2, 128, 23], [256, 1], [129, 63, 65, 23]):
        assert_close(feed(model, toks, sizes), want(toks), dtype)
    check(device)


@device_param
@dtype_param
def test_unequal_batch_equals_each_alone(tmp_path, dtype, device):
    """Prompts of different lengths in one batch, then decoded together; the shorter ones leave earlier; then others
    start while some go on, in slots that have been used before."""
    c, w, model, _ = build(tmp_path, "mixed", device, dtype)
    reqs = {k: tokens_of(n, c, seed=n) for k, n in dict(a=1, b=7, c=153, d=20, e=12).items()}
    alone = {}
    give_caches(model, 1)
    for k, toks in reqs.items():
        alone[k] = feed(model, toks, [len(toks)])
    runner = TraceRunner(model, 512)
    runner._reserve(4)

    def step(parts, end=()):
        entries = [dict(id=k, tokens=reqs[k][lo:hi], want=list(range(hi - lo))) for k, lo, hi in parts]
        out = runner.step(entries, list(end))
        assert_close(out, torch.cat([alone[k][lo:hi] for k, lo, hi in parts]), dtype)

    step([("a", 0, 1), ("b", 0, 4), ("c", 0, 146)], end=["a"])
    step([("b", 4, 5), ("c", 146, 147)])
    step([("b", 5, 6), ("c", 147, 148)])
    step([("c", 148, 149), ("b", 6, 7)], end=["b"])  # another order of the rows
    assert model.sequences.live() == 1
    step([("d", 0, 13), ("c", 149, 150)])            # d starts in a freed slot, next to a single token
    step([("d", 13, 18), ("e", 0, 2), ("c", 150, 153)], end=["c"])
    for t in range(2):
        step([("e", 2 + t, 3 + t), ("d", 18 + t, 19 + t)])
    step([("e", 4, 12)], end=["d", "e"])
    assert model.sequences.live() == 0
    check(device)


@device_param
@dtype_param
def test_long_decoding(tmp_path, dtype, device):
    """Single-token steps through the decoder (captured on a GPU), two sequences at different positions: windows, chunks and kept tokens
    pass over decoded tokens."""
    c, w, model, want = build(tmp_path, "mixed", device, dtype)
    give_caches(model, 2)
    a, b = tokens_of(130, c, seed=5), tokens_of(130, c, seed=6)
    dev = model.lm_head.weight.device
    got = ([], [])
    with torch.inference_mode():
        model(torch.tensor([a[:4], b[:2] + [0, 0]], device=dev), counts=[4, 2])
        dec = Decoder(model, 2, use_graph=device == "cuda")
        for t in range(120):
            out = dec(torch.tensor([[a[4 + t]], [b[2 + t]]], device=dev))[:, 0]
            got[0].append(out[0].clone())
            got[1].append(out[1].clone())
        if device == "cuda":
            assert dec.graph is not None and dec.graph.steps == 118
    assert_close(got[0], want(a)[4:124], dtype)
    assert_close(got[1], want(b)[2:122], dtype)
    assert model.sequences.pos_host == [124, 122] and model.sequences.pos.tolist() == [124, 122]
    check(device)


@device_param
def test_rows_without_tokens_keep_their_state(tmp_path, device):
    c, w, model, want = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 2)
    a, b = tokens_of(12, c, seed=7), tokens_of(12, c, seed=8)
    dev = model.lm_head.weight.device
    with torch.inference_mode():
        model(torch.tensor([a[:6], b[:6]], device=dev))
        model(torch.tensor([a[6:9], [0, 0, 0]], device=dev), counts=[3, 0])
        model(torch.tensor([[0], b[6:7]], device=dev), counts=[0, 1])
        out = model(torch.tensor([a[9:12], b[7:10]], device=dev))
    assert_close(out[0], want(a)[9:12], torch.float32)
    assert_close(out[1], want(b)[7:10], torch.float32)


# ------------------------------------------------------------------------------------------------------ the caches
@device_param
@dtype_param
def test_windows_keep_a_ring_of_tokens_and_all_blocks(tmp_path, monkeypatch, dtype, device):
    """A cache far longer than the windows takes rows for these, a pass and the blocks only; prompts in portions and decoding use the tokens'
    rows again and again."""
    monkeypatch.setattr(GroupedKVCache, "max_pass", 40)
    c, w, model, want = build(tmp_path, "mixed", device, dtype)
    give_caches(model, 1, length=650)
    plans = {i: x.parts[0].plan for i, x in enumerate(model.get_kv_caches()) if isinstance(x, SideBySideCache)}
    assert plans == {3: RowPlan(256, 128), 6: RowPlan(128, 128)}
    toks = tokens_of(330, c, seed=9)
    got = feed(model, toks, [40] * 6 + [31, 1, 1, 1, 2, 35, 1])
    assert_close(got, want(toks), dtype)
    held = model.get_kv_caches()[3].token_positions()[0, 0]
    assert sorted(held.tolist()) == list(range(202, 330))
    with torch.inference_mode(), pytest.raises(IndexError, match="smaller portions"):
        model(torch.tensor([tokens_of(130, c)], device=got.device))
    check(device)


@device_param
@dtype_param
def test_keys_of_another_layer(tmp_path, dtype, device):
    """Layers that share keys and values hold none of their own; what they read is what the first one wrote for this sequence."""
    c, w, model, want = build(tmp_path, "mixed", device, dtype)
    give_caches(model, 2)
    caches = model.get_kv_caches()
    assert [i for i, x in enumerate(caches) if isinstance(x, BorrowedKVCache)] == [2, 5]
    a, b = tokens_of(60, c, seed=11), tokens_of(60, c, seed=12)
    dev = model.lm_head.weight.device
    with torch.inference_mode():
        out = model(torch.tensor([a[:50], b[:30] + [0] * 20], device=dev), counts=[50, 30])
        nxt = model(torch.tensor([[a[50]], [b[30]]], device=dev))
    for i in (2, 5):
        assert caches[i].size_estimate()[0] == 0 and caches[i].allocate(dev, dtype)[0] is caches[0].rows
    assert_close(torch.cat((out[0], nxt[0])), want(a)[:51], dtype)
    assert_close(torch.cat((out[1, :30], nxt[1])), want(b)[:31], dtype)
    check(device)


@device_param
def test_cache_refuses_more_than_it_holds(tmp_path, device):
    c, w, model, want = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 1, length=12)
    toks = tokens_of(13, c)
    got = feed(model, toks[:12], [5, 1])
    assert_close(got, want(toks)[:12], torch.float32)
    with torch.inference_mode(), pytest.raises(IndexError, match="exceed the cache of 12"):
        model(torch.tensor([toks[12:]], device=got.device))


@device_param
def test_position_table_bounds_the_context(tmp_path, device):
    c, w, model, want = build(tmp_path, "odd", device, torch.float32)
    give_caches(model, 1, length=500)
    toks = tokens_of(400, c)
    got = feed(model, toks, [399, 1])
    assert_close(got[-1:], want(toks)[-1:], torch.float32)
    with torch.inference_mode(), pytest.raises((IndexError, ValueError), match="exceed|max_seq_length"):
        model(torch.tensor([toks[:1]], device=got.device))
    model.max_seq_length = 1000
    with torch.inference_mode(), pytest.raises(IndexError, match="table of 400 positions"):
        model(torch.tensor([toks[:1]], device=got.device))


def test_caches_fit_their_layers():
    model = create_model(Config.from_name("tiny-dotorax"))
    for name in ("h2o-default", "latent-default"):
        with pytest.raises(ValueError):
            KVCacheFactory.create(model, name, 1, 64)
    model.set_kv_caches(2, max_seq_length=100)
    caches = model.get_kv_caches()
    assert [type(x) for x in caches] == [GroupedKVCache, GatedLinearCache, BorrowedKVCache, SideBySideCache]
    s, t = caches[0].shape, caches[1].shape
    assert caches[0].size_estimate()[0] == 2 * 100 * s.kv_heads * s.row * 32
    assert caches[1].size_estimate()[0] == 2 * t.heads * t.np * t.vdp * 32
    a, r = (x.shape for x in caches[3].parts)
    assert caches[3].size_estimate()[0] == 2 * 32 * ((128 + 128) * a.kv_heads * a.row + r.channels * (1 + r.taps))
    model.config.layers[1]["mixer"]["dim"] += 8
    other = create_model(model.config)
    with pytest.raises(ValueError, match="needs a"):
        create_model(Config.from_name("tiny-dotorax")).assign_kv_caches(KVCacheFactory.create(other, "layered-default", 1, 64))
    with pytest.raises(NotImplementedError, match="inference"):
        model(torch.zeros(1, 3, dtype=torch.int64))


def test_clone_keeps_the_state(tmp_path):
    c, w, model, want = build(tmp_path, "mixed", "cpu", torch.float32)
    give_caches(model, 1)
    toks = tokens_of(6, c)
    with torch.inference_mode():
        model(torch.tensor([toks[:5]]))
        other = model.clone()
        assert other.sequences is not model.sequences and other.get_kv_caches()[0].sequences is other.sequences
        got = feed(other, toks, [6])
        assert_close(got, want(toks), torch.float32)
        assert_close(model(torch.tensor([toks[5:]]))[0], want(toks)[5:], torch.float32)


# --------------------------------------------------------------------------------------------------- generation
@device_param
@pytest.mark.parametrize("chunk", [4, 1024])
def test_greedy_generation_matches_oracle(tmp_path, chunk, device):
    c, w, model, _ = build(tmp_path, "mixed", device, torch.float32)
    dev = model.lm_head.weight.device
    prompt, n_new = tokens_of(19, c, seed=8), 5
    want = oracle.greedy(prompt, n_new, w, c)
    give_caches(model, 1, length=len(prompt) + n_new)
    got = generate(model, torch.tensor(prompt, device=dev), len(prompt) + n_new, prompt_chunksize=chunk, temperature=0.0, include_prompt=False)
    assert got.view(-1).tolist() == want
    # prompts of different lengths in one batch
    prompts = [prompt[:1], prompt, prompt[3:14]]
    give_caches(model, 3, length=64)
    rows = list(batched_generate_fn(model, [torch.tensor(p, device=dev) for p in prompts], len(prompt) + n_new, prompt_chunksize=chunk,
                                    sample_args=dict(temperature=0.0), include_prompt=False))
    for b, p in enumerate(prompts):
        assert [int(r[b]) for r in rows] == oracle.greedy(p, n_new, w, c), b


@device_param
def test_chunked_prefill_of_unequal_rows_in_several_cells(tmp_path, monkeypatch, device):
    """Cells end before, inside and after the rows' last tokens."""
    c, w, model, want = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 3)
    monkeypatch.setattr(LayeredGPT, "max_pass_tokens", lambda self, batch: 8)
    lengths = [30, 5, 16]
    toks = [tokens_of(n, c, seed=20 + n) for n in lengths]
    idx = torch.tensor([t + [0] * (30 - len(t)) for t in toks], device=model.lm_head.weight.device)
    lcm = LongContextInferenceModel(model, CrossEntropyOnLogits(model.config), chunk_size=4)
    logits = lcm(idx, None, lengths=lengths)
    assert len(lcm.cells) == 4
    for b, t in enumerate(toks):
        assert_close(logits[b], want(t)[-1:], torch.float32)


def test_generate_command_with_token_ids(tmp_path, capsys):
    c, w, _, _ = build(tmp_path, "odd", "cpu", torch.float32)
    prompt = tokens_of(6, c)
    from keys_values_b200.__main__ import main

    main(["generate", str(tmp_path / "m"), "--prompt-tokens", ",".join(map(str, prompt)), "--max_new_tokens", "4", "--temperature", "0.0",
          "--precision", "32-true", "--device", "cpu"])
    assert capsys.readouterr().out.strip() == ",".join(map(str, oracle.greedy(prompt, 4, w, c)))


@device_param
def test_trace_replay_program(tmp_path, device):
    c, w, _, want = build(tmp_path, "mixed", device, torch.float32)
    a, b = tokens_of(14, c, seed=3), tokens_of(9, c, seed=4)
    steps = [
        dict(step=0, entries=[dict(id="x", tokens=a[:10], want=[0, 9]), dict(id="y", tokens=b[:8], want=[7])], end=[]),
        dict(step=1, entries=[dict(id="x", tokens=a[10:11], want=[]), dict(id="y", tokens=b[8:], want=[])], end=["y"]),
        dict(step=2, entries=[dict(id="x", tokens=a[11:12], want=[0])], end=["x"]),
        dict(step=3, entries=[dict(id="x", tokens=b[:5], want=[4])], end=["x"]),  # a new request of the same name
    ]
    report = io.StringIO()
    run(tmp_path / "m", "float32", tmp_path / "out", 64, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), report, torch.device(device))
    assert report.getvalue().split("\n")[:4] == [f"done {i}" for i in range(4)]
    la, lb = want(a), want(b)
    for i, rows in {0: torch.stack((la[0], la[9], lb[7])), 2: la[11:12], 3: lb[4:5]}.items():
        got = torch.frombuffer(bytearray((tmp_path / "out" / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, c["vocab"])
        assert_close(got, rows, torch.float32)


# --------------------------------------------------------------------------------------- configuration and loading
def test_config_reader_and_registry(tmp_path):
    c, w, model, _ = build(tmp_path, "mixed", "cpu", torch.bfloat16)
    cfg = Config.from_checkpoint(tmp_path / "m")
    assert isinstance(model, LayeredGPT) and cfg.architecture == "Dotorax" and cfg.n_layer == 7 and cfg.norm_eps == c["norm"]["eps"]
    assert (cfg.input_conv, cfg.residual_mult, cfg.block_size) == (c["canon"]["taps"], c["residual_mult"], c["max_positions"])
    assert [x["mixer"]["kind"] for x in cfg.layers] == ["grouped_attention", "gated_linear_attention", "grouped_attention", "side_by_side",
                                                        "gated_linear_attention", "grouped_attention", "side_by_side"]
    assert cfg.layers[2]["mixer"]["kv_from"] == 0 and "kv_from" not in cfg.layers[0]["mixer"] and cfg.layers[4]["mlp"] is None
    assert cfg.layers[1]["mixer"]["rank"] == 5  # known from the weights only
    assert default_cache_name(cfg) == "layered-default"
    # the config survives a round trip through model_config.yaml
    cfg.save(tmp_path / "model_config.yaml")
    assert Config.from_file(tmp_path / "model_config.yaml") == cfg
    assert isinstance(create_model(Config.from_name("tiny-dotorax")), LayeredGPT)


@pytest.mark.parametrize("change", ["missing", "extra", "shape", "keys"])
def test_loading_checks_every_tensor(tmp_path, change):
    c, w = MODELS["mixed"], dict(weights("mixed"))
    if change == "missing":
        w.pop("l3.mix.left.temp")
    elif change == "extra":
        w["l1.mix.q.b"] = w["l1.mix.a2.b"]
    elif change == "keys":  # of a layer that has none
        w["l2.mix.k"] = w["l0.mix.k"]
    else:
        w["l0.mix.g"] = w["l0.mix.g"][1:]
    oracle.write_model(tmp_path / "m", c, w)
    with pytest.raises((KeyError, RuntimeError)):
        load_model(tmp_path / "m", torch.float32, torch.device("cpu"))


def test_unknown_and_impossible_parts_are_refused(tmp_path):
    def config(*layers):
        (tmp_path / "config.json").write_text(json.dumps(oracle.content(list(layers))))
        return Config.from_checkpoint(tmp_path)

    for layer in (dict(A(), type="mamba2"), dict(A(), mlp={"kind": "moe", "ff": 8})):
        with pytest.raises(ValueError, match="not part of the design"):
            config(layer)
    for layers in ((A(heads=5),), (A(dims=15),), (A(scale=0.0),), (A(kv_from=0),), (R(), A(kv_from=0)), (A(), A(kv_from=0, dim=24)),
                   (A(), A(kv_from=0), A(kv_from=1)), (A(), A(kv_from=0, base=901.0)), (P(blocks=5),), (R(tau=0.0),), (P(pool=-1),), (A(mlp=dense(limit=0.0)),)):
        with pytest.raises((ValueError, AssertionError)):
            create_model(config(*layers))
