"""Models described layer by layer against the plain oracle (``layered_oracle.py``): whole prompts, decoding, portions,
batches of unequal requests, slots that are used again, windows, generation, loading. Every case runs on the CPU restatement
and, marked ``gpu``, on the kernels."""
import io
import json

import pytest
import torch

import layered_oracle as oracle
from keys_values_b200.config import Config
from keys_values_b200.generate.base import batched_generate_fn, generate, main as generate_main
from keys_values_b200.generate.decode_graph import Decoder
from keys_values_b200.kvcache.factory import KVCacheFactory
from keys_values_b200.kvcache.latent import LatentKVCache
from keys_values_b200.long_context import LongContextInferenceModel
from keys_values_b200.models.head_model import CrossEntropyOnLogits
from keys_values_b200.models.layered import LayeredGPT
from keys_values_b200.models.model import GPT
from keys_values_b200.models.registry import create_model, default_cache_name
from keys_values_b200.tools.trace_run import TraceRunner, load_model, run

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
device_param = pytest.mark.parametrize("device", DEVICES)

# rms error of logits relative to their rms
TOLERANCE = {torch.float32: 2e-4, torch.bfloat16: 4e-2}

MODELS = {
    # layers that differ in everything, one without a feed-forward
    "mixed": oracle.content([oracle.layer(window=9), oracle.layer(heads=2, dim=20, rot_dim=8, vdim=12, kv_rank=33, window=5, base=90.0, experts=4, top=4, ff=10),
                             oracle.layer(window=16, experts=0), oracle.layer(heads=1, window=3, experts=3, top=1, scale=0.4)]),
    # sizes that no vector width divides
    "odd": oracle.content([oracle.layer(heads=3, dim=5, rot_dim=2, vdim=3, kv_rank=7, window=4, experts=3, top=2, ff=9),
                           oracle.layer(heads=2, dim=3, rot_dim=6, vdim=9, kv_rank=11, window=7, experts=1, top=1, ff=5)], width=31, vocab=43),
    # a window of one token
    "one": oracle.content([oracle.layer(window=1), oracle.layer(window=2)], width=24),
}


def build(tmp_path, name, device, dtype, seed=0):
    c = MODELS[name] if isinstance(name, str) else name
    w = oracle.tensors(c, seed)
    oracle.write_model(tmp_path / "m", c, w)
    return c, w, load_model(tmp_path / "m", dtype, torch.device(device))


def give_caches(model, batch, length=4096):
    p = model.lm_head.weight
    model.assign_kv_caches(KVCacheFactory.create(model, "latent-default", batch, length, device=p.device, dtype=p.dtype))
    return model


def tokens_of(n, c, seed=1):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return float((got - want).square().mean().sqrt() / want.square().mean().sqrt())


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
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_matches_oracle(tmp_path, name, dtype, device):
    c, w, model = build(tmp_path, name, device, dtype)
    give_caches(model, 1)
    toks = tokens_of(45, c)
    streams = []
    model.set_start_of_layer_hook(lambda x, i: streams.append(x.clone()))
    got = feed(model, toks, [len(toks)])
    want, after = oracle.forward(toks, w, c)
    for s, a in zip(streams[1:], after):
        assert s.dtype == torch.float32 and rel(s[0], a) < TOLERANCE[dtype]
    assert rel(got, want) < TOLERANCE[dtype]
    # token by token, every position
    tol = TOLERANCE[dtype] * (1 if dtype == torch.float32 else 8)  # bf16: a close call of a router may show at one position
    errors = [rel(got[t], want[t]) for t in range(len(toks))]
    assert max(errors) < tol, errors


@device_param
@pytest.mark.parametrize("name", list(MODELS))
@pytest.mark.parametrize("sizes", [[1], [2], [3], [1, 7], [20, 1], [17, 2, 1, 5, 1, 1, 11]])
def test_portions_and_single_tokens_match_oracle(tmp_path, name, sizes, device):
    c, w, model = build(tmp_path, name, device, torch.float32)
    give_caches(model, 1)
    toks = tokens_of(41, c, seed=2)
    want, _ = oracle.forward(toks, w, c)
    got = feed(model, toks, sizes)
    errors = [rel(got[t], want[t]) for t in range(len(toks))]
    assert max(errors) < TOLERANCE[torch.float32], errors


@device_param
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_batch_equals_each_alone(tmp_path, dtype, device):
    """Prompts of different lengths in one batch, then decoded together; the shorter ones leave earlier; then others
    start while some go on, in slots that have been used before."""
    c, w, model = build(tmp_path, "mixed", device, dtype)
    reqs = {k: tokens_of(n, c, seed=n) for k, n in dict(a=1, b=7, c=33, d=20, e=12).items()}
    alone = {}
    give_caches(model, 1)
    for k, toks in reqs.items():
        alone[k] = feed(model, toks, [len(toks)])
    runner = TraceRunner(model, 4096)
    runner._reserve(4)

    def step(parts, end=()):
        entries = [dict(id=k, tokens=reqs[k][lo:hi], want=list(range(hi - lo))) for k, lo, hi in parts]
        out = runner.step(entries, list(end))
        want = torch.cat([alone[k][lo:hi] for k, lo, hi in parts])
        assert rel(out, want.cpu()) < TOLERANCE[dtype]
        assert max(rel(o, x.cpu()) for o, x in zip(out, want)) < TOLERANCE[dtype] * (1 if dtype == torch.float32 else 8)

    step([("a", 0, 1), ("b", 0, 4), ("c", 0, 26)], end=["a"])
    step([("b", 4, 5), ("c", 26, 27)])
    step([("b", 5, 6), ("c", 27, 28)])
    step([("c", 28, 29), ("b", 6, 7)], end=["b"])  # another order of the rows
    assert model.sequences.live() == 1
    step([("d", 0, 13), ("c", 29, 30)])            # d starts in a freed slot, next to a single token
    step([("d", 13, 18), ("e", 0, 2), ("c", 30, 33)], end=["c"])
    for t in range(2):
        step([("e", 2 + t, 3 + t), ("d", 18 + t, 19 + t)])
    step([("e", 4, 12)], end=["d", "e"])
    assert model.sequences.live() == 0


@device_param
def test_long_decoding_wraps_every_ring(tmp_path, device):
    """Single-token steps through the decoder (captured on a GPU) far beyond all windows."""
    c, w, model = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 2)
    a, b = tokens_of(90, c, seed=5), tokens_of(90, c, seed=6)
    want = [oracle.forward(t, w, c)[0] for t in (a, b)]
    dev = model.lm_head.weight.device
    with torch.inference_mode():
        idx = torch.tensor([a[:4], b[:2] + [0, 0]], device=dev)
        model(idx, counts=[4, 2])
        dec = Decoder(model, 2, use_graph=device == "cuda")
        for t in range(80):
            out = dec(torch.tensor([[a[4 + t]], [b[2 + t]]], device=dev))[:, 0]
            assert rel(out[0], want[0][4 + t]) < 2e-4 and rel(out[1], want[1][2 + t]) < 2e-4, t
        if device == "cuda":
            assert dec.graph is not None and dec.graph.steps == 78
    assert model.get_kv_caches()[0].input_pos == 84 and model.sequences.pos_host == [84, 82]
    assert model.sequences.pos.tolist() == [84, 82]
    held = model.get_kv_caches()[0].token_positions()[0, 0].tolist()
    assert sorted(held) == list(range(75, 84))


@device_param
def test_ring_shorter_than_window_refuses_more(tmp_path, device):
    c, w, model = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 1, length=12)  # one layer wants 16
    toks = tokens_of(13, c)
    want, _ = oracle.forward(toks[:12], w, c)
    got = feed(model, toks[:12], [5, 1])
    assert rel(got, want) < 2e-4
    with torch.inference_mode(), pytest.raises(IndexError, match="exceed the cache of 12"):
        model(torch.tensor([toks[12:]], device=got.device))


# --------------------------------------------------------------------------------------------------- generation
@device_param
@pytest.mark.parametrize("chunk", [4, 1024])
def test_greedy_generation_matches_oracle(tmp_path, chunk, device):
    c, w, model = build(tmp_path, "mixed", device, torch.float32)
    dev = model.lm_head.weight.device
    prompt, n_new = tokens_of(19, c, seed=8), 8
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


def test_generation_yields_prompts_of_unequal_rows(tmp_path):
    c, w, model = build(tmp_path, "one", "cpu", torch.float32)
    give_caches(model, 2)
    rows = list(batched_generate_fn(model, [torch.tensor([1, 2, 3]), torch.tensor([4])], 5, include_prompt=True))
    assert [None if r is None else int(r) for r in [x[1] for x in rows[:3]]] == [4, None, None]
    assert [int(x[0]) for x in rows[:3]] == [1, 2, 3] and len(rows) == 5


@device_param
def test_chunked_prefill_of_unequal_rows_in_several_cells(tmp_path, monkeypatch, device):
    """Cells end before, inside and after the rows' last tokens."""
    c, w, model = build(tmp_path, "mixed", device, torch.float32)
    give_caches(model, 3)
    monkeypatch.setattr(LayeredGPT, "max_pass_tokens", lambda self, batch: 8)
    lengths = [30, 5, 16]
    toks = [tokens_of(n, c, seed=20 + n) for n in lengths]
    idx = torch.tensor([t + [0] * (30 - len(t)) for t in toks], device=model.lm_head.weight.device)
    lcm = LongContextInferenceModel(model, CrossEntropyOnLogits(model.config), chunk_size=4)
    logits = lcm(idx, None, lengths=lengths)
    assert len(lcm.cells) == 4
    for b, t in enumerate(toks):
        assert rel(logits[b, 0], oracle.forward(t, w, c)[0][-1]) < 2e-4
    # the loss over target tokens of equal rows
    loss = lcm(idx[:, :16], idx[:, 1:17])
    ref = torch.log_softmax(oracle.forward(idx[0, :16].tolist(), w, c)[0], -1)
    nll = -ref[torch.arange(16), idx[0, 1:17].cpu()].mean()
    assert abs(float(loss[0]) - float(nll)) < 1e-3


def test_generate_command_with_token_ids(tmp_path, capsys):
    c, w, _ = build(tmp_path, "mixed", "cpu", torch.float32)
    prompt = tokens_of(6, c)
    from keys_values_b200.__main__ import main

    main(["generate", str(tmp_path / "m"), "--prompt-tokens", ",".join(map(str, prompt)), "--max_new_tokens", "4", "--temperature", "0.0",
          "--precision", "32-true", "--device", "cpu"])
    assert capsys.readouterr().out.strip() == ",".join(map(str, oracle.greedy(prompt, 4, w, c)))
    with pytest.raises(ValueError, match="prompt_tokens"):
        generate_main(str(tmp_path / "m"), prompt_tokens="1,999", device="cpu", precision="32-true")


@device_param
def test_trace_replay_program(tmp_path, device):
    c, w, _ = build(tmp_path, "mixed", device, torch.float32)
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
    la, lb = oracle.forward(a, w, c)[0], oracle.forward(b, w, c)[0]
    for i, want in {0: torch.stack((la[0], la[9], lb[7])), 2: la[11:12], 3: lb[4:5]}.items():
        got = torch.frombuffer(bytearray((tmp_path / "out" / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, c["vocab"])
        assert rel(got, want) < 2e-4
    assert not (tmp_path / "out" / "1.f32").exists()


# ------------------------------------------------------------------------------- configuration, loading, slots
def test_config_reader_and_registry(tmp_path):
    c, w, model = build(tmp_path, "mixed", "cpu", torch.bfloat16)
    cfg = Config.from_checkpoint(tmp_path / "m")
    assert isinstance(model, LayeredGPT) and cfg.architecture == "Mezilix" and cfg.n_layer == 4 and cfg.norm_eps == c["norm"]["eps"]
    assert cfg.layers[2]["mlp"] is None and cfg.layers[1]["mixer"]["kv_rank"] == 33 and cfg.layers[3]["mixer"]["scale"] == 0.4
    assert torch.equal(model.state_dict()["transformer.h.1.mlp.down"][3], w["l1.mlp.e3.down"])
    assert default_cache_name(cfg) == "latent-default" and default_cache_name(Config.from_name("tiny-gpt")) == "h2o-default"
    # the config survives a round trip through model_config.yaml
    cfg.save(tmp_path / "model_config.yaml")
    again = Config.from_file(tmp_path / "model_config.yaml")
    assert again == cfg
    named = Config.from_name("tiny-mezilix")
    assert isinstance(create_model(named), LayeredGPT)
    (tmp_path / "other").mkdir()
    (tmp_path / "other" / "config.json").write_text(json.dumps(dict(architecture="Nothing")))
    with pytest.raises(ValueError, match="not registered"):
        Config.from_checkpoint(tmp_path / "other")


@pytest.mark.parametrize("change", ["missing", "extra", "shape"])
def test_loading_checks_every_tensor(tmp_path, change):
    c = MODELS["one"]
    w = oracle.tensors(c)
    if change == "missing":
        w.pop("l1.mlp.e2.up")
    elif change == "extra":
        w["l0.mix.gate"] = w["l0.shift"]
    else:
        w["l0.mix.uk"] = w["l0.mix.uk"][:, 1:]
    oracle.write_model(tmp_path / "m", c, w)
    with pytest.raises((KeyError, RuntimeError)):
        load_model(tmp_path / "m", torch.float32, torch.device("cpu"))


def test_caches_fit_their_models():
    layered = create_model(Config.from_name("tiny-mezilix"))
    with pytest.raises(ValueError, match="does not fit"):
        KVCacheFactory.create(layered, "h2o-default", 1, 64)
    plain = create_model(Config.from_name("tiny-gpt"))
    with pytest.raises(ValueError, match="does not fit"):
        KVCacheFactory.create(plain, "latent-default", 1, 64)
    with pytest.raises(ValueError, match="describes its layers"):
        GPT(Config.from_name("tiny-mezilix"))
    with pytest.raises(ValueError, match="equal length"):
        plain(torch.zeros(2, 3, dtype=torch.int64), counts=[3, 1])
    layered.set_kv_caches(2, max_seq_length=100)
    caches = layered.get_kv_caches()
    assert all(isinstance(x, LatentKVCache) and x.ring_length == 48 and x.max_prefill_length is None for x in caches)
    assert caches[0].size_estimate()[0] == 2 * 48 * (72 + 8) * 32
    with pytest.raises(NotImplementedError, match="inference"):
        layered(torch.zeros(1, 3, dtype=torch.int64))


def test_slots_are_checked():
    layered = create_model(Config.from_name("tiny-mezilix"))
    layered.set_kv_caches(2, max_seq_length=100)
    t = layered.sequences
    a, b = t.acquire(), t.acquire()
    with pytest.raises(RuntimeError, match="in use"):
        t.acquire()
    with pytest.raises(ValueError):
        t.set_batch([a, a])
    t.release(a)
    for bad in (lambda: t.release(a), lambda: t.set_batch([a]), lambda: t.release(7)):
        with pytest.raises(ValueError):
            bad()
    t.set_batch([b])
    with pytest.raises(ValueError, match="differs"):
        t.begin(2, 4)
    with pytest.raises(ValueError, match="counts"):
        t.begin(1, 4, [5])
    assert t.acquire() == a


def test_trace_runner_checks_its_input(tmp_path):
    c, w, model = build(tmp_path, "one", "cpu", torch.float32)
    r = TraceRunner(model, 64)
    for entries in ([dict(id="a", tokens=[c["vocab"]], want=[])], [dict(id="a", tokens=[], want=[])], [dict(id="a", tokens=[1], want=[1])],
                    [dict(id="a", tokens=[1], want=[])] * 2):
        with pytest.raises(ValueError):
            r.step(entries, [])
    with pytest.raises(NotImplementedError):
        TraceRunner(create_model(Config.from_name("tiny-gpt")), 64)


def test_clone_keeps_the_state(tmp_path):
    c, w, model = build(tmp_path, "one", "cpu", torch.float32)
    give_caches(model, 1)
    toks = tokens_of(6, c)
    with torch.inference_mode():
        model(torch.tensor([toks[:5]]))
        other = model.clone()
        assert other.sequences is not model.sequences and other.get_kv_caches()[0].sequences is other.sequences
        got = feed(other, toks, [6])
        assert rel(model(torch.tensor([toks[5:]]))[0, 0], got[5].double()) < 1e-4
