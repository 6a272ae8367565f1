"""Prefill and decode throughput of a model with described layers beside the closest LitGPT-shaped model of equal size, and the
time of every kernel of the design beside the like kernel of that model, each against its roofline.

    python -m keys_values_b200.tools.layered_bench [--model Mezilix-2k] [--batch 32] [--prompt 8192] [--decode 128] [--kernels]

Random-init weights, synthetic tokens. For Mezilix the closest model has the same width, depth, heads, window and experts
(count, chosen per token, expert weights per token): grouped-query attention over a sliding window, SwiGLU experts
(``LLaMAMoE``), or a dense SwiGLU of the width that a token's chosen experts add up to. For Pazenex, Ladadra and Dotorax it has the same width,
depth, heads and key/value heads, attention in every layer and a dense SwiGLU that makes the number of weights that a token meets
equal. Kernel times are
CUDA-event medians with an L2 flush (256 MB written, another 256 MB read) before every launch.
"""
from __future__ import annotations

import argparse
import json
from pathlib import Path
from typing import Callable, Dict, List, Optional

import torch

from keys_values_b200.config import Config


def closest_config(config: Config, dense: bool = False) -> Config:
    """LitGPT-shaped model of the same size: heads of 128, all of them keys and values, the same window; expert (or dense) width
    such that a token meets the same number of feed-forward weights (three matrices instead of two)."""
    if any(x["mixer"]["kind"] != "latent_attention" for x in config.layers):
        return closest_attention_config(config)
    m, f = config.layers[0]["mixer"], config.layers[0]["mlp"]
    ff = f["ff"] * 2 // 3 // 8 * 8
    kw = dict(
        name=f"closest-to-{config.name}", block_size=1 << 17, vocab_size=config.vocab_size, padded_vocab_size=config.padded_vocab_size,
        n_layer=config.n_layer, n_embd=config.n_embd, n_head=m["n_head"], n_query_groups=m["n_head"], head_size=128, rotary_percentage=1.0,
        parallel_residual=False, bias=False, norm_class_name="RMSNorm", norm_eps=config.norm_eps, sliding_window_size=m["window"],
    )
    if dense:
        return Config(mlp_class_name="LLaMAMLP", intermediate_size=ff * f["top"], **kw)
    return Config(mlp_class_name="LLaMAMoE", intermediate_size=ff, moe_intermediate_size=ff, n_expert=f["n_expert"], n_expert_per_token=f["top"], **kw)


def mixer_weights(x: Dict, width: int) -> int:
    """Weights of the products that a token meets in a mixer."""
    if x["kind"] == "side_by_side":
        return mixer_weights(x["left"], width) + mixer_weights(x["right"], width)
    if x["kind"] == "gated_recurrence":
        return 3 * width * x["width"] + 2 * x["width"] ** 2 // x["blocks"]
    if x["kind"] == "gated_linear_attention":
        return width * (x["n_head"] * (2 * x["dim"] + 3 * x["v_dim"]) + x["rank"]) + x["rank"] * x["n_head"] * x["dim"]
    if x["kind"] == "mamba2":
        inner, bc = x["n_head"] * x["v_dim"], x["groups"] * x["state"]
        n = width * (3 * inner + 2 * bc + x["n_head"])
    elif x["kind"] == "retention":
        n = width * x["n_head"] * (2 * x["dim"] + 3 * x["v_dim"])
    else:
        maps = 1 if x.get("differential") is None else 2
        H, G = x["n_head"], x["n_kv_head"]
        n = width * ((H + G) * maps * x["dim"] + H * x["v_dim"])
        n += width * ((0 if x.get("shared_value") else G * x["v_dim"]) + {True: H * x["v_dim"], "head": H}.get(x.get("gate"), 0))
        if x.get("kv_from") is not None:
            n -= width * G * (x["dim"] + x["v_dim"])
    return n


def layer_weights(layer: Dict, width: int) -> int:
    """Weights of the products that a token meets in one sequential layer."""
    n, f = mixer_weights(layer["mixer"], width), layer["mlp"]
    if f is None:
        return n
    if f["kind"] == "routed":
        return n + width * (f["n_expert"] + 3 * (f["top"] * f["ff"] + (f.get("shared") or 0)))
    return n + (3 if f["kind"] == "gated" else 2) * width * f["ff"]


def closest_attention_config(config: Config) -> Config:
    """Llama-shaped model of the same depth, width, heads and number of layer weights that a token meets."""
    m = next(x["mixer"] for x in config.layers if x["mixer"]["kind"] == "grouped_attention")
    H, G, W, n = m["n_head"], m["n_kv_head"], config.n_embd, config.n_layer
    weights = sum(layer_weights(layer, W) for layer in config.layers)
    ff = (weights // n - W * (2 * H + 2 * G) * 128) // (3 * W) // 8 * 8
    return Config(
        name=f"closest-to-{config.name}", block_size=1 << 17, vocab_size=config.vocab_size, padded_vocab_size=config.padded_vocab_size, n_layer=n,
        n_embd=W, n_head=H, n_query_groups=G, head_size=128, rotary_percentage=1.0, parallel_residual=False, bias=False,
        norm_class_name="RMSNorm", norm_eps=config.norm_eps, mlp_class_name="LLaMAMLP", intermediate_size=ff,
    )


def compared(config: Config) -> Dict[str, Config]:
    """The model and the closest ones, by what they are."""
    if any(x["mixer"]["kind"] != "latent_attention" for x in config.layers):
        return {"this design": config, "closest, dense": closest_config(config)}
    return {"this design": config, "closest, LLaMAMoE": closest_config(config), "closest, dense": closest_config(config, dense=True)}


def cache_lengths(config: Config, prompt: int, decode: int) -> int:
    """Tokens a layer keeps: its window, or (without windows) everything in described layers and the last ``prompt`` tokens in
    the closest model, whose decode steps can be captured once its caches are full."""
    window = config.layers[0]["mixer"].get("window") if config.layers is not None else config.sliding_window_size
    if window is not None:
        return window
    return prompt + decode + 32 if config.layers is not None else prompt


def _build(config: Config, batch: int, cache_length: int, dev: torch.device):
    from keys_values_b200.kvcache.factory import KVCacheFactory
    from keys_values_b200.models.registry import create_model, default_cache_name

    torch.manual_seed(0)
    with torch.device(dev):
        model = create_model(config).to(torch.bfloat16).eval()
    name = "lastrec-default" if config.layers is None else default_cache_name(config)
    kw = dict(init_grace_tokens=0) if config.layers is None else None
    model.assign_kv_caches(KVCacheFactory.create(model, name, batch, cache_length, device=dev, dtype=torch.bfloat16, cache_kwargs=kw))
    return model


@torch.inference_mode()
def throughput(config: Config, batch: int, prompt: int, decode: int, chunk: int = 2048, repeats: int = 2) -> Dict:
    """Best of ``repeats`` runs: prompts from pinned host memory, generated tokens read back inside the timed regions."""
    from keys_values_b200 import ops
    from keys_values_b200.generate.base import _prefill, batched_sample
    from keys_values_b200.generate.decode_graph import Decoder

    dev = torch.device("cuda", torch.cuda.current_device())
    length = cache_lengths(config, prompt, decode)
    model = _build(config, batch, length, dev)
    host = torch.randint(0, config.vocab_size, (batch, prompt), generator=torch.Generator().manual_seed(7)).pin_memory()
    greedy, warm = dict(temperature=0.0), 8
    total = prompt + decode + warm + 8
    _prefill(model, host[:, : min(prompt, length + 2 * chunk)].to(dev), chunk, total)
    best: Optional[Dict] = None
    for _ in range(repeats):
        torch.cuda.synchronize(dev)
        launches = ops.native_launches()
        e = [torch.cuda.Event(enable_timing=True) for _ in range(4)]
        e[0].record()
        logits = _prefill(model, host.to(dev, non_blocking=True), chunk, total)
        e[1].record()
        tokens = logits.argmax(-1).view(batch, 1)
        decoder = Decoder(model, batch)
        for _ in range(warm):
            tokens = batched_sample(decoder(tokens)[:, -1:], greedy).view(batch, 1)
        torch.cuda.synchronize(dev)
        e[2].record()
        out = []
        for _ in range(decode):
            tokens = batched_sample(decoder(tokens)[:, -1:], greedy).view(batch, 1)
            out.append(tokens)
        torch.cat(out, dim=1).cpu()
        e[3].record()
        torch.cuda.synchronize(dev)
        t_pre, t_dec = e[0].elapsed_time(e[1]) / 1e3, e[2].elapsed_time(e[3]) / 1e3
        if best is None or t_pre + t_dec < best["prefill_s"] + best["decode_s"]:
            best = dict(
                model=config.name, batch=batch, prompt=prompt, decode_steps=decode, prefill_s=t_pre, decode_s=t_dec,
                prefill_tokens_per_s=batch * prompt / t_pre, decode_tokens_per_s=batch * decode / t_dec, ms_per_decode_step=1e3 * t_dec / decode,
                decode_mode="cuda graph" if decoder.graph is not None else f"eager ({decoder.reason})",
                native_launches=ops.native_launches() - launches, peak_mem_gb=torch.cuda.max_memory_allocated(dev) / 2**30,
                parameters=sum(p.numel() for p in model.parameters()),
            )
    ops.check_status(dev)
    return best


# ------------------------------------------------------------------------------------------------- kernels
def _peaks() -> Dict[str, float]:
    file = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    got = json.loads(file.read_text()) if file.is_file() else {}
    return dict(gbs=got.get("hbm_gbs", 6650.0), tflops=got.get("bf16_tflops", 1590.0))


def time_us(fn: Callable[[], None], flush: torch.Tensor, n: int = 15) -> float:
    """Median time. Before every launch a buffer larger than L2 is written and another one read, so that the launch
    finds L2 full of clean lines (dirty ones would be written back inside the timed region)."""
    times = []
    for i in range(n + 3):
        flush[0].fill_(i & 127)
        flush[1].sum()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= 3:
            times.append(a.elapsed_time(b) * 1e3)
    return sorted(times)[len(times) // 2]


class KernelTable:
    def __init__(self):
        self.peaks = _peaks()
        self.flush = torch.zeros(2, 64 * 2**20, dtype=torch.float32, device="cuda")
        self.rows: List[Dict] = []

    def add(self, what: str, fn: Callable[[], None], gbytes: float = 0.0, tflop: float = 0.0) -> None:
        us = time_us(fn, self.flush)
        roof = 1e6 * max(gbytes / self.peaks["gbs"], tflop / self.peaks["tflops"])
        self.rows.append(dict(kernel=what, us=round(us, 1), roofline_us=round(roof, 1), fraction=round(roof / us, 3),
                              bound="memory" if gbytes / self.peaks["gbs"] > tflop / self.peaks["tflops"] else "math"))
        print(f"{what:64s} {us:9.1f} us   roofline {roof:8.1f} us   {roof / us:6.3f}", flush=True)


def _window_pairs(T: int, P: int, window: int) -> int:
    """Visible (query, key) pairs of T new tokens after P cached ones."""
    return sum(min(P + t + 1, window) for t in range(T))


@torch.inference_mode()
def kernel_table(config: Config, batch: int, tokens: int = 8192, dense_like: bool = True) -> List[Dict]:
    """Kernels of one middle layer of ``config`` (Pazenex: of one layer of each kind): a pass of ``tokens`` new tokens of one sequence with a full window before them,
    and a single-token pass of ``batch`` sequences with full rings; like kernels of the closest model after each."""
    if any(x["mixer"]["kind"] == "side_by_side" for x in config.layers):
        return side_by_side_kernel_table(config, batch, tokens)
    if any(x["mixer"]["kind"] == "retention" for x in config.layers):
        return output_norm_kernel_table(config, batch, tokens)
    if any(x["mixer"]["kind"] != "latent_attention" for x in config.layers):
        return sequential_kernel_table(config, batch, tokens)
    from keys_values_b200 import ops
    from keys_values_b200.kvcache.sequences import SequenceTable
    from keys_values_b200.models.layered import latent_shape
    from keys_values_b200.ops import cuda as cu
    from keys_values_b200.ops import layers as L
    from keys_values_b200.ops import layers_cuda as LC

    dev, bf = torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    m, f = config.layers[0]["mixer"], config.layers[0]["mlp"]
    s, W, win = latent_shape(m), config.n_embd, m["window"]
    H, E, top, ff = s.heads, f["n_expert"], f["top"], f["ff"]
    mid, eps = config.n_layer // 2, config.norm_eps
    rand = lambda *shape: torch.randn(*shape, device=dev, dtype=bf)  # noqa: E731

    def sequences(B, start):
        t = SequenceTable(B, dev, 1, W)
        t.set_batch([t.acquire() for _ in range(B)])
        t.pos.fill_(start)
        t.pos_host = [start] * B
        return t

    up, down = 0.02 * rand(E, ff, W), 0.02 * rand(E, W, ff)
    gain, blend, coef = torch.ones((), device=dev), torch.rand(W, device=dev), torch.rand(mid + 2, device=dev)
    for B, T in ((1, tokens), (batch, 1)):
        n = B * T
        tag = f"prefill {T} tokens" if T > 1 else f"decode {B} rows"
        seq = sequences(B, 2 * win).begin(B, T)
        seq.start = seq.start.clone()
        # ---- layer edge
        hist = torch.randn(mid + 2, B, T, W, device=dev)
        x, out, mix = torch.randn(B, T, W, device=dev), torch.empty(B, T, W, device=dev), rand(B, T, W)
        h, hs = torch.empty_like(mix), torch.empty_like(mix)
        ex = rand(n * top, W)
        row = torch.randperm(n * top, device=dev).int().view(n, top)
        wt = torch.rand(n, top, device=dev)
        state = torch.zeros(B, W, device=dev)
        tab.add(f"{tag}: layer edge ({mid + 1} streams, {top} experts)",
                lambda: LC.layer_edge(x, mix, ex, row, wt, hist, mid + 1, coef, out, gain, blend, state, h, hs, seq, eps),
                gbytes=n * W * (4 * (mid + 1) + 4 + 2 + 2 * top + 4 + 4 + 2 + 2) / 1e9)
        a, r, w1 = rand(n, W), rand(n, W), rand(W)
        if cu.add_rmsnorm_supported(a):
            tab.add(f"{tag}:   like: add + RMSNorm", lambda: cu.add_rmsnorm_fwd(a, r, w1, eps, False), gbytes=n * W * 8 / 1e9)
        else:
            tab.add(f"{tag}:   like: RMSNorm", lambda: cu.rmsnorm_fwd(a, w1, eps, False), gbytes=n * W * 4 / 1e9)
        del hist, ex
        # ---- latent prep
        qkv = rand(B, T, H * (s.dim + s.rot) + s.kv_rank + s.rot)
        norm, freq = torch.ones(s.kv_rank, device=dev), torch.rand(s.rot_dims // 2, device=dev)
        ring = rand(B, win, s.row)
        P = win - 1 if T > 1 else 0
        lat = rand(B, P + T, s.row)
        if T > 1:
            prep = lambda: LC.latent_prep(qkv, norm, freq, lat, ring, seq, P, s, eps)  # noqa: E731
        else:
            prep = lambda: LC.latent_prep(qkv, norm, freq, None, ring, seq, 0, s, eps)  # noqa: E731
        tab.add(f"{tag}: split, latent norm, rotation, into the ring", prep,
                gbytes=2 * (n * (qkv.shape[2] + H * (s.dimp + s.rp) + s.row) + B * min(T, win) * s.row) / 1e9)
        qkv2, cs = rand(B, T, 3 * H * 128), torch.rand(T, 128, device=dev)
        tab.add(f"{tag}:   like: split + RoPE", lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, None, None, H, H, 128, eps, 128, False),
                gbytes=n * 2 * 2 * qkv2.shape[2] / 1e9)
        if T > 1:
            tab.add(f"{tag}: ring gather", lambda: LC.ring_gather(ring, lat, seq, P), gbytes=B * P * s.row * 4 / 1e9)
            kb, vb, tp = (rand(B, H, win, 128) for _ in range(2)), None, torch.zeros(B, H, win, dtype=torch.int32, device=dev)
            kb, vb = kb
            nk, slots = rand(B, H, min(T, win), 128), torch.arange(min(T, win), device=dev).int().view(1, 1, -1).expand(B, H, -1)
            tab.add(f"{tag}:   like: cache write", lambda: cu.cache_write(kb, vb, tp, slots, nk, nk, 0), gbytes=B * H * min(T, win) * 128 * 8 / 1e9)
            # ---- attention over expanded keys
            q, kv = rand(B, T, H, s.dimp + s.rp), rand(B * (P + T), H * (s.dimp + s.vdp))
            pairs = B * H * _window_pairs(T, P, win)
            tab.add(f"{tag}: attention {s.dim}+{s.rot} / {s.vdim}, window {win}", lambda: LC.latent_attend(q, kv, lat, seq, P, s, win, 0.07),
                    tflop=2 * pairs * (s.dim + s.rot + s.vdim) / 1e12)
            q2, k2 = rand(B, H, T, 128), rand(B, H, P + T, 128)
            tab.add(f"{tag}:   like: attention 128 / 128, window {win}", lambda: cu.sdpa_fwd(q2, k2, k2, 0.09, P, None, False, win, None),
                    tflop=2 * pairs * 256 / 1e12)
            del q, kv, q2, k2, kb, vb
        else:
            q, qa = rand(B, 1, H, s.dimp + s.rp), rand(H, B, s.kvp)
            tab.add(f"{tag}: attention over the ring of {win}", lambda: LC.latent_decode(qa, q, ring, seq, s, 0.07),
                    gbytes=B * win * s.row * 2 / 1e9, tflop=2 * B * win * H * (2 * s.kv_rank + s.rot) / 1e12)
            q2, k2, v2 = rand(B, H, 1, 128), rand(B, H, win, 128), rand(B, H, win, 128)
            tp = torch.arange(win, device=dev, dtype=torch.int32).expand(B, H, win).contiguous()
            tab.add(f"{tag}:   like: attention over {win} slots", lambda: cu.decode_attention(q2, k2, v2, 0.09, win, False, sliding_window=win,
                    token_pos=tp, query_pos=win - 1), gbytes=2 * B * H * win * 128 * 2 / 1e9)
            del k2, v2
        # ---- routed experts
        hn = rand(n, W)
        logits = torch.randn(n, E, device=dev)
        used = E if n * top >= 4 * E else E * (1 - (1 - 1 / E) ** (n * top))
        tab.add(f"{tag}: routed experts, all kernels ({E} x {ff}, top {top})",
                lambda: LC.moe_forward(hn, logits, up, down, top, 1, L.RouterRule(), ff, W),
                gbytes=2 * (used * 2 * ff * W + n * W * (1 + top)) / 1e9, tflop=4 * n * top * ff * W / 1e12)
        from keys_values_b200.models.model import LLaMAMLP, LLaMAMoE

        for dense in (False, True):
            cc = closest_config(config, dense)
            with torch.device(dev):
                mlp = (LLaMAMLP if dense else LLaMAMoE)(cc).to(bf)
            x3 = hn.view(1, n, W)
            fl = 6 * n * cc.intermediate_size * (1 if dense else top) * W / 1e12
            by = 2 * (3 * cc.intermediate_size * W * (1 if dense else used) + 2 * n * W) / 1e9
            tab.add(f"{tag}:   like: {'dense SwiGLU' if dense else 'LLaMAMoE'}, all kernels", lambda: mlp(x3), gbytes=by, tflop=fl)
            del mlp
        tile = LC.moe_tile(n * top, E, bf)
        cap = n * top // tile + min(E, n * top)
        buf, hid = rand(cap * tile, W), torch.empty(cap * tile, ff, device=dev, dtype=bf)
        ids = torch.randint(0, E, (n * top,), device=dev)
        cnt = torch.bincount(ids, minlength=E)
        tiles = ((cnt + tile - 1) // tile)
        te = torch.repeat_interleave(torch.arange(E, device=dev), tiles).int()
        plan = torch.tensor([te.numel()], device=dev, dtype=torch.int32)
        tr = (torch.arange(te.numel(), device=dev) * tile).int()
        st = cu.status_word(dev)
        ll, p_ = cu._ll, cu._p

        def grouped(src, w, dst, n_out, k, act):
            cu._check(LC.lib().kvb_moe_gemm(p_(src), p_(w), p_(dst), p_(plan), p_(te), p_(tr), tile, cap, E, n_out, k, ll(k), ll(n_out), act, 1, 0,
                                            p_(st), cu._stream(src)), "moe_gemm")

        us_e = int((cnt > 0).sum())
        tab.add(f"{tag}: grouped product up (tile {tile})", lambda: grouped(buf, up, hid, ff, W, 1),
                gbytes=2 * (us_e * ff * W + n * top * (W + ff)) / 1e9, tflop=2 * n * top * ff * W / 1e12)
        tab.add(f"{tag}: grouped product down (tile {tile})", lambda: grouped(hid, down, buf, W, ff, 0),
                gbytes=2 * (us_e * ff * W + n * top * (W + ff)) / 1e9, tflop=2 * n * top * ff * W / 1e12)
        w2, a2 = rand(ff * top, W), rand(n, W)
        tab.add(f"{tag}:   like: library product {n} x {ff * top} x {W}", lambda: torch.mm(a2, w2.t()),
                gbytes=2 * (ff * top * W + n * (W + ff * top)) / 1e9, tflop=2 * n * ff * top * W / 1e12)
        del buf, hid
    ops.check_status(dev)
    return tab.rows


@torch.inference_mode()
def sequential_kernel_table(config: Config, batch: int, tokens: int = 8192) -> List[Dict]:
    """Kernels of a Mamba-2 and of an attention layer between norms: a prompt of ``tokens`` tokens of one sequence, and a
    single-token pass of ``batch`` sequences at that position; like kernels of the closest model after each."""
    from keys_values_b200 import ops
    from keys_values_b200.kvcache.sequences import SequenceTable
    from keys_values_b200.models.grouped_attention import grouped_shape
    from keys_values_b200.models.state_space import state_shape
    from keys_values_b200.ops import cuda as cu
    from keys_values_b200.ops import layers as L
    from keys_values_b200.ops import layers_cuda as LC

    dev, bf = torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    mixer = {x["mixer"]["kind"]: x["mixer"] for x in config.layers}
    s, m = grouped_shape(mixer["grouped_attention"]), state_shape(mixer["mamba2"])
    W, ff, eps = config.n_embd, config.layers[0]["mlp"]["ff"], config.norm_eps
    H, G, D = s.heads, s.kv_heads, s.dimp
    rand = lambda *shape: torch.randn(*shape, device=dev, dtype=bf)  # noqa: E731
    f32 = lambda *shape: torch.rand(*shape, device=dev)  # noqa: E731
    for B, T, start in ((1, tokens, 0), (4, tokens, 0), (batch, 1, tokens - 1)):
        n = B * T
        tag = f"prefill {B} x {T} tokens" if T > 1 else f"decode {B} rows"
        table = SequenceTable(B, dev)
        table.set_batch([table.acquire() for _ in range(B)])
        table.pos.fill_(start)
        table.pos_host = [start] * B
        seq = table.begin(B, T)
        seq.start = seq.start.clone()
        # ---- between sublayers
        x, sub, h, w1, w2 = torch.randn(B, T, W, device=dev), rand(B, T, W), rand(B, T, W), f32(W), f32(W)
        tab.add(f"{tag}: norm, residual sum, norm", lambda: LC.norm_edge(x, sub, w1, x, w2, h, None, None, None, eps, True), gbytes=n * W * 12 / 1e9)
        a, r, w = rand(n, W), rand(n, W), rand(W)
        like_norm = lambda: cu.add_rmsnorm_fwd(a, r, w, eps, False) if cu.add_rmsnorm_supported(a) else cu.rmsnorm_fwd(a, w, eps, False)  # noqa: E731
        norm_bytes = n * W * (8 if cu.add_rmsnorm_supported(a) else 4) / 1e9
        tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
        up = rand(n, ff)
        tab.add(f"{tag}: squared relu", lambda: LC.activate(up, 1), gbytes=n * ff * 4 / 1e9)
        tab.add(f"{tag}:   like: SwiGLU", lambda: cu.swiglu_fwd(up, up), gbytes=n * ff * 6 / 1e9)
        del up
        # ---- attention
        cols = s.gate_col + (H * s.vdp if s.gate else 0)
        qkv, nq, nk, freq = rand(B, T, cols), f32(H * D), f32(G * D), f32(s.rot_dims // 2)
        length = tokens + 64
        rows = rand(B, length, G, D + s.vdp)
        kv_bytes = 2 * n * G * (D + s.vdp)
        tab.add(f"{tag}: norm, rotation, into the cache", lambda: LC.grouped_prep(qkv, nq, nk, freq, rows, seq, s, eps, L.RowPlan()),
                gbytes=(2 * n * (2 * H * D + G * D) + kv_bytes) / 1e9)
        qkv2, cs, wq = rand(B, T, (H + 2 * G) * D), f32(T, D), rand(D)
        tab.add(f"{tag}:   like: QK norm, split + RoPE", lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, H, G, D, eps, D, False),
                gbytes=2 * 2 * n * (H + 2 * G) * D / 1e9)
        q = rand(B, T, H, D)
        q2, k2 = rand(B, H, T, D), rand(B, G, tokens, D)
        if T > 1:
            flop = B * H * (T * (T + 1) // 2) * 2 * (s.dim + s.vdim) / 1e12
            tab.add(f"{tag}: attention, {H} heads on {G}, sink and gate", lambda: LC.grouped_attend(q, qkv, rows, seq, s, None, L.RowPlan()), tflop=flop)
            tab.add(f"{tag}:   like: attention, {H} heads on {G}", lambda: cu.sdpa_fwd(q2, k2, k2, 0.09, 0), tflop=flop)
        else:
            by = 2 * B * G * tokens * (s.dim + s.vdim) / 1e9
            v2 = rand(B, G, tokens, D)
            tab.add(f"{tag}: attention over {tokens} positions, {H} heads on {G}", lambda: LC.grouped_attend(q, qkv, rows, seq, s, None, L.RowPlan()), gbytes=by)
            tab.add(f"{tag}:   like: attention over {tokens} slots", lambda: cu.decode_attention(q2, k2, v2, 0.09, tokens), gbytes=by)
        del rows, k2, q2, q, qkv2
        # ---- state space
        u, ring, state = rand(B, T, m.ld), rand(B, m.taps, m.channels), 0.01 * torch.randn(B, m.heads, m.np, m.vdp, device=dev)
        cw, cb, db, al, sk = f32(m.taps, m.channels), f32(m.channels), f32(m.heads) - 4, f32(m.heads), f32(m.heads)
        state_bytes = B * m.heads * m.np * m.vdp * 8
        if T > 1:
            tab.add(f"{tag}: convolution, {m.channels} channels", lambda: LC.short_conv(u, m.inner, cw, cb, ring, seq, True), gbytes=4 * n * m.channels / 1e9)
            xbc = rand(B, T, m.channels)
            flop = n * (m.heads * (4 * m.np * m.vdp + 128 * m.vdp) + m.groups * 128 * m.np) / 1e12
            by = (2 * n * (m.channels + m.inner + m.heads) + state_bytes) / 1e9
            tab.add(f"{tag}: state scan, {m.heads} heads of {m.np} x {m.vdp}", lambda: LC.state_scan(u, xbc, db, al, sk, state, seq, m), gbytes=by, tflop=flop)
            del xbc
        else:
            by = (state_bytes + 2 * n * (m.channels * (1 + m.taps) + m.inner)) / 1e9
            tab.add(f"{tag}: convolution and state step, {m.heads} heads of {m.np} x {m.vdp}",
                    lambda: LC.state_step(u, cw, cb, db, al, sk, ring, state, seq, m), gbytes=by)
        y, gw = rand(B, T, m.inner), f32(m.inner)
        tab.add(f"{tag}: gated norm in {m.norm_groups} parts", lambda: LC.gated_group_norm(y, u, gw, m, eps), gbytes=6 * n * m.inner / 1e9)
        tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
        # ---- products (library, in both models)
        for what, k, cols_out in (("mamba in", W, m.ld), ("up", W, ff)):
            a2, w3 = rand(n, k), rand(cols_out, k)
            tab.add(f"{tag}: library product {what} {n} x {cols_out} x {k}", lambda: torch.mm(a2, w3.t()), gbytes=2 * (n * (k + cols_out) + k * cols_out) / 1e9,
                    tflop=2 * n * k * cols_out / 1e12)
        del u, y, a2, w3, x, sub, h
    ops.check_status(dev)
    return tab.rows


def _like_mlp(width: int, ff: int, dev, dtype):
    from keys_values_b200.models.model import LLaMAMLP

    c = Config(name="like", n_layer=1, n_embd=width, n_head=1, head_size=width, vocab_size=8, padded_vocab_size=8, bias=False, norm_class_name="RMSNorm",
               mlp_class_name="LLaMAMLP", intermediate_size=ff)
    with torch.device(dev):
        return LLaMAMLP(c).to(dtype)


@torch.inference_mode()
def output_norm_kernel_table(config: Config, batch: int, tokens: int = 8192) -> List[Dict]:
    """Kernels of one layer of each kind of a model with retention, differential and chunked attention: prompts of ``tokens`` tokens, and a
    single-token pass of ``batch`` sequences at that position; like kernels of the closest model after each."""
    from keys_values_b200 import ops
    from keys_values_b200.kvcache.sequences import SequenceTable
    from keys_values_b200.models.grouped_attention import grouped_shape
    from keys_values_b200.models.layered import RoutedMLP
    from keys_values_b200.models.retention import retention_shape
    from keys_values_b200.ops import cuda as cu
    from keys_values_b200.ops import layers as L
    from keys_values_b200.ops import layers_cuda as LC

    dev, bf = torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    mixers = [x["mixer"] for x in config.layers]
    diff = grouped_shape(next(x for x in mixers if x.get("differential") is not None))
    diff = L.GroupedShape(**{**diff.__dict__, "lam": 0.4, "eps": config.norm_eps})
    chunked = grouped_shape(next(x for x in mixers if x.get("chunk")))
    r = retention_shape(next(x for x in mixers if x["kind"] == "retention"))
    mlps = [x["mlp"] for x in config.layers if x["mlp"]]
    ff, f = next(x["ff"] for x in mlps if x["kind"] == "gated"), next(x for x in mlps if x["kind"] == "routed")
    W, eps = config.n_embd, config.norm_eps
    plan = L.RowPlan()
    rand = lambda *shape: torch.randn(*shape, device=dev, dtype=bf)  # noqa: E731
    f32 = lambda *shape: torch.rand(*shape, device=dev)  # noqa: E731
    with torch.device(dev):
        routed = RoutedMLP(config, {**f, "shared": None}).to(bf)
        torch.nn.init.normal_(routed.gate.weight, std=0.02)
    shared_mlp, active_mlp = _like_mlp(W, f["shared"], dev, bf), _like_mlp(W, f["top"] * f["ff"], dev, bf)
    for B, T, start in ((1, tokens, 0), (4, tokens, 0), (batch, 1, tokens - 1)):
        n = B * T
        tag = f"prefill {B} x {T} tokens" if T > 1 else f"decode {B} rows"
        table = SequenceTable(B, dev)
        table.set_batch([table.acquire() for _ in range(B)])
        table.pos.fill_(start)
        table.pos_host = [start] * B
        seq = table.begin(B, T)
        seq.start = seq.start.clone()
        # ---- between sublayers
        x, sub, h, w1 = torch.randn(B, T, W, device=dev), rand(B, T, W), rand(B, T, W), f32(W)
        tab.add(f"{tag}: norm, residual sum", lambda: LC.norm_edge(x, sub, w1, x, None, h, None, None, None, eps, False), gbytes=n * W * 12 / 1e9)
        a, rr, w = rand(n, W), rand(n, W), rand(W)
        fused = cu.add_rmsnorm_supported(a)
        like_norm = lambda: cu.add_rmsnorm_fwd(a, rr, w, eps, False) if fused else cu.rmsnorm_fwd(a, w, eps, False)  # noqa: E731
        norm_bytes = n * W * (8 if fused else 4) / 1e9
        tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
        top = f["top"]
        experts = (rand(n * top, W), torch.randperm(n * top, device=dev).int().view(n, top), f32(n, top))
        tab.add(f"{tag}: sum of {top} experts and shared, norm, residual sum",
                lambda: LC.norm_edge(x, sub, w1, x, None, h, None, None, None, eps, False, experts), gbytes=n * W * (12 + 2 * top) / 1e9)
        del experts
        up = rand(n, 2 * ff)
        tab.add(f"{tag}: SwiGLU", lambda: LC.glu(up, ff), gbytes=n * ff * 6 / 1e9)
        u1 = up.view(2, n, ff)
        tab.add(f"{tag}:   like: SwiGLU", lambda: cu.swiglu_fwd(u1[0], u1[1]), gbytes=n * ff * 6 / 1e9)
        del up, u1
        # ---- attentions
        length = tokens + 64
        for what, s in (("chunked", chunked), ("differential", diff)):
            H, G, D, V = s.heads, s.kv_heads, s.dim, s.vdim
            qkv = rand(B, T, s.ld)
            if s.head_norm:
                nq, nk = f32(s.dimp), f32(s.dimp)
            else:
                nq, nk = f32(H * s.dimp), f32(G * s.dimp)
            freq, sink = f32(s.rot_dims // 2), torch.zeros(H, device=dev) if s.sink else None
            rows = rand(B, length, G, s.row)
            tab.add(f"{tag}: {what}: norm, rotation, into the cache", lambda: LC.grouped_prep(qkv, nq, nk, freq, rows, seq, s, eps, plan),
                    gbytes=2 * n * (2 * H * s.maps * D + 2 * G * (s.maps * D + V)) / 1e9)
            qkv2, cs, wq = rand(B, T, (H + 2 * G) * 128), f32(T, 128), rand(128)
            tab.add(f"{tag}:   like: QK norm, split + RoPE", lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, H, G, 128, eps, 128, False),
                    gbytes=2 * 2 * n * (H + 2 * G) * 128 / 1e9)
            q = rand(B, T, H * s.maps, s.dimp)
            seen = s.window or 1 << 40
            q2, k2 = rand(B, H, T, 128), rand(B, G, tokens, 128)
            win = s.window if s.window and s.window < tokens else 0
            if T > 1:
                pairs = B * H * (_window_pairs(T, 0, seen) + (min(s.keep, T) * max(0, T - seen) if s.window else 0))
                tab.add(f"{tag}: {what} attention, {H} heads on {G}" + (f", window {s.window} + {s.keep}" if s.window else ", soft cap, sink, gate"),
                        lambda: LC.grouped_attend(q, qkv, rows, seq, s, sink, plan), tflop=2 * pairs * s.maps * (D + V) / 1e12)
                like = B * H * _window_pairs(T, 0, seen)
                tab.add(f"{tag}:   like: attention 128 / 128" + (f", window {win}" if win else ""),
                        lambda: cu.sdpa_fwd(q2, k2, k2, 0.09, 0, None, False, win, None) if win else cu.sdpa_fwd(q2, k2, k2, 0.09, 0), tflop=2 * like * 256 / 1e12)
            else:
                m = min(tokens, seen) + (s.keep if win else 0)
                tab.add(f"{tag}: {what} attention over {m} positions, {H} heads on {G}", lambda: LC.grouped_attend(q, qkv, rows, seq, s, sink, plan),
                        gbytes=2 * B * G * m * (s.maps * D + V) / 1e9)
                m2 = min(tokens, seen)
                k3, v3 = rand(B, G, m2, 128), rand(B, G, m2, 128)
                tab.add(f"{tag}:   like: attention over {m2} slots", lambda: cu.decode_attention(q2, k3, v3, 0.09, m2), gbytes=2 * B * G * m2 * 256 / 1e9)
                del k3, v3
            del rows, k2, q2, q, qkv2, qkv
        # ---- retention
        state, decay = 0.01 * torch.randn(B, r.heads, r.np, r.vdp, device=dev), 1 - 0.05 * f32(r.heads)
        log2, freq = decay.log2(), f32(r.rot_dims // 2)
        state_bytes = B * r.heads * r.np * r.vdp * 8
        if T > 1:
            qk32, vg = torch.randn(B, T, r.qk, device=dev), rand(B, T, 2 * r.inner)
            tab.add(f"{tag}: retention: rotation", lambda: LC.retention_prep(qk32, freq, seq, r, bf), gbytes=6 * n * r.qk / 1e9)
            qkv2, cs, wq = rand(B, T, 2 * r.qk), f32(T, 128), rand(128)
            tab.add(f"{tag}:   like: QK norm, split + RoPE",
                    lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, 2 * r.qk // 384, r.qk // 384, 128, eps, 128, False) if r.qk % 384 == 0
                    else cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, 2 * r.qk // 128 - 16, 8, 128, eps, 128, False), gbytes=8 * n * r.qk / 1e9)
            qk = rand(B, T, r.qk)
            flop = n * r.heads * (4 * r.np * r.vdp + 128 * (r.np + r.vdp)) / 1e12
            tab.add(f"{tag}: retention scan, {r.heads} heads of {r.np} x {r.vdp}", lambda: LC.retention_scan(qk, vg, decay, log2, state, seq, r),
                    gbytes=(2 * n * (r.qk + 2 * r.inner) + state_bytes) / 1e9, tflop=flop)
            q2 = rand(B, r.heads, T, 128)
            tab.add(f"{tag}:   like: attention 128 / 128, {r.heads} heads", lambda: cu.sdpa_fwd(q2, q2, q2, 0.09, 0),
                    tflop=2 * B * r.heads * (T * (T + 1) // 2) * 256 / 1e12)
            y = rand(B, T, r.inner)
            tab.add(f"{tag}: retention: norm per head, gate", lambda: LC.head_norm_gate(y, vg[..., r.inner :], r, eps), gbytes=6 * n * r.inner / 1e9)
            tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
            del qk32, vg, qk, q2, qkv2, y
        else:
            u = torch.randn(B, 1, r.qk + 2 * r.inner, device=dev)
            tab.add(f"{tag}: retention step, {r.heads} heads of {r.np} x {r.vdp}", lambda: LC.retention_step(u, freq, decay, state, seq, r, eps, bf),
                    gbytes=(state_bytes + 4 * n * u.shape[-1]) / 1e9)
        del state
        # ---- feed-forwards
        hn = rand(n, W)
        E = f["n_expert"]
        used = E if n * top >= 4 * E else E * (1 - (1 - 1 / E) ** (n * top))
        tab.add(f"{tag}: routed experts, all kernels ({E} x {f['ff']}, top {top})", lambda: routed(hn),
                gbytes=2 * (used * 3 * f["ff"] * W + n * W * (1 + top)) / 1e9, tflop=6 * n * top * f["ff"] * W / 1e12)
        tab.add(f"{tag}:   like: dense SwiGLU of {top * f['ff']}, all kernels", lambda: active_mlp(hn.view(1, n, W)),
                gbytes=2 * (3 * top * f["ff"] * W + 2 * n * W) / 1e9, tflop=6 * n * top * f["ff"] * W / 1e12)
        tab.add(f"{tag}: shared expert (library products, SwiGLU)", lambda: shared_mlp(hn.view(1, n, W)),
                gbytes=2 * (3 * f["shared"] * W + 2 * n * W) / 1e9, tflop=6 * n * f["shared"] * W / 1e12)
        w3 = rand(r.qk, W)
        tab.add(f"{tag}: library product with fp32 result {n} x {r.qk} x {W}", lambda: L.linear_fp32(hn, w3),
                gbytes=(2 * n * W + 2 * r.qk * W + 4 * n * r.qk) / 1e9, tflop=2 * n * r.qk * W / 1e12)
        tab.add(f"{tag}:   like: with bf16 result", lambda: torch.mm(hn, w3.t()), gbytes=2 * (n * W + r.qk * W + n * r.qk) / 1e9, tflop=2 * n * r.qk * W / 1e12)
        del hn, w3, x, sub, h, a, rr
        torch.cuda.empty_cache()
    ops.check_status(dev)
    return tab.rows


@torch.inference_mode()
def side_by_side_kernel_table(config: Config, batch: int, tokens: int = 8192) -> List[Dict]:
    """Kernels of one layer of each kind of a model with gated linear attention and a pooled window side by side with a gated recurrence: prompts
    of ``tokens`` tokens, and a single-token pass of ``batch`` sequences at that position; like kernels of the closest model after each."""
    from keys_values_b200 import ops
    from keys_values_b200.kvcache.sequences import SequenceTable
    from keys_values_b200.models.gated_linear import gated_linear_shape
    from keys_values_b200.models.gated_recurrence import recurrence_shape
    from keys_values_b200.models.grouped_attention import grouped_shape
    from keys_values_b200.ops import cuda as cu
    from keys_values_b200.ops import layers as L
    from keys_values_b200.ops import layers_cuda as LC

    dev, bf = torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    mixers = [x["mixer"] for x in config.layers]
    both = next(x for x in mixers if x["kind"] == "side_by_side")
    plain = grouped_shape(next(x for x in mixers if x["kind"] == "grouped_attention" and x.get("kv_from") is None))
    borrowed = grouped_shape(next(x for x in mixers if x.get("kv_from") is not None))
    pooled, r = grouped_shape(both["left"]), recurrence_shape(both["right"])
    m = gated_linear_shape(next(x for x in mixers if x["kind"] == "gated_linear_attention"))
    ff, limit = config.layers[0]["mlp"]["ff"], config.layers[0]["mlp"]["limit"]
    W, eps, taps = config.n_embd, config.norm_eps, config.input_conv
    rand = lambda *shape: torch.randn(*shape, device=dev, dtype=bf)  # noqa: E731
    f32 = lambda *shape: torch.rand(*shape, device=dev)  # noqa: E731
    tiles = lambda n: -(-n // 128) * 128  # noqa: E731
    for B, T, start in ((1, tokens, 0), (4, tokens, 0), (batch, 1, tokens - 2)):
        n = B * T
        tag = f"prefill {B} x {T} tokens" if T > 1 else f"decode {B} rows"
        table = SequenceTable(B, dev)
        table.set_batch([table.acquire() for _ in range(B)])
        table.pos.fill_(start)
        table.pos_host = [start] * B
        seq = table.begin(B, T)
        seq.start = seq.start.clone()
        # ---- between sublayers
        x, sub, h, w1, w2 = torch.randn(B, T, W, device=dev), rand(B, T, W), rand(B, T, W), f32(W), f32(W)
        ring, cw = rand(B, taps, W), f32(taps, W)
        edge = L.EdgeTokens(seq, None, cw, ring) if T == 1 else None
        tab.add(f"{tag}: norm, residual sum, norm" + (", convolution" if T == 1 else ""),
                lambda: LC.norm_edge(x, sub, w1, x, w2, h, None, None, None, eps, False, None, edge), gbytes=(n * W * 12 + (0 if T > 1 else B * taps * W * 2)) / 1e9)
        a, rr, w = rand(n, W), rand(n, W), rand(W)
        fused = cu.add_rmsnorm_supported(a)
        like_norm = lambda: cu.add_rmsnorm_fwd(a, rr, w, eps, False) if fused else cu.rmsnorm_fwd(a, w, eps, False)  # noqa: E731
        norm_bytes = n * W * (8 if fused else 4) / 1e9
        tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
        if T > 1:
            tab.add(f"{tag}: convolution of {W} inputs", lambda: LC.short_conv(sub, 0, cw, None, ring, seq, False, h), gbytes=4 * n * W / 1e9)
        up = rand(n, 2 * ff)
        tab.add(f"{tag}: clamped unit", lambda: LC.glu(up, ff, limit), gbytes=n * ff * 6 / 1e9)
        u1 = up.view(2, n, ff)
        tab.add(f"{tag}:   like: SwiGLU", lambda: cu.swiglu_fwd(u1[0], u1[1]), gbytes=n * ff * 6 / 1e9)
        del up, u1
        # ---- attentions
        for what, s in (("attention", plain), ("attention over another layer's keys", borrowed), ("pooled window", pooled)):
            H, G, D, V = s.heads, s.kv_heads, s.dim, s.vdim
            plan = L.RowPlan(tiles(tokens // s.pool), tiles(tokens + 64)) if s.pool else L.RowPlan()
            length = sum(plan) if s.pool else tokens + 64
            qkv, freq, rows = rand(B, T, s.ld), f32(s.rot_dims // 2), rand(B, length, G, s.row)
            unit, temp = (torch.ones(s.dimp, device=dev), f32(H)) if s.pool else (None, None)
            own = 0 if s.borrowed else G * (D + V)
            tab.add(f"{tag}: {what}: " + ("norm, " if s.pool else "") + "rotation" + ("" if s.borrowed else ", into the cache") + (", means of blocks" if s.pool else ""),
                    lambda: LC.grouped_prep(qkv, unit, unit, freq, rows, seq, s, eps, plan, temp), gbytes=2 * n * 2 * (H * D + own) / 1e9)
            qkv2, cs, wq = rand(B, T, (H + 2 * G) * 128), f32(T, 128), rand(128)
            tab.add(f"{tag}:   like: QK norm, split + RoPE", lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, H, G, 128, eps, 128, False),
                    gbytes=2 * 2 * n * (H + 2 * G) * 128 / 1e9)
            q = rand(B, T, H, s.dimp)
            q2, k2 = rand(B, H, T, 128), rand(B, G, tokens, 128)
            seen = s.window or 1 << 40
            win = s.window if s.window and s.window < tokens else 0
            blocks = lambda t: max(0, (start + t - s.window + 1) // s.pool) if s.pool else 0  # noqa: E731
            if T > 1:
                pairs = B * H * (_window_pairs(T, 0, seen) + sum(blocks(t) for t in range(T)))
                tab.add(f"{tag}: {what}, {H} heads on {G}" + (f", {s.window} tokens and blocks of {s.pool}" if s.pool else ", gate"),
                        lambda: LC.grouped_attend(q, qkv, rows, seq, s, None, plan), tflop=2 * pairs * (D + V) / 1e12)
                like = B * H * _window_pairs(T, 0, seen)
                tab.add(f"{tag}:   like: attention 128 / 128" + (f", window {win}" if win else ""),
                        lambda: cu.sdpa_fwd(q2, k2, k2, 0.09, 0, None, False, win, None) if win else cu.sdpa_fwd(q2, k2, k2, 0.09, 0), tflop=2 * like * 256 / 1e12)
            else:
                k = min(tokens, seen) + blocks(0)
                tab.add(f"{tag}: {what} over {k} rows, {H} heads on {G}", lambda: LC.grouped_attend(q, qkv, rows, seq, s, None, plan),
                        gbytes=2 * B * G * k * (D + V) / 1e9)
                k3, v3 = rand(B, G, min(tokens, seen), 128), rand(B, G, min(tokens, seen), 128)
                tab.add(f"{tag}:   like: attention over {k3.shape[2]} slots", lambda: cu.decode_attention(q2, k3, v3, 0.09, k3.shape[2]),
                        gbytes=2 * B * G * k3.shape[2] * 256 / 1e9)
                del k3, v3
            del rows, k2, q2, q, qkv2, qkv
        # ---- gated linear attention
        state = 0.01 * torch.randn(B, m.heads, m.np, m.vdp, device=dev)
        decay, wn = L.DecayWeights(0.3 * torch.randn(m.rank, m.keys, device=dev), 2 + f32(m.keys)), f32(m.vdp)
        state_bytes = B * m.heads * m.np * m.vdp * 8
        if T > 1:
            qka, vg = torch.randn(B, T, m.qk + m.rp, device=dev), rand(B, T, 2 * m.inner)
            g, chunks = LC._gated_linear(qka, decay, m), -(-T // 128)
            qk, factor = torch.empty(B, T, m.qk, device=dev, dtype=bf), torch.empty(B, chunks, m.keys, 2, device=dev)
            far = torch.zeros(B, m.heads, dtype=torch.int32, device=dev)
            prep = lambda: cu._check(LC.lib().kvb_gated_linear_prep(LC.ctypes.byref(g), cu._p(qk), cu._p(factor), cu._p(far), cu._p(seq.count), B, T,  # noqa: E731
                                                                    cu._stream(qka)), "prep")
            tab.add(f"{tag}: gated linear: decays, queries and keys", prep, gbytes=n * (6 * m.qk + 4 * m.rp) / 1e9)
            qkv2, cs, wq = rand(B, T, 2 * m.qk), f32(T, 128), rand(128)
            tab.add(f"{tag}:   like: QK norm, split + RoPE", lambda: cu.qknorm_rope_fwd(qkv2, cs, cs, wq, wq, 2 * m.qk // 128 - 16, 8, 128, eps, 128, False),
                    gbytes=8 * n * m.qk / 1e9)
            flop = n * m.heads * (4 * m.np * m.vdp + 128 * (m.np + m.vdp)) / 1e12
            y = torch.empty(B, T, m.inner, device=dev, dtype=bf)
            nbytes = int(LC.lib().kvb_gated_linear_scan_tc_scratch_bytes(B, T, m.heads, m.vdp, m.np))
            scratch = torch.empty(max(nbytes, 16), dtype=torch.uint8, device=dev)
            alone = lambda: cu._check(LC.lib().kvb_gated_linear_scan_tc(  # noqa: E731
                cu._p(vg), cu._ll(2 * m.inner), cu._p(qk), cu._p(factor), cu._p(far), cu._p(state), cu._p(y), cu._p(scratch), cu._p(seq.slots),
                cu._p(seq.start), cu._p(seq.count), B, T, m.heads, m.vdp, m.np, cu._p(cu.status_word(dev)), cu._stream(vg)), "scan")
            tab.add(f"{tag}: gated linear scan, {m.heads} heads of {m.np} x {m.vdp}", alone, gbytes=(n * (2 * m.qk + 4 * m.inner) + state_bytes) / 1e9, tflop=flop)
            tab.add(f"{tag}: gated linear scan with its preparation, {m.heads} heads of {m.np} x {m.vdp}", lambda: LC.gated_linear_scan(qka, vg, decay, state, seq, m),
                    gbytes=(n * (4 * (m.qk + m.rp) + 4 * m.inner) + state_bytes) / 1e9, tflop=flop)
            q2 = rand(B, m.heads, T, 128)
            tab.add(f"{tag}:   like: attention 128 / 128, {m.heads} heads", lambda: cu.sdpa_fwd(q2, q2, q2, 0.09, 0),
                    tflop=2 * B * m.heads * (T * (T + 1) // 2) * 256 / 1e12)
            y = rand(B, T, m.inner)
            tab.add(f"{tag}: gated linear: norm per head, gate", lambda: LC.head_norm_gate(y, vg[..., m.inner :], m, eps, wn), gbytes=6 * n * m.inner / 1e9)
            tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
            del qka, vg, qk, q2, qkv2, y, factor, scratch
        else:
            u = torch.randn(B, 1, m.qk + m.rp + 2 * m.inner, device=dev)
            tab.add(f"{tag}: gated linear step, {m.heads} heads of {m.np} x {m.vdp}", lambda: LC.gated_linear_step(u, decay, wn, state, seq, m, eps, bf),
                    gbytes=(state_bytes + 4 * n * u.shape[-1]) / 1e9)
        del state
        # ---- gated recurrence
        C = r.channels
        u, ring, state, y = rand(B, T, 2 * C), rand(B, r.taps, C), f32(B, C), rand(B, T, C)
        gw = L.RecurrenceWeights(f32(r.taps, C), f32(C), 0.1 * rand(r.blocks, r.pp, 2 * r.pp), f32(C), f32(C), -f32(C))
        if T > 1:
            tab.add(f"{tag}: convolution, {C} channels", lambda: LC.short_conv(u, C, gw.conv, gw.conv_bias, ring, seq, False), gbytes=4 * n * C / 1e9)
            tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
            xc = rand(n, r.blocks, r.pp).transpose(0, 1)
            tab.add(f"{tag}: library products of the gates, fp32 results", lambda: LC.bmm_fp32(xc, gw.gates), gbytes=n * C * 10 / 1e9, tflop=4 * n * C * r.pp / 1e12)
            z, xs = LC.bmm_fp32(xc, gw.gates), rand(B, T, C)
            g = LC._GatedRecurrence(*(t.data_ptr() for t in (gw.conv, gw.conv_bias, gw.bias_r, gw.bias_i, gw.rate, gw.gates)), r.blocks, r.pp, r.taps, 1.0)
            scan = lambda: cu._check(LC.lib().kvb_gated_recurrence_scan(LC.ctypes.byref(g), cu._p(xs), cu._p(z), cu._p(u), cu._ll(2 * C), cu._p(state), cu._p(y),  # noqa: E731
                                                                        cu._ll(C), cu._p(seq.slots), cu._p(seq.start), cu._p(seq.count), B, T, 1,
                                                                        cu._p(cu.status_word(dev)), cu._stream(u)), "scan")
            tab.add(f"{tag}: gated recurrence scan, {C} channels", scan, gbytes=n * C * 14 / 1e9)
            tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
            del z, xs, xc
        else:
            tab.add(f"{tag}: convolution, gates and recurrence step, {C} channels", lambda: LC.gated_recurrence(u, gw, ring, state, seq, r, 1.0, y),
                    gbytes=(n * C * (2 * (2 + r.taps) + 8 + 2) + 4 * C * r.pp) / 1e9)
            tab.add(f"{tag}:   like: (add +) RMSNorm", like_norm, gbytes=norm_bytes)
        # ---- products (library, in both models)
        hn, w3 = rand(n, W), rand(m.qk + m.rp, W)
        tab.add(f"{tag}: library product with fp32 result {n} x {m.qk + m.rp} x {W}", lambda: L.linear_fp32(hn, w3),
                gbytes=(2 * n * W + 2 * m.qk * W + 4 * n * m.qk) / 1e9, tflop=2 * n * m.qk * W / 1e12)
        tab.add(f"{tag}:   like: with bf16 result", lambda: torch.mm(hn, w3.t()), gbytes=2 * (n * W + m.qk * W + n * m.qk) / 1e9, tflop=2 * n * m.qk * W / 1e12)
        del hn, w3, x, sub, h, a, rr, u, ring, state, y
        torch.cuda.empty_cache()
    ops.check_status(dev)
    return tab.rows


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--model", default="Mezilix-2k")
    ap.add_argument("--batch", type=int, default=32)
    ap.add_argument("--prompt", type=int, default=8192)
    ap.add_argument("--decode", type=int, default=128)
    ap.add_argument("--kernels", action="store_true", help="kernel table instead of model throughput")
    ap.add_argument("--n-layer", type=int, default=None)
    args = ap.parse_args()
    config = Config.from_name(args.model)
    if args.n_layer is not None:
        config.layers, config.n_layer = config.layers[: args.n_layer], args.n_layer
    if args.kernels:
        kernel_table(config, args.batch)
        return
    for c in compared(config).values():
        print(json.dumps(throughput(c, args.batch, args.prompt, args.decode)), flush=True)


if __name__ == "__main__":
    main()
