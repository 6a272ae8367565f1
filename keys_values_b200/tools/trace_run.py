"""Replays a trace: feeds given token ids through a model, step by step, and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl
    python -m keys_values_b200 trace_run ...          (the same)

Every line of standard input is a step, ``{"step": 4, "entries": [{"id": "req7", "tokens": [812, 40], "want": [1]}], "end": ["req7"]}``:
the next tokens of each request of the batch and the places among them whose logits are wanted; ``end`` names the requests
that are finished after the step, whose slots are given back. A step with wanted logits writes ``OUT/<step>.f32``
(little-endian fp32, ``[wanted, vocab]``, in the order of the entries); after every step ``done <step>`` is printed.

The model is the one that generation uses, driven through the same calls: several tokens per request are one
:meth:`forward` over right-padded rows, single tokens go through :class:`keys_values_b200.generate.decode_graph.Decoder`
(captured steps while the batch stays the same). With ``float32`` every product is in full 32 bits.
"""
from __future__ import annotations

import json
import sys
from pathlib import Path
from typing import Dict, List, Optional, TextIO

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class TraceRunner:
    """Slots, batches and steps of one model; ``step`` is one line of a trace."""

    def __init__(self, model, max_tokens: int, cache_name: Optional[str] = None, use_graph: bool = True):
        from keys_values_b200.models.registry import default_cache_name

        if model.config.layers is None:
            raise NotImplementedError("trace replay needs a model that keeps a position per request")
        self.model = model
        self.max_tokens = max_tokens
        self.cache_name = default_cache_name(model.config, cache_name)
        self.use_graph = use_graph
        self.slots: Dict[str, int] = {}
        self.lengths: Dict[str, int] = {}
        self._decoder = None
        self._decoder_slots = None
        self.capacity = 0

    def _reserve(self, n: int) -> None:
        """Caches for ``n`` requests at a time; they can only be made anew while no request is live."""
        if n <= self.capacity:
            return
        if self.slots:
            raise ValueError(f"{n} requests at a time, but the caches were made for {self.capacity}")
        from keys_values_b200.kvcache.factory import KVCacheFactory

        m = self.model
        w = m.lm_head.weight
        self._decoder = None
        m.assign_kv_caches(KVCacheFactory.create(m, self.cache_name, n, self.max_tokens, device=w.device, dtype=w.dtype))
        self.capacity = n

    @torch.inference_mode()
    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """Logits of the wanted places ``(wanted, vocab)`` fp32, or ``None`` if there are none."""
        m, vocab = self.model, self.model.config.padded_vocab_size
        ids = [e["id"] for e in entries]
        if len(set(ids)) != len(ids):
            raise ValueError("a request occurs twice in a step")
        for e in entries:
            if not e["tokens"] or any(not 0 <= t < vocab for t in e["tokens"]):
                raise ValueError(f"request {e['id']}: tokens must be non-empty and lie in [0, {vocab})")
            if any(not 0 <= w < len(e["tokens"]) for w in e["want"]):
                raise ValueError(f"request {e['id']}: wanted places lie outside of the step")
        out = None
        if entries:
            new = [i for i in ids if i not in self.slots]
            self._reserve(len(self.slots) + len(new))
            for i in new:
                self.slots[i] = m.sequences.acquire()
                self.lengths[i] = 0
            batch = tuple(self.slots[i] for i in ids)
            m.sequences.set_batch(batch)
            dev = m.lm_head.weight.device
            counts = [len(e["tokens"]) for e in entries]
            T = max(counts)
            idx = torch.tensor([e["tokens"] + [0] * (T - len(e["tokens"])) for e in entries], dtype=torch.int64).to(dev)
            want = [b * T + w for b, e in enumerate(entries) for w in e["want"]]
            rows = torch.tensor(want, dtype=torch.int64).to(dev)
            if T == 1 and not new:
                out = self._decode(batch, idx)[:, 0].float()
                out = out.index_select(0, rows) if want else None
            elif want:
                out = m(idx, counts=counts, rows=rows)
            else:
                m(idx, counts=counts, skip_lm_head=True)
            for e in entries:
                self.lengths[e["id"]] += len(e["tokens"])
        for i in end:
            m.sequences.release(self.slots.pop(i))
            del self.lengths[i]
        return out

    def _decode(self, batch, idx: torch.Tensor) -> torch.Tensor:
        from keys_values_b200.generate.decode_graph import Decoder

        if self._decoder is None or self._decoder_slots != batch:
            self._decoder = Decoder(self.model, len(batch), use_graph=self.use_graph and idx.is_cuda)
            self._decoder_slots = batch
        return self._decoder(idx)


def load_model(model_dir: Path, dtype: torch.dtype, device: torch.device):
    """The model of a checkpoint directory, with its weights, for inference."""
    from keys_values_b200.config import Config
    from keys_values_b200.finetune.utils import load_model_checkpoint
    from keys_values_b200.models.registry import create_model

    config = Config.from_checkpoint(model_dir)
    with torch.device(device):
        model = create_model(config).to(dtype)
    load_model_checkpoint(model, model_dir)
    return model.eval()


def run(model_dir: Path, dtype: str, out_dir: Path, max_tokens: int, steps: TextIO, report: TextIO, device: Optional[torch.device] = None) -> None:
    from keys_values_b200 import ops

    device = torch.device("cuda", 0) if device is None else device
    if device.type == "cuda":
        from keys_values_b200 import build_ext

        build_ext.build(libs=[build_ext.LAYERS_LIB])  # first call in a fresh checkout; otherwise nothing to do
        if not torch.cuda.is_available():
            raise RuntimeError("trace replay needs a GPU")
    torch.set_float32_matmul_precision("highest")
    runner = TraceRunner(load_model(model_dir, DTYPES[dtype], device), max_tokens)
    out_dir.mkdir(parents=True, exist_ok=True)
    for line in steps:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step(step["entries"], step.get("end", []))
        if logits is not None:
            data = logits.contiguous().cpu().numpy().astype("<f4", copy=False)
            ops.check_status(device)
            part = out_dir / f"{step['step']}.f32.part"
            part.write_bytes(data.tobytes())
            part.replace(out_dir / f"{step['step']}.f32")
        print(f"done {step['step']}", file=report, flush=True)


def setup(model: Path, dtype: str, out: Path, max_tokens: int) -> None:
    """Entry point of ``python -m keys_values_b200 trace_run``."""
    if dtype not in DTYPES:
        raise SystemExit(f"--dtype must be one of {sorted(DTYPES)}")
    run(Path(model), dtype, Path(out), int(max_tokens), sys.stdin, sys.stdout)
