"""Decoder models whose layers are described one by one (``config.layers``).

Each entry of ``config.layers`` names its mixer and its feed-forward with their own sizes, so the layers of a model may
differ. The mechanisms are modules of their own, picked by the description:

* :class:`LatentAttention`: low-rank keys and values (one latent per token plus one rotated key part that the heads
  share), optional sliding window, ring cache of latents (:class:`keys_values_b200.kvcache.latent.LatentKVCache`);
* :class:`keys_values_b200.models.grouped_attention.GroupedAttention`: grouped-query attention with optional norm of queries and
  keys, windows (also with pooled blocks before them) or chunks, keys and values of another layer, values shared with the keys, soft cap, softmax
  sink, output gate and differential maps;
* :class:`keys_values_b200.models.state_space.Mamba2Mixer`: state-space recurrence;
* :class:`keys_values_b200.models.retention.Retention`: linear attention with a fixed decay per head;
* :class:`keys_values_b200.models.gated_linear.GatedLinearAttention`: linear attention with a decay per token and key channel;
* :class:`keys_values_b200.models.gated_recurrence.GatedRecurrence`: short convolution and a gated recurrence per channel;
* :class:`keys_values_b200.models.side_by_side.SideBySide`: two mixers on the same input;
* :class:`RoutedMLP`: softmax or sigmoid router, top-k experts with or without gates, optionally a shared expert;
  :class:`DenseMLP`: two matrices and an activation; :class:`GatedMLP`: three matrices, silu or a clamped unit;
* :class:`ScalarRMSNorm`: RMS norm with one gain for all coordinates; :class:`StreamNorm`: layer or RMS norm of the fp32 stream;
* token shift (``config.token_shift``): the mixer reads a learned blend of the token's normed input and the previous token's;
* depth average (``config.depth_average``): what goes on to the next layer is a learned average of the embedding output
  and all layers' results so far;
* bigram embedding (``config.bigram``): a hashed row for the pair (previous token, token) is added to the embedding;
* position table (``config.position_table``): a learned vector per position is added to the embedding;
* input convolution (``config.input_conv``): what a sublayer reads becomes itself plus a causal convolution of itself;
* loop (``config.loop``): a run of layers is passed several times, with a cache or state of its own each time.

Two kinds of layers: :class:`ParallelBlock` (mixer and feed-forward read one norm's output) and :class:`SequentialBlock` (one
after the other, each with a norm before it, after it or both). The residual stream and the depth history are fp32. What lies between two sublayers
that depend on each other (residual sum, norms, weighted expert outputs, depth average, token shift, what a loop adds) is one
kernel, :func:`keys_values_b200.ops.layers.layer_edge` or :func:`keys_values_b200.ops.layers.norm_edge`; therefore the stream
that :meth:`LayeredGPT.run_layer` hands on is a :class:`LayerStream`, which carries the next layer's normed inputs along.
"""
from __future__ import annotations

from functools import partial
from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from keys_values_b200.config import STREAM_NORMS, Config
from keys_values_b200.kvcache.grouped import BorrowedKVCache
from keys_values_b200.kvcache.layer_cache import MAX_PASS_TOKENS, LayerCache
from keys_values_b200.kvcache.sequences import SequencePass, SequenceTable
from keys_values_b200.models.gated_linear import GatedLinearAttention
from keys_values_b200.models.gated_recurrence import GatedRecurrence
from keys_values_b200.models.grouped_attention import GroupedAttention
from keys_values_b200.models.model import GPT
from keys_values_b200.models.packed import Packed, pad_groups, pad_last
from keys_values_b200.models.retention import Retention
from keys_values_b200.models.side_by_side import SideBySide
from keys_values_b200.models.state_space import Mamba2Mixer
from keys_values_b200.ops import layers as L

# fp32 bytes of residual streams (depth history included) that one pass of a chunked prefill may hold
MAX_STREAM_BYTES = 4 * 2**30


def latent_shape(spec: Dict[str, Any]) -> L.LatentShape:
    return L.LatentShape(heads=spec["n_head"], dim=spec["dim"], rot=spec["rot_dim"], vdim=spec["v_dim"], kv_rank=spec["kv_rank"],
                         rot_dims=spec.get("rope_dims", spec["rot_dim"]))


class ScalarRMSNorm(nn.Module):
    """``x / rms(x) · weight`` with a single number as weight."""

    def __init__(self, size: int, eps: float = 1e-5) -> None:
        super().__init__()
        self.weight = nn.Parameter(torch.ones(()))
        self.size = size
        self.eps = eps

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        y = L.scalar_rmsnorm(x.reshape(-1, self.size).float(), self.weight.float(), self.eps, self.weight.dtype)
        return y.view(x.shape)

    def reset_parameters(self) -> None:
        nn.init.ones_(self.weight)


class StreamNorm(Packed):
    """Layer norm (``center``) or RMS norm of fp32 rows with one weight per coordinate and no bias. ``unit_offset``: the weight is stored
    around zero, the norm is multiplied by 1 + weight."""

    def __init__(self, size: int, eps: float = 1e-5, center: bool = True, unit_offset: bool = False) -> None:
        super().__init__()
        self.weight = nn.Parameter(torch.zeros(size) if unit_offset else torch.ones(size))
        self.eps = eps
        self.center = center
        self.unit_offset = unit_offset

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        rows = x.reshape(-1, self.weight.numel()).float().contiguous()
        return L.row_norm(rows, self.packed()["weight"], self.eps, self.center, self.weight.dtype).view(x.shape)

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        w = self.weight.float()
        return {"weight": (1.0 + w if self.unit_offset else w).contiguous()}

    def reset_parameters(self) -> None:
        nn.init.constant_(self.weight, 0.0 if self.unit_offset else 1.0)


class LatentAttention(Packed):
    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        spec = config.layers[block_idx]["mixer"]
        s = self.shape = latent_shape(spec)
        if not spec["scale"] > 0:
            raise ValueError(f"layer {block_idx}: attention scale must be positive")
        self.scale = float(spec["scale"])
        self.window = int(spec.get("window") or 0)
        self.rope_base = float(spec["rope_base"])
        self.eps = config.norm_eps
        # rows: queries head by head [unrotated | rotated], latent, shared rotated key part
        self.qkv = nn.Linear(config.n_embd, s.heads * (s.dim + s.rot) + s.kv_rank + s.rot, bias=False)
        self.norm_kv = nn.Parameter(torch.ones(s.kv_rank))
        self.key = nn.Linear(s.kv_rank, s.heads * s.dim, bias=False)
        self.value = nn.Linear(s.kv_rank, s.heads * s.vdim, bias=False)
        self.proj = nn.Linear(s.heads * s.vdim, config.n_embd, bias=False)
        self.kv_cache = kv_cache
        self.config = config
        self.block_idx = block_idx

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        s = self.shape
        w = self.qkv.weight
        key = F.pad(self.key.weight.view(s.heads, s.dim, s.kv_rank), (0, s.kvp - s.kv_rank, 0, s.dimp - s.dim)).contiguous()
        value = F.pad(self.value.weight.view(s.heads, s.vdim, s.kv_rank), (0, s.kvp - s.kv_rank, 0, s.vdp - s.vdim))
        exps = torch.arange(s.rot_dims // 2, dtype=torch.float64) * (-2.0 / s.rot_dims)
        return {
            "norm": self.norm_kv.float().contiguous(),
            "freq": (self.rope_base**exps).to(device=w.device, dtype=torch.float32),
            "key": key,  # (heads, dimp, kvp)
            "value_t": value.transpose(1, 2).contiguous(),  # (heads, kvp, vdp)
            "key_value": torch.cat((key, value), dim=1).view(-1, s.kvp).contiguous(),  # rows of a head: [key | value]
            "proj": pad_last(self.proj.weight.view(-1, s.heads, s.vdim), s.vdp).view(-1, s.heads * s.vdp),
        }

    def forward(self, x: torch.Tensor, seq: SequencePass, turn: int = 0) -> torch.Tensor:
        """``x (B, T, width)`` → ``(B, T, width)``; the cache takes the rows of the pass."""
        B, T, _ = x.shape
        s, w = self.shape, self.packed()
        qkv = F.linear(x, self.qkv.weight)
        ring = self.kv_cache.allocate(x.device, x.dtype)[0][turn]
        if T == 1:
            q = L.latent_prep(qkv, w["norm"], w["freq"], None, ring, seq, 0, s, self.eps)
            q_abs = torch.bmm(q[:, 0, :, : s.dimp].transpose(0, 1), w["key"])  # W_uk folded into the query
            lat = L.latent_decode(q_abs, q, ring, seq, s, self.scale)
            y = torch.empty((B, s.heads, s.vdp), dtype=x.dtype, device=x.device)
            torch.bmm(lat, w["value_t"], out=y.transpose(0, 1))
            return F.linear(y.view(B, 1, -1), w["proj"])
        # rows before the pass that its first tokens still see
        P = seq.max_start if self.window == 0 else min(seq.max_start, self.window - 1)
        latent = torch.empty((B, P + T, s.row), dtype=x.dtype, device=x.device)
        L.ring_gather(ring, latent, seq, P)
        q = L.latent_prep(qkv, w["norm"], w["freq"], latent, ring, seq, P, s, self.eps)
        kv = torch.mm(latent.view(-1, s.row)[:, : s.kvp], w["key_value"].t())
        y = L.latent_attend(q, kv, latent, seq, P, s, self.window, self.scale)
        return F.linear(y, w["proj"])

    def check_kv_cache(self, cache) -> None:
        from keys_values_b200.kvcache.latent import LatentKVCache

        if not isinstance(cache, LatentKVCache):
            raise ValueError(f"{type(cache).__name__} does not fit a latent-attention layer (use cache name 'latent-default')")
        if cache.shape != self.shape:
            raise ValueError(f"cache of layer {cache.block_idx} has sizes {cache.shape}, the layer has {self.shape}")

    def create_default_kv_cache(self, batch_size: int, dtype=None, max_sequence_length: Optional[int] = None, device=None) -> None:
        from keys_values_b200.kvcache.latent import LatentKVCache

        length = self.config.block_size if max_sequence_length is None else max_sequence_length
        self.kv_cache = LatentKVCache(self.config, batch_size, length, self.block_idx, dtype=dtype, device=device)


class RoutedMLP(Packed):
    """``Σ over the chosen experts of weight_e · down_e(act(up_e(x)))``. Returns the experts' outputs unsummed (the sum is
    part of the kernel that closes the sublayer).

    Entries of the description: ``n_expert``, ``top``, ``ff``; ``activation`` (``"silu_gated"``: the rows of ``up`` are those of
    the gate projection, then those of the up projection); ``score`` ``"softmax"`` or ``"sigmoid"``; ``renormalize`` (the chosen scores
    are divided by their sum + ``renormalize_eps``); ``correction``: a learned number per expert that is added to the scores for the choice
    only; ``groups`` ``{"count", "keep"}``: only experts of the best groups can be chosen; ``shared``: width of a gated
    feed-forward that every token passes (``self.shared``, summed by the caller)."""

    def __init__(self, config: Config, spec: Dict[str, Any]) -> None:
        super().__init__()
        E, ff, width = spec["n_expert"], spec["ff"], config.n_embd
        groups = spec.get("groups") or dict(count=1, keep=1)
        if not 0 < spec["top"] <= E:
            raise ValueError(f"top = {spec['top']} of {E} experts")
        if E % groups["count"] or not 0 < groups["keep"] <= groups["count"] or spec["top"] > groups["keep"] * (E // groups["count"]):
            raise ValueError(f"top = {spec['top']} of {E} experts in groups {groups}")
        self.activation = spec.get("activation", "relu_squared")
        if self.activation not in L.ACTIVATIONS:
            raise ValueError(f"activation {spec['activation']!r}")
        if spec.get("score", "softmax") not in ("softmax", "sigmoid"):
            raise ValueError(f"score {spec['score']!r}")
        self.spec = spec
        self.rule = L.RouterRule(score=spec.get("score", "softmax"), groups=groups["count"], keep=groups["keep"],
                                 renormalize=bool(spec.get("renormalize", False)), eps=float(spec.get("renormalize_eps", 0.0)))
        self.ff = ff
        self.gate = nn.Linear(width, E, bias=False)
        self.correction = nn.Parameter(torch.zeros(E)) if spec.get("correction") else None
        self.up = nn.Parameter(torch.empty(E, 2 * ff if self.activation == "silu_gated" else ff, width))
        self.down = nn.Parameter(torch.empty(E, width, ff))
        self.shared = GatedMLP(config, dict(ff=spec["shared"])) if spec.get("shared") else None
        for p in (self.up, self.down):
            nn.init.normal_(p, mean=0.0, std=0.02)

    def _make_pack(self) -> Dict[str, Optional[torch.Tensor]]:
        E, rows, width = self.up.shape
        up = self.up.detach()
        if self.activation == "silu_gated":  # gate and up projection of a result in neighbouring rows
            up = up.view(E, 2, self.ff, width).transpose(1, 2).reshape(E, rows, width)
        return {"up": pad_last(up, L.round8(width)), "down": pad_last(self.down.detach(), L.round8(self.ff)),
                "correction": None if self.correction is None else self.correction.float().contiguous()}

    def forward(self, x: torch.Tensor):
        width = self.up.shape[2]
        w = self.packed()
        x = x.reshape(-1, width)
        logits = L.linear_fp32(x, self.gate.weight)
        return L.routed_experts(x, logits, w["up"], w["down"], self.spec["top"], self.activation, self.rule, self.ff, width, w["correction"])


class GatedMLP(Packed):
    """``down(silu(gate x) · up x)``; gate and up projection are one product, rows ``[gate | up]``. With a ``limit``: the clamped unit of
    :func:`keys_values_b200.ops.layers.glu` instead."""

    def __init__(self, config: Config, spec: Dict[str, Any]) -> None:
        super().__init__()
        self.ff = spec["ff"]
        self.limit = None if spec.get("limit") is None else float(spec["limit"])
        if self.limit is not None and not self.limit > 0:
            raise ValueError(f"limit = {self.limit} of a gated feed-forward must be positive")
        self.up = nn.Linear(config.n_embd, 2 * self.ff, bias=False)
        self.down = nn.Linear(self.ff, config.n_embd, bias=False)

    def _make_pack(self) -> Dict[str, torch.Tensor]:
        n = L.round8(self.ff)
        return {"up": pad_groups(self.up.weight.detach(), 2, n), "down": pad_last(self.down.weight.detach(), n)}

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        w = self.packed()
        return F.linear(L.glu(F.linear(x, w["up"]), self.ff, self.limit), w["down"])


class DenseMLP(nn.Module):
    """``down(act(up x))``."""

    def __init__(self, config: Config, spec: Dict[str, Any]) -> None:
        super().__init__()
        self.activation = spec.get("activation", "relu_squared")
        if self.activation not in ("none", "relu_squared"):
            raise ValueError(f"activation {self.activation!r}")
        self.up = nn.Linear(config.n_embd, spec["ff"], bias=False)
        self.down = nn.Linear(spec["ff"], config.n_embd, bias=False)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return F.linear(L.activate(F.linear(x, self.up.weight), self.activation), self.down.weight)


MIXERS = {
    "latent_attention": LatentAttention, "grouped_attention": GroupedAttention, "mamba2": Mamba2Mixer, "retention": Retention,
    "gated_linear_attention": GatedLinearAttention, "gated_recurrence": GatedRecurrence, "side_by_side": SideBySide,
}
FEED_FORWARDS = {"routed": RoutedMLP, "dense": DenseMLP, "gated": GatedMLP}


class ParallelBlock(Packed):
    """Mixer and feed-forward read the output of one norm; token shift and depth average belong to the layer's edge."""

    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        spec = config.layers[block_idx]
        self.norm_1 = config.norm_class(config.n_embd, eps=config.norm_eps)
        self.attn = MIXERS[spec["mixer"]["kind"]](config, block_idx, kv_cache)
        self.mlp = None if spec.get("mlp") is None else FEED_FORWARDS[spec["mlp"]["kind"]](config, spec["mlp"])
        self.shift = nn.Parameter(torch.zeros(config.n_embd)) if config.token_shift else None
        self.depth = None
        if config.depth_average:  # the identity: all weight on the layer's own result
            self.depth = nn.Parameter(F.one_hot(torch.tensor(block_idx + 1), block_idx + 2).float())
        if config.input_conv or config.residual_mult != 1.0 or config.position_table:
            raise NotImplementedError("input convolution, residual factor and position table go with sequential layers")
        if config.loop is not None or not (self.mlp is None or isinstance(self.mlp, RoutedMLP) and self.mlp.shared is None):
            raise NotImplementedError("parallel layers are not run in loops and have routed feed-forwards without a shared expert")
        if not (config.norm_1 and config.norm_2) or config.post_attention_norm or config.post_mlp_norm:
            raise NotImplementedError("parallel layers have one norm, ahead of mixer and feed-forward")
        self.config = config
        self.block_idx = block_idx

    def _make_pack(self) -> Dict[str, Optional[torch.Tensor]]:
        return {
            "gain": self.norm_1.weight.float().contiguous(),
            "shift": None if self.shift is None else self.shift.float().contiguous(),
            "depth": None if self.depth is None else self.depth.float().contiguous(),
        }

    @staticmethod
    def _shift_state(model: "LayeredGPT", block_idx: int) -> Optional[torch.Tensor]:
        return None if model.sequences.shift is None else model.sequences.shift[block_idx]

    def enter(self, model: "LayeredGPT", idx: torch.Tensor, seq: SequencePass) -> "LayerStream":
        """The stream in front of this (the first) layer."""
        c = self.config
        wte = model.transformer.wte.weight
        B, T = idx.shape
        dev, dt = wte.device, wte.dtype
        history = torch.empty((c.n_layer + 1, B, T, c.n_embd), dtype=torch.float32, device=dev) if c.depth_average else None
        x = history[0] if history is not None else torch.empty((B, T, c.n_embd), dtype=torch.float32, device=dev)
        h = torch.empty((B, T, c.n_embd), dtype=dt, device=dev)
        shifted = torch.empty_like(h) if c.token_shift else None
        w = self.packed()
        bg = c.bigram or dict(buckets=0, mul_prev=0, mul_cur=0)
        L.embed_edge(idx, model.sequences.prev_token, wte, None if model.bigram is None else model.bigram.weight, bg["buckets"], bg["mul_prev"],
                     bg["mul_cur"], x, w["gain"], w["shift"], self._shift_state(model, 0), h, shifted, seq, c.norm_eps)
        return LayerStream(seq, x, history, h, shifted)

    def run(self, model: "LayeredGPT", run: int, x: "LayerStream", idx: torch.Tensor) -> "LayerStream":
        c, block_idx = self.config, self.block_idx
        mixed = self.attn(x.h if x.shifted is None else x.shifted, x.seq)
        experts = None if self.mlp is None else self.mlp(x.h)
        nxt = model.transformer.h[block_idx + 1].packed() if block_idx + 1 < c.n_layer else {"gain": None, "shift": None}
        state = self._shift_state(model, block_idx + 1) if nxt["shift"] is not None else None
        out = x.spare if x.spare is not None else torch.empty_like(x.x)
        L.layer_edge(x.x, mixed, experts, x.history, block_idx + 1, self.packed()["depth"], out, nxt["gain"], nxt["shift"], state,
                     x.h, x.shifted, x.seq, c.norm_eps)
        x.spare = None if x.history is not None and block_idx == 0 else x.x  # the embedding output stays in the history
        x.x = out
        return x


class SequentialBlock(Packed):
    """Norm, mixer, norm, residual sum; then the same with the feed-forward. The norms before the sublayers (``config.norm_1``,
    ``norm_2``; without them a sublayer reads the stream itself) and after them (``post_attention_norm``, ``post_mlp_norm``) are
    optional."""

    def __init__(self, config: Config, block_idx: int, kv_cache=None) -> None:
        super().__init__()
        spec = config.layers[block_idx]
        if config.norm_class_name not in STREAM_NORMS:
            raise ValueError(f"norm {config.norm_class_name!r}: sequential layers take one of {sorted(STREAM_NORMS)}")
        norm = partial(config.norm_class, config.n_embd, eps=config.norm_eps)
        self.norm_1 = norm() if config.norm_1 else None
        self.attn = MIXERS[spec["mixer"]["kind"]](config, block_idx, kv_cache)
        self.post_attention_norm = norm() if config.post_attention_norm else None
        self.mlp = None if spec.get("mlp") is None else FEED_FORWARDS[spec["mlp"]["kind"]](config, spec["mlp"])
        self.norm_2 = norm() if self.mlp is not None and config.norm_2 else None
        self.post_mlp_norm = norm() if self.mlp is not None and config.post_mlp_norm else None
        if config.token_shift or config.depth_average or config.bigram is not None:
            raise NotImplementedError("token shift, depth average and bigram embedding go with parallel layers")
        self.conv_1 = self.conv_2 = None
        if config.input_conv:  # (width, taps), the last column meets the token itself
            self.conv_1 = nn.Parameter(torch.zeros(config.n_embd, config.input_conv))
            self.conv_2 = None if self.mlp is None else nn.Parameter(torch.zeros(config.n_embd, config.input_conv))
        if config.residual_mult != 1.0 and (self.post_attention_norm is None or self.mlp is not None and self.post_mlp_norm is None):
            raise NotImplementedError("a residual factor goes with norms after the sublayers, whose weights take it")
        self.center = STREAM_NORMS[config.norm_class_name]["center"]
        self.config = config
        self.block_idx = block_idx

    def _make_pack(self) -> Dict[str, Optional[torch.Tensor]]:
        mult = self.config.residual_mult
        norms = dict(norm_1=(self.norm_1, 1.0), after_1=(self.post_attention_norm, mult), norm_2=(self.norm_2, 1.0), after_2=(self.post_mlp_norm, mult))
        pack = {k: None if n is None else n.packed()["weight"] * f for k, (n, f) in norms.items()}
        for k, w in dict(conv_1=self.conv_1, conv_2=self.conv_2).items():
            pack[k] = None
            if w is not None:  # h + convolution of h as one convolution
                pack[k] = w.detach().float().t().clone(memory_format=torch.contiguous_format)
                pack[k][-1] += 1
        return pack

    def _edge(self, model: "LayeredGPT", x: "LayerStream", y, after, before, conv, edge: int, want_h: bool = True, **kw: Any) -> None:
        """From a sublayer's result to the next one's input, the ``edge``-th in the pass; ``conv``: what that input passes."""
        tokens = None if conv is None else L.EdgeTokens(x.seq, None, conv, model.sequences.conv[edge])
        L.norm_edge(x.x, y, after, x.x, before, x.h if want_h else None, kw.get("idx"), kw.get("embed"), kw.get("step"), self.config.norm_eps, self.center,
                    kw.get("experts"), tokens)

    def enter(self, model: "LayeredGPT", idx: torch.Tensor, seq: SequencePass) -> "LayerStream":
        """The stream in front of this (the first) layer."""
        wte = model.transformer.wte.weight
        x = torch.empty((*idx.shape, self.config.n_embd), dtype=torch.float32, device=wte.device)
        h = torch.empty(x.shape, dtype=wte.dtype, device=wte.device)
        w, table = self.packed(), None if model.positions is None else model.positions.weight
        ring = None if w["conv_1"] is None else model.sequences.conv[0]
        tokens = None if table is None and ring is None else L.EdgeTokens(seq, table, w["conv_1"], ring)
        L.norm_edge(None, None, None, x, w["norm_1"], h, idx, wte, model.ahead_of_run(0)[1], self.config.norm_eps, self.center, None, tokens)
        return LayerStream(seq, x, None, h, None)

    def run(self, model: "LayeredGPT", run: int, x: "LayerStream", idx: torch.Tensor) -> "LayerStream":
        w = self.packed()
        y, after, experts = self.attn(x.h, x.seq, model.runs[run][1]), w["after_1"], None
        if self.mlp is not None:
            self._edge(model, x, y, after, w["norm_2"], w["conv_2"], 2 * run + 1)
            after = w["after_2"]
            if isinstance(self.mlp, RoutedMLP):
                y = None if self.mlp.shared is None else self.mlp.shared(x.h)
                experts = self.mlp(x.h)
            else:
                y = self.mlp(x.h)
        last = run + 1 == model.n_runs
        nxt = {"norm_1": None, "conv_1": None} if last else model.transformer.h[model.runs[run + 1][0]].packed()
        add_embedding, step = (False, None) if last else model.ahead_of_run(run + 1)
        self._edge(model, x, y, after, nxt["norm_1"], nxt["conv_1"], 2 * run + 2, not last, idx=idx.contiguous() if add_embedding else None,
                   embed=model.transformer.wte.weight if add_embedding else None, step=step, experts=experts)
        return x


class LayerStream:
    """What one layer hands to the next: the fp32 residual stream, the depth history and the next layer's inputs."""

    carries_state = True  # not replaceable by its dense tensor

    def __init__(self, seq: SequencePass, x: torch.Tensor, history: Optional[torch.Tensor], h: torch.Tensor, shifted: Optional[torch.Tensor]):
        self.seq = seq
        self.x = x  # (B, T, width) fp32
        self.history = history  # (n_layer + 1, B, T, width) fp32: embedding output, then every layer's result
        self.h = h  # normed input of the next layer
        self.shifted = shifted  # what the next layer's mixer reads
        self.spare: Optional[torch.Tensor] = None  # retired stream buffer

    def full(self) -> torch.Tensor:
        return self.x


class LayeredGPT(GPT):
    """:class:`GPT` for configs with ``layers``. Rows of a batch may have different lengths: ``counts`` of
    :meth:`forward` says how many tokens of each (right-padded) row are real."""

    tracks_positions = True

    def __init__(self, config: Config, **mha_kwargs) -> None:
        if config.layers is None or len(config.layers) != config.n_layer:
            raise ValueError("config.layers must describe every layer")
        super().__init__(config, **mha_kwargs)
        self.runs: List[Tuple[int, int]] = config.layer_runs()
        self.loop_step = None
        if config.loop is not None and config.loop.get("step_vectors"):
            self.loop_step = nn.Parameter(torch.zeros(config.loop["times"], config.n_embd))
        self._loop_pack: Optional[torch.Tensor] = None
        self.bigram = None
        if config.bigram is not None:  # the last row is for tokens without a predecessor
            self.bigram = nn.Embedding(config.bigram["buckets"] + 1, config.n_embd)
        self.positions = nn.Embedding(config.block_size, config.n_embd) if config.position_table else None
        self.sequences: Optional[SequenceTable] = None
        if config.tie_embeddings:
            self.lm_head.weight = self.transformer.wte.weight

    def _make_block(self, config: Config, block_idx: int) -> nn.Module:
        return (ParallelBlock if config.parallel_residual else SequentialBlock)(config, block_idx)

    @property
    def n_runs(self) -> int:
        return len(self.runs)

    def block_of_run(self, run: int) -> int:
        return self.runs[run % len(self.runs)][0]

    def ahead_of_run(self, run: int) -> Tuple[bool, Optional[torch.Tensor]]:
        """What the loop adds to the stream right before layer run ``run``: the embedding output or not, a vector or none."""
        loop = self.config.loop
        block_idx, turn = self.runs[run]
        if loop is None or block_idx != loop["start"]:
            return False, None
        if self.loop_step is None:
            return turn > 0 and bool(loop.get("add_embedding")), None
        if self._loop_pack is None:
            with torch.inference_mode(False), torch.no_grad():
                self._loop_pack = self.loop_step.float().contiguous()
        return turn > 0 and bool(loop.get("add_embedding")), self._loop_pack[turn]

    def _apply(self, fn, *args, **kwargs):
        self._loop_pack = None
        return super()._apply(fn, *args, **kwargs)

    def _load_from_state_dict(self, *args: Any, **kwargs: Any) -> None:
        self._loop_pack = None
        super()._load_from_state_dict(*args, **kwargs)

    def _make_mha(self, config: Config, **mha_kwargs) -> None:
        return None  # positions, windows and scales belong to the layers

    def _init_weights(self, module: nn.Module) -> None:
        super()._init_weights(module)
        if isinstance(module, RoutedMLP):
            nn.init.normal_(module.up, mean=0.0, std=0.02)
            nn.init.normal_(module.down, mean=0.0, std=0.02)
        if isinstance(module, (Mamba2Mixer, GatedLinearAttention, GatedRecurrence)):
            module.reset_parameters()
        if isinstance(module, Packed):
            module.drop_pack()

    @property
    def max_seq_length(self) -> int:
        return self._max_seq_length

    @max_seq_length.setter
    def max_seq_length(self, value: int) -> None:
        if value <= 0:
            raise ValueError(f"value = {value}, must be positive")
        self._max_seq_length = value  # angles are computed per position: nothing is sized by the context

    # ---------------------------------------------------------------- caches
    def _check_kv_cache(self, cache) -> None:
        if cache is None:
            return
        if not isinstance(cache, LayerCache):
            raise ValueError(f"{type(cache).__name__} does not fit a model with described layers (use cache name 'layered-default')")
        self.transformer.h[cache.block_idx].attn.check_kv_cache(cache)

    def assign_kv_caches(self, kv_caches: Sequence[Any]) -> None:
        super().assign_kv_caches(kv_caches)
        self._make_sequences()

    def set_kv_caches(self, batch_size: int, dtype=None, max_seq_length: Optional[int] = None, device=None) -> None:
        super().set_kv_caches(batch_size, dtype, max_seq_length, device)
        self._make_sequences()

    def _make_sequences(self) -> None:
        caches = self.get_kv_caches()
        self.sequences = None
        if any(c is None for c in caches):
            return
        c = self.config
        self.sequences = SequenceTable(min(x.max_batch_size for x in caches), self.lm_head.weight.device,
                                       c.n_layer if c.token_shift else 0, c.n_embd, 2 * self.n_runs if c.input_conv else 0, c.input_conv,
                                       self.lm_head.weight.dtype)
        for x in caches:
            x.sequences = self.sequences
            if isinstance(x, BorrowedKVCache):
                x.set_source(caches[x.spec["kv_from"]])

    def clear_kv_caches(self) -> None:
        super().clear_kv_caches()
        self.sequences = None

    def reset(self) -> None:
        super().reset()
        if self.sequences is not None:
            self.sequences.reset()

    def advance_host_counters(self) -> None:
        end = 1 + max(self.sequences.pos_host[s] for s in self.sequences.batch)
        self._check_positions(end)
        for cache in self.get_kv_caches():
            cache.check_capacity(end)
        self.sequences.advance_host()

    def _check_positions(self, end: int) -> None:
        if self.positions is not None and end > self.positions.num_embeddings:
            raise IndexError(f"{end} tokens exceed the table of {self.positions.num_embeddings} positions")

    def max_pass_tokens(self, batch_size: int) -> int:
        """Tokens per row that one pass of a chunked prefill may take."""
        c = self.config
        per_token = 4 * c.n_embd * ((c.n_layer + 1 if c.depth_average else 0) + 2)
        return max(1, min(MAX_STREAM_BYTES // per_token, MAX_PASS_TOKENS) // batch_size)

    # --------------------------------------------------------------- forward
    def embed(self, idx: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError("the embedding is part of begin_pass")

    def begin_pass(self, idx: torch.Tensor, counts: Optional[Sequence[int]] = None) -> LayerStream:
        if self.sequences is None:
            raise ValueError("KV caches must be assigned to the model (see KVCacheFactory.create)")
        if torch.is_grad_enabled():
            raise NotImplementedError("models with described layers run in inference only (use torch.inference_mode())")
        seq = self.sequences.begin(*idx.shape, counts)
        self._check_positions(seq.max_end)
        for cache in self.get_kv_caches():
            cache.check_pass(seq)
        return self.transformer.h[0].enter(self, idx.contiguous(), seq)

    def run_layer(self, run: int, x: LayerStream, idx: torch.Tensor, chunk_sizes: Optional[Sequence[int]] = None) -> LayerStream:
        return self.transformer.h[self.runs[run][0]].run(self, run, x, idx)

    def end_pass(self, x: LayerStream, idx: torch.Tensor) -> torch.Tensor:
        self.sequences.finish(x.seq, idx.contiguous())
        return x.x

    def head(self, x: torch.Tensor) -> torch.Tensor:
        """Logits in fp32."""
        rows = x.reshape(-1, self.config.n_embd).contiguous()
        return L.linear_fp32(self.transformer.ln_f(rows), self.lm_head.weight).view(*x.shape[:-1], -1)

    def clone(self, device: Optional[torch.device] = None) -> "LayeredGPT":
        sequences, self.sequences = self.sequences, None
        try:
            other = super().clone(device)
        finally:
            self.sequences = sequences
            for cache in self.get_kv_caches():
                if cache is not None:
                    cache.sequences = sequences
        return other
