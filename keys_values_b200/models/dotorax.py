"""Reader of Dotorax checkpoints: ``config.json`` → :class:`Config`, tensor names → state dict of
:class:`keys_values_b200.models.layered.LayeredGPT`.

The design: sequential layers with RMS norms (weights stored around zero) before and after each sublayer and a factor on what a sublayer adds;
what a sublayer reads passes a short causal convolution; a learned vector per position at the input. Mixers are attention with a gate per
head (its keys and values possibly those of an earlier layer), gated linear attention, and a window with pooled blocks (interleaved rotation,
norms without weights, a temperature per head) side by side with a gated recurrence; feed-forwards are clamped gated units.
"""
from __future__ import annotations

from typing import Any, Dict, Mapping, Optional, Sequence

import torch

from keys_values_b200.config import Config

# rank of the decays' projection where there are no weights to tell it
DEFAULT_RANK = 16


def _attention(m: Dict[str, Any]) -> Dict[str, Any]:
    spec = dict(kind="grouped_attention", n_head=m["heads"], n_kv_head=m["kv_heads"], dim=m["dim"], v_dim=m["vdim"], scale=float(m["scale"]), rope_dims=0)
    rot = m.get("rot")
    if rot and rot.get("dims"):
        spec.update(rope_base=float(rot["base"]), rope_dims=rot["dims"])
    return spec


def _mixer(i: int, layer: Dict[str, Any], shapes: Mapping[str, Sequence[int]]) -> Dict[str, Any]:
    m, kind = layer["mixer"], layer["type"]
    if kind == "attention":
        spec = dict(_attention(m), gate="head")
        if m.get("kv_from") is not None:
            spec["kv_from"] = m["kv_from"]
        return spec
    if kind == "gla":
        low = shapes.get(f"l{i}.mix.a1")
        return dict(kind="gated_linear_attention", n_head=m["heads"], dim=m["dim"], v_dim=m["vdim"], tau=float(m["tau"]), rank=low[0] if low else DEFAULT_RANK)
    if kind == "parallel":
        a, r = m["left"], m["right"]
        left = dict(_attention(a), rope_interleaved=True, qk_norm="unit", temperature=True, window=a["mask"]["size"], pool=a["mask"]["pool"])
        right = dict(kind="gated_recurrence", width=r["width"], blocks=r["blocks"], conv=r["conv"])
        return dict(kind="side_by_side", left=left, left_scale=float(m["left_scale"]), right=right, right_scale=float(m["right_scale"]))
    raise ValueError(f"mixer {kind!r} is not part of the design")


def _feed_forward(layer: Dict[str, Any]) -> Optional[Dict[str, Any]]:
    f = layer.get("mlp")
    if f is None:
        return None
    if f["kind"] != "dense":
        raise ValueError(f"feed-forward {f['kind']!r} is not part of the design")
    return dict(kind="gated", ff=f["ff"], limit=float(f["limit"]))


def config_from_json(content: Dict[str, Any], shapes: Mapping[str, Sequence[int]]) -> Config:
    layers = [dict(mixer=_mixer(i, x, shapes), mlp=_feed_forward(x)) for i, x in enumerate(content["layers"])]
    first = next((x["mixer"] for x in layers if x["mixer"]["kind"] == "grouped_attention"), None)
    return Config(
        name=content.get("name", "Dotorax"), architecture="Dotorax", block_size=content["max_positions"], n_layer=len(layers), n_embd=content["width"],
        vocab_size=content["vocab"], padded_vocab_size=content["vocab"], n_head=1 if first is None else first["n_head"],
        n_query_groups=1 if first is None else first["n_kv_head"], head_size=content["width"] if first is None else first["dim"],
        norm_class_name="StreamOffsetRMSNorm", norm_eps=float(content["norm"]["eps"]), parallel_residual=False, post_attention_norm=True,
        post_mlp_norm=True, bias=False, input_conv=content["canon"]["taps"], residual_mult=float(content["residual_mult"]), position_table=True,
        layers=layers,
    )


def state_dict(tensors: Mapping[str, torch.Tensor], config: Config) -> Dict[str, torch.Tensor]:
    """Tensors under the design's names to the names of the model. Every tensor must be used."""
    left = dict(tensors)

    def take(name: str) -> torch.Tensor:
        if name not in left:
            raise KeyError(f"tensor {name!r} is missing")
        return left.pop(name)

    def join(prefix: str, *names: str) -> torch.Tensor:
        return torch.cat([take(prefix + n) for n in names])

    out = {"transformer.wte.weight": take("embed"), "positions.weight": take("pos"), "transformer.ln_f.weight": take("final.norm"),
           "lm_head.weight": take("head")}
    for i, layer in enumerate(config.layers):
        src, dst, m = f"l{i}.", f"transformer.h.{i}.", layer["mixer"]
        mix, attn = src + "mix.", dst + "attn."
        out[dst + "norm_1.weight"], out[dst + "post_attention_norm.weight"] = take(src + "norm1"), take(src + "norm1b")
        out[dst + "conv_1"] = take(src + "canon1")
        if m["kind"] == "grouped_attention":
            out[attn + "qkv.weight"] = join(mix, "q", "g") if m.get("kv_from") is not None else join(mix, "q", "k", "v", "g")
            out[attn + "proj.weight"] = take(mix + "o")
        elif m["kind"] == "gated_linear_attention":
            out[attn + "proj_in.weight"] = join(mix, "q", "k", "a1", "v", "g")
            for name, to in {"a2": "decay", "a2.b": "decay_bias", "norm": "norm", "o": "proj.weight"}.items():
                out[attn + to] = take(mix + name)
        else:
            out[attn + "left.qkv.weight"] = join(mix + "left.", "q", "k", "v")
            out[attn + "left.temperature"], out[attn + "left.proj.weight"] = take(mix + "left.temp"), take(mix + "left.o")
            out[attn + "right.proj_in.weight"], out[attn + "right.proj_in.bias"] = join(mix + "right.", "y", "x"), join(mix + "right.", "y.b", "x.b")
            names = {"conv": "conv", "conv.b": "conv_bias", "ra": "gate_r", "ra.b": "gate_r_bias", "ri": "gate_i", "ri.b": "gate_i_bias", "lam": "lam",
                     "o": "proj.weight"}
            for name, to in names.items():
                out[f"{attn}right.{to}"] = take(f"{mix}right.{name}")
        if layer["mlp"] is None:
            for name in ("norm2", "norm2b", "canon2"):
                left.pop(src + name, None)  # nothing to norm
            continue
        out[dst + "norm_2.weight"], out[dst + "post_mlp_norm.weight"] = take(src + "norm2"), take(src + "norm2b")
        out[dst + "conv_2"] = take(src + "canon2")
        out[dst + "mlp.up.weight"], out[dst + "mlp.down.weight"] = join(src + "mlp.", "gate", "up"), take(src + "mlp.down")
    if left:
        raise KeyError(f"tensors without a place in the model: {sorted(left)[:5]}")
    return out
