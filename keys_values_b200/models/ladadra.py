"""Reader of Ladadra checkpoints: ``config.json`` → :class:`Config`, tensor names → state dict of
:class:`keys_values_b200.models.layered.LayeredGPT`.

The design: sequential layers whose sublayers read the stream itself and have an RMS norm on their output; mixers are retention,
chunked attention (biases, norms over the whole projections, banded rotation, soft cap, learned sink, one gate per head) and
differential attention over a window with kept first tokens (norms per head, no rotation); feed-forwards are gated with silu, dense or
routed (sigmoid scores, corrected choice out of the best groups, weights that sum to one, a shared expert). The output head is the
embedding table.
"""
from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

import torch

from keys_values_b200.config import Config

# the design itself bounds no context: angles are computed per position
BLOCK_SIZE = 1 << 20


def _rotation(rot: Optional[Dict[str, Any]]) -> Dict[str, Any]:
    if not rot or not rot.get("dims"):
        return dict(rope_dims=0)
    out: Dict[str, Any] = dict(rope_base=float(rot["base"]), rope_dims=rot["dims"])
    bands = rot.get("scaling")
    if bands:
        out["rope_bands"] = {k: float(bands[k]) for k in ("factor", "low", "high", "original")}
    return out


def _mixer(layer: Dict[str, Any]) -> Dict[str, Any]:
    m, kind = layer["mixer"], layer["type"]
    mask = m.get("mask") or {}
    if kind == "retention":
        return dict(kind="retention", n_head=m["heads"], dim=m["dim"], v_dim=m["vdim"], decay=[float(d) for d in m["decay"]], **_rotation(m.get("rot")))
    if kind not in ("attention", "attention_2"):
        raise ValueError(f"mixer {kind!r} is not part of the design")
    spec = dict(kind="grouped_attention", n_head=m["heads"], n_kv_head=m["kv_heads"], dim=m["dim"], v_dim=m["vdim"], scale=float(m["scale"]))
    if kind == "attention":
        return dict(spec, **_rotation(m.get("rot")), qkv_bias=True, qk_norm=True, softcap=float(m.get("softcap") or 0.0), chunk=mask.get("size"),
                    sink="learned", gate="head")
    return dict(spec, qk_norm="head", window=mask.get("size"), keep_first=mask.get("keep_first"), differential=float(m["diff"]))


def _feed_forward(layer: Dict[str, Any]) -> Optional[Dict[str, Any]]:
    f = layer.get("mlp")
    if f is None:
        return None
    if f["kind"] == "dense":
        return dict(kind="gated", ff=f["ff"])
    if f["kind"] != "moe":
        raise ValueError(f"feed-forward {f['kind']!r} is not part of the design")
    r, groups = f["router"], f["router"].get("groups")
    return dict(kind="routed", n_expert=r["experts"], top=r["top"], ff=f["expert"]["ff"], activation="silu_gated", score="sigmoid",
                correction=True, renormalize=True, renormalize_eps=1e-20,
                groups=None if not groups else dict(count=groups["count"], keep=groups["keep"]),
                shared=f["shared"]["ff"] if f.get("shared") else None)


def config_from_json(content: Dict[str, Any]) -> Config:
    layers = [dict(mixer=_mixer(x), mlp=_feed_forward(x)) for x in content["layers"]]
    first = next((x["mixer"] for x in layers if x["mixer"]["kind"] == "grouped_attention"), None)
    return Config(
        name=content.get("name", "Ladadra"), architecture="Ladadra", block_size=BLOCK_SIZE, n_layer=len(layers), n_embd=content["width"],
        vocab_size=content["vocab"], padded_vocab_size=content["vocab"], n_head=1 if first is None else first["n_head"],
        n_query_groups=1 if first is None else first["n_kv_head"], head_size=content["width"] if first is None else first["dim"],
        norm_class_name="StreamRMSNorm", norm_eps=float(content["norm"]["eps"]), parallel_residual=False, norm_1=False, norm_2=False,
        post_attention_norm=True, post_mlp_norm=True, bias=False, tie_embeddings=True, layers=layers,
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

    embed = take("embed")
    out = {"transformer.wte.weight": embed, "lm_head.weight": embed, "transformer.ln_f.weight": take("final.norm")}
    for i, layer in enumerate(config.layers):
        src, dst, m, mlp = f"l{i}.", f"transformer.h.{i}.", layer["mixer"], layer["mlp"]
        mix, attn = src + "mix.", dst + "attn."
        out[dst + "post_attention_norm.weight"] = take(src + "norm1")
        out[attn + "proj.weight"] = take(mix + "o")
        if m["kind"] == "retention":
            out[attn + "qkvg.weight"] = join(mix, "q", "k", "v", "g")
        else:
            out[attn + "norm_q"], out[attn + "norm_k"] = take(mix + "q.norm"), take(mix + "k.norm")
            if m.get("differential") is not None:
                out[attn + "qkv.weight"] = join(mix, "q", "k", "v")
                out[attn + "map_weights"] = torch.stack([take(mix + n) for n in ("lq1", "lk1", "lq2", "lk2")])
            else:
                out[attn + "qkv.weight"] = join(mix, "q", "k", "v", "g")
                out[attn + "qkv_bias"] = join(mix, "q.b", "k.b", "v.b")
                out[attn + "sink"] = take(mix + "sink")
        if mlp is None:
            left.pop(src + "norm2", None)  # nothing to norm
            continue
        out[dst + "post_mlp_norm.weight"] = take(src + "norm2")
        if mlp["kind"] == "gated":
            out[dst + "mlp.up.weight"], out[dst + "mlp.down.weight"] = join(src + "mlp.", "gate", "up"), take(src + "mlp.down")
            continue
        experts = [f"{src}mlp.e{e}." for e in range(mlp["n_expert"])]
        out[dst + "mlp.gate.weight"], out[dst + "mlp.correction"] = take(src + "mlp.router"), take(src + "mlp.correction")
        out[dst + "mlp.up"] = torch.stack([join(e, "gate", "up") for e in experts])
        out[dst + "mlp.down"] = torch.stack([take(e + "down") for e in experts])
        if mlp.get("shared"):
            out[dst + "mlp.shared.up.weight"] = join(src + "mlp.shared.", "gate", "up")
            out[dst + "mlp.shared.down.weight"] = take(src + "mlp.shared.down")
    if left:
        raise KeyError(f"tensors without a place in the model: {sorted(left)[:5]}")
    return out
