"""Reader of Mezilix checkpoints: ``config.json`` → :class:`Config`, tensor names → state dict of
:class:`keys_values_b200.models.layered.LayeredGPT`.

The design: token and bigram embedding; parallel layers under one scalar-gain RMS norm, whose mixer (sliding-window latent
attention) reads a token-shifted input and whose feed-forward is a mixture of ungated squared-relu experts chosen by a softmax
router (weights not renormalised); a learned average over the embedding output and all layers' results goes on to the
next layer.
"""
from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

import torch

from keys_values_b200.config import Config

# the design itself bounds no context: angles are computed per position
BLOCK_SIZE = 1 << 20


def _mixer(layer: Dict[str, Any]) -> Dict[str, Any]:
    if layer["type"] != "latent_attention":
        raise ValueError(f"mixer {layer['type']!r} is not part of the design")
    m = layer["mixer"]
    rot = m["rot"]
    return dict(
        kind="latent_attention", n_head=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], kv_rank=m["kv_rank"],
        scale=float(m["scale"]), window=m["mask"]["size"] if m.get("mask") else None, rope_base=float(rot["base"]),
        rope_dims=rot.get("dims", m["rot_dim"]),
    )


def _feed_forward(layer: Dict[str, Any]) -> Optional[Dict[str, Any]]:
    f = layer.get("mlp")
    if f is None:
        return None
    if f["kind"] != "moe":
        raise ValueError(f"feed-forward {f['kind']!r} is not part of the design")
    return dict(kind="routed", n_expert=f["router"]["experts"], top=f["router"]["top"], ff=f["expert"]["ff"],
                activation="relu_squared", renormalize=False)


def config_from_json(content: Dict[str, Any]) -> Config:
    layers = [dict(mixer=_mixer(x), mlp=_feed_forward(x)) for x in content["layers"]]
    first = layers[0]["mixer"]
    bigram = content.get("embedding", {}).get("bigram")
    return Config(
        name=content.get("name", "Mezilix"), architecture="Mezilix", block_size=BLOCK_SIZE, n_layer=len(layers), n_embd=content["width"],
        vocab_size=content["vocab"], padded_vocab_size=content["vocab"], n_head=first["n_head"], head_size=first["dim"] + first["rot_dim"],
        norm_class_name="ScalarRMSNorm", norm_eps=float(content["norm"]["eps"]), shared_attention_norm=True, bias=False,
        layers=layers, bigram=None if bigram is None else {k: int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")},
        token_shift=True, depth_average=True,
    )


def state_dict(tensors: Mapping[str, torch.Tensor], config: Config) -> Dict[str, torch.Tensor]:
    """Tensors under the design's names to the names of the model. Every tensor must be used."""
    left = dict(tensors)

    def take(name: str) -> torch.Tensor:
        if name not in left:
            raise KeyError(f"tensor {name!r} is missing")
        return left.pop(name)

    out = {
        "transformer.wte.weight": take("embed"),
        "transformer.ln_f.weight": take("final.norm").reshape(()),
        "lm_head.weight": take("head"),
    }
    if config.bigram is not None:
        out["bigram.weight"] = take("bigram")
    for i, layer in enumerate(config.layers):
        src, dst = f"l{i}.", f"transformer.h.{i}."
        out[dst + "norm_1.weight"] = take(src + "norm1").reshape(())
        out[dst + "shift"] = take(src + "shift")
        out[dst + "depth"] = take(src + "dwa")
        out[dst + "attn.qkv.weight"] = torch.cat((take(src + "mix.q"), take(src + "mix.dkv")))
        out[dst + "attn.norm_kv"] = take(src + "mix.dkv.norm")
        out[dst + "attn.key.weight"] = take(src + "mix.uk")
        out[dst + "attn.value.weight"] = take(src + "mix.uv")
        out[dst + "attn.proj.weight"] = take(src + "mix.o")
        mlp = layer["mlp"]
        if mlp is not None:
            out[dst + "mlp.gate.weight"] = take(src + "mlp.router")
            for name in ("up", "down"):
                out[f"{dst}mlp.{name}"] = torch.stack([take(f"{src}mlp.e{e}.{name}") for e in range(mlp["n_expert"])])
    if left:
        raise KeyError(f"tensors without a place in the model: {sorted(left)[:5]}")
    return out
