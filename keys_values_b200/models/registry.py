"""Model classes and checkpoint readers by architecture.

A LitGPT-shaped checkpoint (``lit_model.pth`` + ``model_config.yaml``) is a :class:`GPT`. Other architectures register a
reader here; their checkpoint directories hold ``config.json`` (with an ``"architecture"`` entry) and ``model.safetensors``
under the architecture's own tensor names.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable, Dict, Mapping, Optional, Sequence, Union

import torch

from keys_values_b200.config import Config


@dataclass(frozen=True)
class Architecture:
    name: str
    # content of config.json and shapes of the checkpoint's tensors by name (some sizes may stand there only)
    config_from_json: Callable[[Dict[str, Any], Mapping[str, Sequence[int]]], Config]
    # the architecture's tensors (by name) -> state dict of the model class
    state_dict: Callable[[Mapping[str, torch.Tensor], Config], Dict[str, torch.Tensor]]


def _from_content(reader: Callable[[Dict[str, Any]], Config]):
    """Reader of a design whose configuration gives every size."""
    return lambda content, shapes: reader(content)


def _architectures() -> Dict[str, Architecture]:
    from keys_values_b200.models import dotorax, ladadra, mezilix, pazenex

    known = (
        Architecture("Dotorax", dotorax.config_from_json, dotorax.state_dict),
        Architecture("Ladadra", _from_content(ladadra.config_from_json), ladadra.state_dict),
        Architecture("Mezilix", _from_content(mezilix.config_from_json), mezilix.state_dict),
        Architecture("Pazenex", _from_content(pazenex.config_from_json), pazenex.state_dict),
    )
    return {a.name: a for a in known}


def architecture_names():
    return sorted(_architectures())


def get_architecture(name: str) -> Architecture:
    known = _architectures()
    if name not in known:
        raise ValueError(f"architecture {name!r} is not registered; known: {sorted(known)}")
    return known[name]


def config_from_directory(path: Union[str, Path], **kwargs: Any) -> Optional[Config]:
    """Config of a checkpoint directory with a registered architecture's ``config.json``, else ``None``."""
    file = Path(path) / "config.json"
    if not file.is_file():
        return None
    content = json.loads(file.read_text(encoding="utf-8"))
    if not isinstance(content, dict) or "architecture" not in content:
        return None
    config = get_architecture(content["architecture"]).config_from_json(content, tensor_shapes(path))
    for k, v in kwargs.items():
        setattr(config, k, v)
    return config


def model_class(config: Config):
    from keys_values_b200.models.layered import LayeredGPT
    from keys_values_b200.models.model import GPT

    return GPT if config.layers is None else LayeredGPT


def create_model(config: Config, **mha_kwargs):
    """The model of ``config``, with whatever class its description needs."""
    return model_class(config)(config, **mha_kwargs)


def default_cache_name(config: Config, name: Optional[str] = None) -> str:
    """``name``, or for models with described layers the caches that fit them."""
    if config.layers is None:
        return name or "h2o-default"
    fits = "latent-default" if all(x["mixer"]["kind"] == "latent_attention" for x in config.layers) else "layered-default"
    return name if name in ("layered-default", fits) else fits


def tensor_shapes(checkpoint_dir: Union[str, Path]) -> Dict[str, Sequence[int]]:
    """Shapes of a directory's ``*.safetensors`` by tensor name, from the files' headers."""
    shapes: Dict[str, Sequence[int]] = {}
    for file in sorted(Path(checkpoint_dir).glob("*.safetensors")):
        with open(file, "rb") as f:
            header = json.loads(f.read(int.from_bytes(f.read(8), "little")))
        shapes.update({name: tuple(x["shape"]) for name, x in header.items() if name != "__metadata__"})
    return shapes


def read_safetensors(path: Path) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file

    return load_file(str(path))


def load_architecture_weights(model, checkpoint_dir: Union[str, Path]) -> bool:
    """Weights of a registered architecture's ``*.safetensors`` into ``model``; ``False`` if the directory is not one."""
    checkpoint_dir = Path(checkpoint_dir)
    files = sorted(checkpoint_dir.glob("*.safetensors"))
    if not model.config.architecture or not files:
        return False
    tensors: Dict[str, torch.Tensor] = {}
    for f in files:
        tensors.update(read_safetensors(f))
    model.load_state_dict(get_architecture(model.config.architecture).state_dict(tensors, model.config), strict=True)
    return True
