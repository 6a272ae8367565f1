"""Model configuration.

A self-contained dataclass that uses the LitGPT field names, so that a
``model_config.yaml`` written next to a ``lit_model.pth`` loads unchanged
(parity: ``keys_values/config.py:23-43`` and the LitGPT ``Config`` it extends;
field list as in ``keys_values/scripts/convert_lora_to_litgpt/model_config.yaml``).
A small registry of named architectures replaces LitGPT's ``name_to_config``.
"""
from __future__ import annotations

import copy
from dataclasses import asdict, dataclass, field, fields
from pathlib import Path
from typing import Any, Dict, List, Optional, Tuple, Type, Union

import yaml


# norms of an fp32 residual stream by their names in `norm_class_name`: the mean taken off or not, weights stored around one or zero
STREAM_NORMS = {
    "StreamLayerNorm": dict(center=True),
    "StreamRMSNorm": dict(center=False),
    "StreamOffsetRMSNorm": dict(center=False, unit_offset=True),
}


def find_multiple(n: int, k: int) -> int:
    """Smallest multiple of ``k`` that is ``>= n``."""
    if n % k == 0:
        return n
    return n + k - (n % k)


@dataclass
class Config:
    name: str = ""
    hf_config: dict = field(default_factory=dict)
    # General size parameters
    block_size: int = 4096
    n_layer: int = 16
    n_embd: int = 4096
    vocab_size: int = 50254
    padding_multiple: int = 512
    padded_vocab_size: Optional[int] = None
    # Transformer block (structure, normalizations)
    norm_class_name: str = "LayerNorm"
    norm_eps: float = 1e-5
    norm_qk: bool = False
    norm_qk_type: str = "default"
    post_attention_norm: bool = False
    post_mlp_norm: bool = False
    parallel_residual: bool = True
    shared_attention_norm: bool = False
    norm_1: bool = True
    norm_2: bool = True
    # Transformer block (self-attention)
    n_head: int = 32
    head_size: Optional[int] = None
    n_query_groups: Optional[int] = None
    attn_bias: bool = False
    attention_scores_scalar: Optional[int] = None
    sliding_window_size: Optional[int] = None
    sliding_window_indices: Optional[List[int]] = None
    attention_logit_softcapping: Optional[float] = None
    latent_attention: Optional[dict] = None
    # Rotary position embedding
    rope_base: int = 10000
    rotary_percentage: float = 0.25
    rope_condense_ratio: int = 1
    rope_adjustments: Optional[dict] = None
    rope_local_base_freq: Optional[float] = None
    rope_indices: Optional[List[int]] = None
    # Transformer block (MLP)
    intermediate_size: Optional[int] = None
    moe_intermediate_size: Optional[int] = None
    bias: bool = True
    mlp_class_name: str = "GptNeoxMLP"
    gelu_approximate: str = "none"
    n_expert: int = 0
    n_shared_expert: Optional[int] = None
    n_expert_groups: Optional[int] = None
    n_topk_groups: Optional[int] = None
    n_topk_scores_per_group: Optional[int] = None
    n_expert_per_token: int = 0
    first_k_dense_replace: Optional[int] = None
    routed_scaling_factor: float = 1.0
    norm_topk_prob: bool = False
    # GPT before/after blocks
    scale_embeddings: bool = False
    lm_head_bias: bool = False
    final_logit_softcapping: Optional[float] = None
    # Models described layer by layer (models/layered.py). Each entry: {"mixer": {"kind": ..., sizes and constants},
    # "mlp": None or {"kind": ..., sizes}}; the kinds and their entries are those of the mixer and feed-forward classes there.
    # With parallel_residual mixer and feed-forward read one norm's output; without, each has a norm before it (norm_1 / norm_2) and, with
    # post_attention_norm / post_mlp_norm, one after it.
    layers: Optional[List[dict]] = None
    # {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row with the same weights. Before each
    # pass but the first the embedding output is added to the stream ("add_embedding"), before each pass a learned vector
    # ("step_vectors").
    loop: Optional[dict] = None
    bigram: Optional[dict] = None  # {"buckets", "mul_prev", "mul_cur"}: hashed embedding of (previous token, token)
    token_shift: bool = False  # the mixer reads a learned blend of this and the previous token's normed input
    depth_average: bool = False  # learned average over the embedding output and all layers' results
    tie_embeddings: bool = False  # described layers: the output head is the embedding table
    # Sequential layers: what a sublayer reads, h, becomes h + a causal convolution over time of h, this many taps (0: none)
    input_conv: int = 0
    residual_mult: float = 1.0  # sequential layers: factor of what a sublayer adds to the stream
    position_table: bool = False  # described layers: a learned vector per position (block_size of them) is added to the embedding
    architecture: str = ""  # entry of models/registry.py the config was read by
    # Added by keys_values (config.py:26-30): use the in-repo RMSNorm
    own_rms_norm_implementation: bool = True

    def __post_init__(self):
        if not self.name:
            self.name = self.hf_config.get("name", self.name)
        if self.head_size is None:
            assert self.n_embd % self.n_head == 0
            self.head_size = self.n_embd // self.n_head
        if self.padded_vocab_size is None:
            self.padded_vocab_size = find_multiple(self.vocab_size, self.padding_multiple)
        else:
            self.vocab_size = min(self.vocab_size, self.padded_vocab_size)
        if self.n_query_groups is not None:
            assert self.n_head % self.n_query_groups == 0
        else:
            self.n_query_groups = self.n_head
        if self.intermediate_size is None:
            if self.mlp_class_name == "LLaMAMLP":
                raise ValueError(f"The config {self.name!r} needs to set `intermediate_size`")
            self.intermediate_size = 4 * self.n_embd
        self.rope_n_elem = int(self.rotary_percentage * self.head_size)
        if self.sliding_window_size is not None and self.sliding_window_indices is None:
            self.sliding_window_indices = [1] * self.n_layer
        if self.rope_local_base_freq is not None and self.rope_indices is None:
            self.rope_indices = [1] * self.n_layer
        if self.loop is not None and not (0 <= self.loop["start"] < self.loop["stop"] <= self.n_layer and self.loop["times"] >= 1):
            raise ValueError(f"loop = {self.loop} must cover some of {self.n_layer} layers at least once")

    # ------------------------------------------------------- described layers
    def layer_runs(self) -> List[Tuple[int, int]]:
        """Layer and turn (0, 1, … within the loop) of every layer run of a pass, in order."""
        if self.loop is None:
            return [(i, 0) for i in range(self.n_layer)]
        a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
        inside = [(i, t) for t in range(n) for i in range(a, b)]
        return [(i, 0) for i in range(a)] + inside + [(i, 0) for i in range(b, self.n_layer)]

    def layer_turns(self, block_idx: int) -> int:
        """How often layer ``block_idx`` runs in a pass."""
        looped = self.loop is not None and self.loop["start"] <= block_idx < self.loop["stop"]
        return self.loop["times"] if looped else 1

    # ----------------------------------------------------------- construction
    @classmethod
    def from_name(cls, name: str, **kwargs: Any) -> "Config":
        if name not in name_to_config:
            raise ValueError(f"{name!r} is not a supported config name; known: {sorted(name_to_config)}")
        conf = copy.deepcopy(name_to_config[name])
        conf.update(kwargs)
        return cls(**conf)

    @classmethod
    def from_file(cls, path: Union[str, Path], **kwargs: Any) -> "Config":
        with open(path, encoding="utf-8") as fp:
            file_kwargs = yaml.safe_load(fp)
            if file_kwargs is None:
                raise ValueError(f"{path} is empty which is likely unexpected.")
        file_kwargs.update(kwargs)
        known = {f.name for f in fields(cls)}
        file_kwargs = {k: v for k, v in file_kwargs.items() if k in known}
        return cls(**file_kwargs)

    @classmethod
    def from_checkpoint(cls, path: Union[str, Path], **kwargs: Any) -> "Config":
        """``path`` is a checkpoint directory holding ``model_config.yaml``, or the ``config.json`` of a registered
        architecture (``models/registry.py``)."""
        path = Path(path)
        if (config_path := path / "model_config.yaml").is_file():
            return cls.from_file(config_path, **kwargs)
        from keys_values_b200.models.registry import config_from_directory

        if (config := config_from_directory(path, **kwargs)) is not None:
            return config
        if (model_name := path.name) in name_to_config:
            return cls.from_name(model_name, **kwargs)
        raise FileNotFoundError(f"For {str(path)!r} neither 'model_config.yaml' nor matching config exists.")

    def to_dict(self) -> Dict[str, Any]:
        d = asdict(self)
        return d

    def save(self, path: Union[str, Path]) -> None:
        with open(path, "w", encoding="utf-8") as fp:
            yaml.safe_dump(self.to_dict(), fp)

    # ------------------------------------------------------------- factories
    @property
    def mlp_class(self) -> Type:
        from keys_values_b200.models import model as _m

        return getattr(_m, self.mlp_class_name)

    @property
    def norm_class(self) -> Type:
        """Normalization layer constructor (parity: ``keys_values/config.py:32-43``).

        ``RMSNorm`` maps to the in-repo implementation (Gemma configs get
        ``add_unit_offset=True``); any other name is taken from ``torch.nn``.
        """
        from functools import partial

        import torch

        from keys_values_b200.models.model import RMSNorm

        if self.norm_class_name == "ScalarRMSNorm":
            from keys_values_b200.models.layered import ScalarRMSNorm

            return ScalarRMSNorm
        if self.norm_class_name in STREAM_NORMS:
            from keys_values_b200.models.layered import StreamNorm

            return partial(StreamNorm, **STREAM_NORMS[self.norm_class_name])
        if self.norm_class_name == "RMSNorm":
            return partial(RMSNorm, add_unit_offset="Gemma" in self.name)
        if self.norm_class_name == "LayerNorm" and "OLMo" in self.name:
            return partial(torch.nn.LayerNorm, elementwise_affine=False)
        return getattr(torch.nn, self.norm_class_name)


# --------------------------------------------------------------------------
# Registry of named architectures. Only architecture hyper-parameters live here:
# weights come from a ``lit_model.pth`` or from random initialisation.
# --------------------------------------------------------------------------
def _layered(n_layer: int, mixer: dict, mlp: Optional[dict]) -> dict:
    """Fields of a model of ``n_layer`` equal latent-attention layers with routed experts."""
    mixer = dict(kind="latent_attention", **mixer)
    mixer.setdefault("scale", (mixer["dim"] + mixer["rot_dim"]) ** -0.5)
    mlp = None if mlp is None else dict(kind="routed", **mlp)
    return dict(
        n_layer=n_layer, n_head=mixer["n_head"], head_size=mixer["dim"] + mixer["rot_dim"], layers=[dict(mixer=mixer, mlp=mlp)] * n_layer,
        norm_class_name="ScalarRMSNorm", shared_attention_norm=True, bias=False, architecture="Mezilix",
        token_shift=True, depth_average=True,
    )


def _pazenex(width: int, layers: List[dict], **kwargs: Any) -> dict:
    """Fields of a model of sequential layers; ``layers`` as in ``Config.layers``."""
    first = next(x["mixer"] for x in layers if x["mixer"]["kind"] == "grouped_attention")
    return dict(
        n_embd=width, n_layer=len(layers), layers=layers, n_head=first["n_head"], n_query_groups=first["n_kv_head"], head_size=first["dim"],
        norm_class_name="StreamLayerNorm", parallel_residual=False, post_attention_norm=True, post_mlp_norm=True, bias=False,
        architecture="Pazenex", **kwargs,
    )


def _mamba2(heads: int, vdim: int, state: int, groups: int, ff: int, norm_groups: int = 1, conv: int = 4) -> dict:
    return dict(mixer=dict(kind="mamba2", n_head=heads, v_dim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv),
                mlp=dict(kind="dense", ff=ff, activation="relu_squared"))


def _grouped(heads: int, kv_heads: int, dim: int, ff: int, rope_base: float = 500000.0, rope_scale: float = 1.0) -> dict:
    return dict(mixer=dict(kind="grouped_attention", n_head=heads, n_kv_head=kv_heads, dim=dim, v_dim=dim, scale=dim**-0.5, rope_base=rope_base,
                           rope_dims=dim, rope_scale=rope_scale, qk_norm=True, shared_value=True, sink=True, gate=True),
                mlp=dict(kind="dense", ff=ff, activation="relu_squared"))


def _ladadra(width: int, layers: List[dict], **kwargs: Any) -> dict:
    """Fields of a model of sequential layers with norms on the sublayers' outputs only; ``layers`` as in ``Config.layers``."""
    first = next(x["mixer"] for x in layers if x["mixer"]["kind"] == "grouped_attention")
    return dict(
        n_embd=width, n_layer=len(layers), layers=layers, n_head=first["n_head"], n_query_groups=first["n_kv_head"], head_size=first["dim"],
        norm_class_name="StreamRMSNorm", parallel_residual=False, norm_1=False, norm_2=False, post_attention_norm=True, post_mlp_norm=True,
        bias=False, tie_embeddings=True, architecture="Ladadra", **kwargs,
    )


def _retention(heads: int, dim: int, vdim: int, rope_base: float = 10000.0) -> dict:
    """Decays 1 − 2^−5, 1 − 2^−6, … over the heads, repeated after 1 − 2^−12."""
    return dict(kind="retention", n_head=heads, dim=dim, v_dim=vdim, rope_base=rope_base, rope_dims=dim,
                decay=[1.0 - 2.0 ** -(5 + i % 8) for i in range(heads)])


def _chunked(heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, rope_dims: int, softcap: float = 50.0, rope_base: float = 500000.0,
             bands: Optional[dict] = None) -> dict:
    return dict(kind="grouped_attention", n_head=heads, n_kv_head=kv_heads, dim=dim, v_dim=vdim, scale=dim**-0.5, rope_base=rope_base,
                rope_dims=rope_dims, rope_bands=bands or dict(factor=8.0, low=1.0, high=4.0, original=8192), qkv_bias=True, qk_norm=True,
                softcap=softcap, chunk=chunk, sink="learned", gate="head")


def _differential(heads: int, kv_heads: int, dim: int, vdim: int, window: int, keep_first: int, differential: float) -> dict:
    return dict(kind="grouped_attention", n_head=heads, n_kv_head=kv_heads, dim=dim, v_dim=vdim, scale=dim**-0.5, qk_norm="head",
                window=window, keep_first=keep_first, differential=differential)


def _gated(ff: int) -> dict:
    return dict(kind="gated", ff=ff)


def _grouped_experts(n_expert: int, top: int, ff: int, groups: int, keep: int, shared: int) -> dict:
    return dict(kind="routed", n_expert=n_expert, top=top, ff=ff, activation="silu_gated", score="sigmoid", correction=True, renormalize=True,
                renormalize_eps=1e-20, groups=dict(count=groups, keep=keep), shared=shared)


def _dotorax(width: int, layers: List[dict], **kwargs: Any) -> dict:
    """Fields of a model of sequential layers whose inputs pass a short convolution; ``layers`` as in ``Config.layers``."""
    first = next(x["mixer"] for x in layers if x["mixer"]["kind"] == "grouped_attention")
    return dict(
        n_embd=width, n_layer=len(layers), layers=layers, n_head=first["n_head"], n_query_groups=first["n_kv_head"], head_size=first["dim"],
        norm_class_name="StreamOffsetRMSNorm", parallel_residual=False, post_attention_norm=True, post_mlp_norm=True, bias=False,
        position_table=True, architecture="Dotorax", **kwargs,
    )


def _shared_runs(times: int, heads: int, kv_heads: int, dim: int, rope_dims: int, linear: dict, parallel: dict, ff: int, limit: float = 7.0) -> List[dict]:
    """``times`` runs of: attention, gated linear attention, attention over the first one's keys and values, two mixers side by side."""
    out = []
    for i in range(times):
        a = dict(kind="grouped_attention", n_head=heads, n_kv_head=kv_heads, dim=dim, v_dim=dim, scale=dim**-0.5, rope_base=500000.0, rope_dims=rope_dims,
                 gate="head")
        out += [a, linear, dict(a, kv_from=4 * i), parallel]
    return [dict(mixer=m, mlp=dict(kind="gated", ff=ff, limit=limit)) for m in out]


def _gated_linear(heads: int, dim: int, vdim: int, rank: int = 16, tau: float = 16.0) -> dict:
    return dict(kind="gated_linear_attention", n_head=heads, dim=dim, v_dim=vdim, rank=rank, tau=tau)


def _pooled_beside_recurrence(heads: int, kv_heads: int, dim: int, rope_dims: int, window: int, pool: int, width: int, blocks: int,
                              scales: Tuple[float, float] = (0.7, 1.0)) -> dict:
    left = dict(kind="grouped_attention", n_head=heads, n_kv_head=kv_heads, dim=dim, v_dim=dim, scale=dim**-0.5, rope_base=10000.0, rope_dims=rope_dims,
                rope_interleaved=True, qk_norm="unit", temperature=True, window=window, pool=pool)
    return dict(kind="side_by_side", left=left, left_scale=scales[0], right=dict(kind="gated_recurrence", width=width, blocks=blocks, conv=4),
                right_scale=scales[1])


_llama_like = dict(
    rotary_percentage=1.0,
    parallel_residual=False,
    bias=False,
    norm_class_name="RMSNorm",
    mlp_class_name="LLaMAMLP",
)

configs: List[dict] = [
    # Tiny test models
    dict(
        name="tiny-gpt",
        block_size=1024, vocab_size=512, padded_vocab_size=512, n_layer=2, n_embd=64,
        n_head=4, n_query_groups=2, head_size=16, intermediate_size=172,
        norm_eps=1e-5, rope_base=10000, **_llama_like,
    ),
    dict(
        name="tiny-qwen3",
        block_size=4096, vocab_size=1024, padded_vocab_size=1024, n_layer=2, n_embd=256,
        n_head=8, n_query_groups=2, head_size=128, intermediate_size=512, norm_qk=True,
        norm_eps=1e-6, rope_base=1000000, **_llama_like,
    ),
    dict(  # head size 64 (Llama-3.2-1B, Qwen2.5-0.5B shapes)
        name="tiny-llama-d64",
        block_size=4096, vocab_size=1024, padded_vocab_size=1024, n_layer=2, n_embd=256,
        n_head=4, n_query_groups=2, head_size=64, intermediate_size=512,
        norm_eps=1e-5, rope_base=500000, **_llama_like,
    ),
    dict(  # head size 256 with a window layer and capped scores (Gemma-2 2b / 9b shapes): forward kernels only
        name="tiny-gemma2-d256",
        block_size=4096, vocab_size=1024, padded_vocab_size=1024, n_layer=2, n_embd=256,
        n_head=4, n_query_groups=2, head_size=256, intermediate_size=512, norm_eps=1e-6,
        rotary_percentage=1.0, parallel_residual=False, bias=False, norm_class_name="RMSNorm",
        mlp_class_name="GemmaMLP", gelu_approximate="tanh", scale_embeddings=True,
        post_attention_norm=True, post_mlp_norm=True, sliding_window_size=96, sliding_window_indices=[1, 0],
        attention_logit_softcapping=4.0, final_logit_softcapping=30.0,
    ),
    dict(  # Gemma-2 style: every other layer with a sliding window, capped attention scores and logits
        name="tiny-gemma2",
        block_size=4096, vocab_size=1024, padded_vocab_size=1024, n_layer=2, n_embd=256,
        n_head=8, n_query_groups=2, head_size=128, intermediate_size=512, norm_eps=1e-6,
        rotary_percentage=1.0, parallel_residual=False, bias=False, norm_class_name="RMSNorm",
        mlp_class_name="GemmaMLP", gelu_approximate="tanh", scale_embeddings=True,
        post_attention_norm=True, post_mlp_norm=True, sliding_window_size=96, sliding_window_indices=[1, 0],
        attention_logit_softcapping=4.0, final_logit_softcapping=30.0,
    ),
    dict(
        name="pythia-14m",
        block_size=512, n_layer=6, n_embd=128, n_head=4, padding_multiple=128,
    ),
    # Mezilix: latent attention over a window, routed experts, token shift, depth average, bigram embedding
    dict(
        name="tiny-mezilix", block_size=1 << 20, vocab_size=320, padded_vocab_size=320, n_embd=192, norm_eps=1e-5,
        bigram=dict(buckets=211, mul_prev=37, mul_cur=5),
        **_layered(3, dict(n_head=6, dim=24, rot_dim=8, v_dim=40, kv_rank=72, window=48, rope_base=10000.0), dict(n_expert=10, top=3, ff=56)),
    ),
    dict(
        name="Mezilix-2k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, n_embd=2048, norm_eps=1e-5,
        bigram=dict(buckets=65521, mul_prev=8191, mul_cur=31),
        **_layered(16, dict(n_head=16, dim=128, rot_dim=64, v_dim=128, kv_rank=512, window=4096, rope_base=10000.0),
                   dict(n_expert=64, top=6, ff=1408)),
    ),
    dict(
        name="Mezilix-4k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, n_embd=4096, norm_eps=1e-5,
        bigram=dict(buckets=65521, mul_prev=8191, mul_cur=31),
        **_layered(16, dict(n_head=32, dim=128, rot_dim=64, v_dim=128, kv_rank=512, window=4096, rope_base=10000.0),
                   dict(n_expert=16, top=2, ff=6144)),
    ),
    # Pazenex: Mamba-2 and grouped-query attention layers between layer norms, a run of layers passed twice
    dict(
        name="tiny-pazenex", block_size=1 << 20, vocab_size=352, padded_vocab_size=352, norm_eps=1e-5,
        **_pazenex(160, [_mamba2(5, 32, 24, 5, 208), _grouped(10, 2, 16, 208, rope_scale=2.0), _mamba2(4, 40, 16, 2, 176, norm_groups=2)],
                   loop=dict(start=0, stop=2, times=3, add_embedding=True, step_vectors=True)),
    ),
    dict(
        name="Pazenex-2k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5,
        **_pazenex(2048, [_mamba2(64, 64, 128, 8, 8192, norm_groups=8), _grouped(16, 4, 128, 8192, rope_scale=4.0)] * 8),
    ),
    dict(
        name="Pazenex-4k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5,
        **_pazenex(4096, [_mamba2(128, 64, 128, 8, 16384, norm_groups=8), _grouped(32, 8, 128, 16384, rope_scale=4.0)] * 6),
    ),
    # Ladadra: retention, differential attention over a window and chunked attention, dense and routed gated feed-forwards, norms on
    # the sublayers' outputs only
    dict(
        name="tiny-ladadra", block_size=1 << 20, vocab_size=416, padded_vocab_size=416, norm_eps=1e-5,
        **_ladadra(144, [
            dict(mixer=_retention(3, 40, 24), mlp=_gated(200)),
            dict(mixer=_differential(4, 1, 24, 40, window=60, keep_first=12, differential=0.4), mlp=_grouped_experts(8, 3, 40, 4, 2, 56)),
            dict(mixer=_chunked(6, 3, 32, 24, chunk=90, rope_dims=16, bands=dict(factor=2.0, low=1.0, high=4.0, original=512)), mlp=None),
        ]),
    ),
    dict(
        name="Ladadra-2k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5,
        **_ladadra(2048, [
            dict(mixer=_retention(16, 128, 128), mlp=_gated(5632)),
            dict(mixer=_differential(16, 4, 64, 128, window=4096, keep_first=128, differential=0.5), mlp=_grouped_experts(64, 6, 704, 8, 4, 1408)),
            dict(mixer=_chunked(16, 4, 128, 128, chunk=16384, rope_dims=64), mlp=_gated(5632)),
            dict(mixer=_chunked(16, 4, 128, 128, chunk=16384, rope_dims=64), mlp=_grouped_experts(64, 6, 704, 8, 4, 1408)),
        ] * 4),
    ),
    dict(
        name="Ladadra-4k", block_size=1 << 20, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5,
        **_ladadra(4096, [
            dict(mixer=_retention(32, 128, 128), mlp=_gated(11008)),
            dict(mixer=_differential(32, 8, 64, 128, window=4096, keep_first=128, differential=0.5), mlp=_grouped_experts(32, 4, 2048, 4, 2, 2816)),
            dict(mixer=_chunked(32, 8, 128, 128, chunk=16384, rope_dims=64), mlp=_gated(11008)),
            dict(mixer=_chunked(32, 8, 128, 128, chunk=16384, rope_dims=64), mlp=_grouped_experts(32, 4, 2048, 4, 2, 2816)),
        ] * 3),
    ),
    # Dotorax: attention (half of it over another layer's keys and values), gated linear attention, a window with pooled blocks side by side
    # with a gated recurrence; short convolutions in front of the sublayers, a position table
    dict(
        name="tiny-dotorax", block_size=1024, vocab_size=288, padded_vocab_size=288, norm_eps=1e-5, input_conv=3, residual_mult=0.8,
        **_dotorax(112, _shared_runs(1, 6, 3, 24, 16, _gated_linear(3, 40, 24, rank=8),
                                     _pooled_beside_recurrence(4, 2, 24, 8, 48, 6, 120, 5), 152, limit=2.0)),
    ),
    dict(
        name="Dotorax-2k", block_size=1 << 15, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5, input_conv=4, residual_mult=0.9,
        **_dotorax(2048, _shared_runs(4, 16, 4, 128, 64, _gated_linear(16, 128, 128),
                                      _pooled_beside_recurrence(16, 4, 128, 64, 2048, 64, 2048, 16), 5632)),
    ),
    dict(
        name="Dotorax-4k", block_size=1 << 15, vocab_size=32000, padded_vocab_size=32000, norm_eps=1e-5, input_conv=4, residual_mult=0.9,
        **_dotorax(4096, _shared_runs(3, 32, 8, 128, 64, _gated_linear(32, 128, 128),
                                      _pooled_beside_recurrence(32, 8, 128, 64, 2048, 64, 4096, 16), 11008)),
    ),
    # Qwen 2.5
    dict(
        name="Qwen2.5-0.5B", hf_config=dict(org="Qwen", name="Qwen2.5-0.5B"),
        block_size=32768, vocab_size=151643, padded_vocab_size=151936, n_layer=24, n_head=14,
        n_embd=896, n_query_groups=2, attn_bias=True, intermediate_size=4864, norm_eps=1e-6,
        rope_base=1000000, **_llama_like,
    ),
    dict(
        name="Qwen2.5-1.5B", hf_config=dict(org="Qwen", name="Qwen2.5-1.5B"),
        block_size=131072, vocab_size=151643, padded_vocab_size=151936, n_layer=28, n_head=12,
        n_embd=1536, n_query_groups=2, attn_bias=True, intermediate_size=8960, norm_eps=1e-6,
        rope_base=1000000, **_llama_like,
    ),
    dict(
        name="Qwen2.5-7B", hf_config=dict(org="Qwen", name="Qwen2.5-7B"),
        block_size=131072, vocab_size=151643, padded_vocab_size=152064, n_layer=28, n_head=28,
        n_embd=3584, n_query_groups=4, attn_bias=True, intermediate_size=18944, norm_eps=1e-6,
        rope_base=1000000, **_llama_like,
    ),
    # Qwen 3
    dict(
        name="Qwen3-0.6B", hf_config=dict(org="Qwen", name="Qwen3-0.6B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=28, n_head=16,
        n_embd=1024, n_query_groups=8, head_size=128, intermediate_size=3072, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-1.7B", hf_config=dict(org="Qwen", name="Qwen3-1.7B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=28, n_head=16,
        n_embd=2048, n_query_groups=8, head_size=128, intermediate_size=6144, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-4B", hf_config=dict(org="Qwen", name="Qwen3-4B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=36, n_head=32,
        n_embd=2560, n_query_groups=8, head_size=128, intermediate_size=9728, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-4B-Instruct-2507", hf_config=dict(org="Qwen", name="Qwen3-4B-Instruct-2507"),
        block_size=262144, vocab_size=151643, padded_vocab_size=151936, n_layer=36, n_head=32,
        n_embd=2560, n_query_groups=8, head_size=128, intermediate_size=9728, norm_eps=1e-6,
        rope_base=5000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-8B", hf_config=dict(org="Qwen", name="Qwen3-8B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=36, n_head=32,
        n_embd=4096, n_query_groups=8, head_size=128, intermediate_size=12288, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-14B", hf_config=dict(org="Qwen", name="Qwen3-14B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=40, n_head=40,
        n_embd=5120, n_query_groups=8, head_size=128, intermediate_size=17408, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    dict(
        name="Qwen3-32B", hf_config=dict(org="Qwen", name="Qwen3-32B"),
        block_size=40960, vocab_size=151643, padded_vocab_size=151936, n_layer=64, n_head=64,
        n_embd=5120, n_query_groups=8, head_size=128, intermediate_size=25600, norm_eps=1e-6,
        rope_base=1000000, norm_qk=True, **_llama_like,
    ),
    # Llama 3.x
    dict(
        name="Llama-3-8B", hf_config=dict(org="meta-llama", name="Meta-Llama-3-8B"),
        block_size=8192, vocab_size=128000, padded_vocab_size=128256, n_layer=32, n_head=32,
        n_embd=4096, n_query_groups=8, intermediate_size=14336, norm_eps=1e-5, rope_base=500000,
        **_llama_like,
    ),
    dict(
        name="Llama-3.1-8B", hf_config=dict(org="meta-llama", name="Meta-Llama-3.1-8B"),
        block_size=131072, vocab_size=128000, padded_vocab_size=128256, n_layer=32, n_head=32,
        n_embd=4096, n_query_groups=8, intermediate_size=14336, norm_eps=1e-5, rope_base=500000,
        rope_adjustments=dict(factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_seq_len=8192),
        **_llama_like,
    ),
    dict(
        name="Llama-3.2-1B", hf_config=dict(org="meta-llama", name="Llama-3.2-1B"),
        block_size=131072, vocab_size=128000, padded_vocab_size=128256, n_layer=16, n_head=32,
        n_embd=2048, n_query_groups=8, intermediate_size=8192, norm_eps=1e-5, rope_base=500000,
        rope_adjustments=dict(factor=32.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_seq_len=8192),
        **_llama_like,
    ),
    # Gemma 2 (softcapping, sliding window, post norms, GemmaMLP)
    dict(
        name="Gemma-2-2b", hf_config=dict(org="google", name="gemma-2-2b"),
        block_size=8192, vocab_size=256000, padded_vocab_size=256000, n_layer=26, n_head=8,
        n_embd=2304, n_query_groups=4, head_size=256, intermediate_size=9216, norm_eps=1e-6,
        rotary_percentage=1.0, parallel_residual=False, bias=False, norm_class_name="RMSNorm",
        mlp_class_name="GemmaMLP", gelu_approximate="tanh", scale_embeddings=True,
        post_attention_norm=True, post_mlp_norm=True, sliding_window_size=4096,
        sliding_window_indices=[1 if i % 2 == 0 else 0 for i in range(26)],
        attention_scores_scalar=256, attention_logit_softcapping=50.0, final_logit_softcapping=30.0,
    ),
    # Mistral-style with sliding window
    dict(
        name="Mistral-7B-v0.1", hf_config=dict(org="mistralai", name="Mistral-7B-v0.1"),
        block_size=4096, vocab_size=32000, padded_vocab_size=32000, n_layer=32, n_head=32, n_embd=4096,
        n_query_groups=8, intermediate_size=14336, norm_eps=1e-5, sliding_window_size=4096,
        **_llama_like,
    ),
    # Phi-like parallel residual with partial rotary and LayerNorm
    dict(
        name="phi-2", hf_config=dict(org="microsoft", name="phi-2"),
        block_size=2048, vocab_size=50257, padded_vocab_size=51200, n_layer=32, n_head=32, n_embd=2560,
        rotary_percentage=0.4, shared_attention_norm=True, lm_head_bias=True, gelu_approximate="tanh",
    ),
]

name_to_config: Dict[str, dict] = {c["name"]: c for c in configs}
