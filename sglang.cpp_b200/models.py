"""Model registry: ``config.json`` -> configuration, checkpoint -> engine, chosen by architecture name.

``REGISTRY`` maps the architecture a configuration names ("architectures" of a Hugging Face file, or
"architecture") to the function that reads it.  Two kinds of configuration come out:

* ``ModelConfig``: one layer repeated (Llama, Qwen2, Qwen3, Qwen3-MoE; the fields of
  include/sglang/models/config.h:15-42);
* ``StackConfig``: layers listed one by one (Rapizen).  Each is a ``LayerSpec`` that names its mixer and
  its feed-forward with their sizes; another design made of the same parts needs a reader here and a
  packing in ``weights.py``.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Callable, Optional

import torch

from . import _lib
from .engine import Engine, EngineConfig


@dataclass
class ModelConfig:
    num_layers: int
    hidden_size: int
    num_qo_heads: int
    num_kv_heads: int
    head_dim: int
    intermediate_size: int
    vocab_size: int
    rms_norm_eps: float
    rope_theta: float
    max_position: int
    tie_word_embeddings: bool
    qk_norm: bool
    fused_residual: bool
    hidden_act: str = "silu"
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    attention_bias: bool = False


@dataclass
class LayerSpec:
    """b200_layer_config: one layer of a ``StackConfig``."""
    heads: int
    head_dim: int
    value_dim: int
    q_rank: int
    kv_rank: int
    score_scale: float
    mlp: int = _lib.MLP_NONE
    intermediate: int = 0
    epilogue: int = _lib.EPILOGUE_NONE
    num_experts: int = 0
    experts_per_tok: int = 0
    mixer: int = _lib.MIXER_LATENT_ATTENTION

    def as_tuple(self) -> tuple:
        return (self.mixer, self.heads, self.head_dim, self.value_dim, self.q_rank, self.kv_rank, self.score_scale,
                self.mlp, self.intermediate, self.epilogue, self.num_experts, self.experts_per_tok)


@dataclass
class StackConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: list = field(default_factory=list)
    norm_offset: float = 0.0      # stored norm weights are the gain minus this
    logit_scale: float = 1.0
    tie_word_embeddings: bool = False
    torch_dtype: torch.dtype = torch.bfloat16

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def expands_keys(self, c: LayerSpec) -> bool:
        """Does this layer's prefill expand keys and values (csrc/layer_stack.cu, can_expand)?"""
        return (self.torch_dtype == torch.bfloat16 and c.head_dim <= 128 and c.value_dim <= 128
                and c.score_scale > 0 and c.heads <= 65535)


def _uniform(qk_norm: bool, fused_residual: bool, attention_bias: bool = False, moe: bool = False) -> Callable:
    def read(c: dict) -> ModelConfig:
        heads = c["num_attention_heads"]
        return ModelConfig(
            c["num_hidden_layers"], c["hidden_size"], heads, c.get("num_key_value_heads", heads),
            c.get("head_dim") or c["hidden_size"] // heads, c["intermediate_size"], c["vocab_size"],
            c.get("rms_norm_eps", 1e-6), c.get("rope_theta", 10000.0), c.get("max_position_embeddings", 4096),
            bool(c.get("tie_word_embeddings", False)), qk_norm, fused_residual, c.get("hidden_act", "silu"),
            c.get("num_experts", 0) if moe else 0, c.get("num_experts_per_tok", 0) if moe else 0,
            c.get("moe_intermediate_size", 0) if moe else 0, bool(c.get("norm_topk_prob", True)), attention_bias)
    return read


def read_rapizen(c: dict) -> StackConfig:
    layers = []
    for i, entry in enumerate(c["layers"]):
        if entry["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
        m = entry["mixer"]
        spec = LayerSpec(m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]))
        ff = entry.get("mlp")
        if ff is not None:
            if ff["kind"] == "dense":
                spec.mlp, spec.intermediate, spec.epilogue = _lib.MLP_DENSE, ff["ff"], _lib.EPILOGUE_GEGLU
            elif ff["kind"] == "moe":
                spec.mlp, spec.intermediate, spec.epilogue = _lib.MLP_TABLE_MOE, ff["expert"]["ff"], _lib.EPILOGUE_RELU2
                spec.num_experts, spec.experts_per_tok = ff["router"]["experts"], ff["router"]["top"]
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {ff['kind']!r}")
        layers.append(spec)
    return StackConfig(c["width"], c["vocab"], float(c["norm"]["eps"]), layers, norm_offset=1.0,
                       logit_scale=float(c.get("logit_scale", 1.0)))


REGISTRY: dict[str, Callable] = {
    "LlamaForCausalLM": _uniform(qk_norm=False, fused_residual=False),
    "Qwen2ForCausalLM": _uniform(qk_norm=False, fused_residual=False, attention_bias=True),
    "Qwen3ForCausalLM": _uniform(qk_norm=True, fused_residual=True),
    "Qwen3MoeForCausalLM": _uniform(qk_norm=True, fused_residual=True, moe=True),
    "Rapizen": read_rapizen,
}


def architecture_of(raw: dict) -> str:
    names = raw.get("architectures") or [raw.get("architecture")]
    if names[0] not in REGISTRY:
        raise ValueError(f"unknown architecture {names[0]!r}; known: {', '.join(sorted(REGISTRY))}")
    return names[0]


def read_config(directory, dtype: str = "bfloat16"):
    """The configuration in ``directory/config.json``, to be run in ``dtype``."""
    raw = json.loads((Path(directory) / "config.json").read_text())
    cfg = REGISTRY[architecture_of(raw)](raw)
    if dtype == "float32":
        if not isinstance(cfg, StackConfig):
            raise ValueError("only models whose layers are listed one by one run in float32")
        cfg.torch_dtype = torch.float32
    elif dtype != "bfloat16":
        raise ValueError(f"unknown dtype {dtype!r}")
    return cfg


def load_model(directory, engine_config: EngineConfig, dtype: str = "bfloat16", config: Optional[object] = None) -> Engine:
    """An engine with the checkpoint of ``directory`` uploaded."""
    from .weights import load_checkpoint

    cfg = config if config is not None else read_config(directory, dtype)
    engine = Engine(cfg, engine_config)
    engine.load_weights(load_checkpoint(cfg, directory))
    return engine
