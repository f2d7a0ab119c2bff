"""Model registry: ``config.json`` -> configuration, checkpoint -> engine, chosen by architecture name.

``REGISTRY`` maps the architecture a configuration names ("architectures" of a Hugging Face file, or
"architecture") to the function that reads it.  Two kinds of configuration come out:

* ``ModelConfig``: one layer repeated (Llama, Qwen2, Qwen3, Qwen3-MoE; the fields of
  include/sglang/models/config.h:15-42);
* ``StackConfig``: layers listed one by one (Rapizen, Dilalix, Saluzen, Retotar).  Each is a ``LayerSpec`` that names its mixer and
  its feed-forward with their sizes; another design made of the same parts needs a reader here (and a
  packing in ``weights.py`` where its tensors are named differently).

A reader takes the configuration and the shapes of the checkpoint's tensors (name -> shape), for sizes that
only those give.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field, fields
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


NO_WINDOW = 2 ** 31 - 1


@dataclass
class LayerSpec:
    """b200_layer_config: one layer of a ``StackConfig``."""
    heads: int
    head_dim: int
    value_dim: int
    q_rank: int = 0
    kv_rank: int = 0
    score_scale: float = 1.0
    mlp: int = _lib.MLP_NONE
    intermediate: int = 0
    epilogue: int = _lib.EPILOGUE_NONE
    num_experts: int = 0
    experts_per_tok: int = 0
    mixer: int = _lib.MIXER_LATENT_ATTENTION
    # window attention
    kv_heads: int = 0
    window: int = NO_WINDOW
    keep_first: int = 0
    rotary_dim: int = 0
    rope_base: float = 1.0
    value_mix: bool = False
    # linear attention
    decay_rank: int = 0
    decay_tau: float = 1.0
    # scored experts
    router_groups: int = 1
    router_keep: int = 1
    router_scale: float = 1.0
    shared_intermediate: int = 0
    act_limit: float = 0.0
    shared_act_limit: float = 0.0
    # window attention
    head_norm: int = _lib.HEAD_NORM_WEIGHTED
    gate: int = _lib.GATE_ELEMENT
    qkv_bias: bool = False
    sink: bool = False            # a score per head in the softmax's denominator ...
    sink_learned: bool = True     # ... from the checkpoint, or 0
    chunk: int = 0                # keys of the query's own chunk, instead of a window
    # rotations whose long wavelengths are stretched (or, with rope_original 0, all of them); latent attention counts its rotary_dim rotated dimensions in
    # head_dim
    rope_factor: float = 0.0
    rope_low: float = 1.0
    rope_high: float = 1.0
    rope_original: float = 0.0
    kv_from: int = -1             # latent and window attention: the layer whose cache is read
    # recurrences: head_dim state rows, kv_heads heads of k and q
    conv_taps: int = 1
    norm_groups: int = 1
    # window attention: cached values turn with their position, the output turns back; heads mix their weights
    value_rotary: bool = False
    head_mix: bool = False
    gate_cap: float = 0.0         # matrix memory
    # scored experts: by sigmoid or softmax scores; experts that return their input
    score: int = _lib.SCORE_SIGMOID
    identity_experts: int = 0
    decays: tuple = ()            # lightning: one per head
    # a second mixer on the same input, and how the results meet
    beside: Optional["LayerSpec"] = None
    join: int = _lib.JOIN_SUM
    out_scale: float = 1.0

    def as_struct(self) -> _lib.LayerConfigStruct:
        """(``beside`` becomes an index once the whole stack is known: Engine.)"""
        values = {f.name: getattr(self, f.name) for f in fields(self) if f.name not in ("beside", "sink_learned", "decays")}
        return _lib.LayerConfigStruct(beside=-1, **{k: int(v) if isinstance(v, bool) else v for k, v in values.items()})


@dataclass
class StackConfig:
    hidden_size: int
    vocab_size: int
    rms_norm_eps: float
    layers: list = field(default_factory=list)
    norm_offset: float = 0.0      # stored norm weights are the gain minus this
    logit_scale: float = 1.0
    norm_output: int = _lib.NORM_INPUT   # norms on what the blocks read, on what they return, or on both
    tie_word_embeddings: bool = False
    torch_dtype: torch.dtype = torch.bfloat16
    norm_kind: int = _lib.NORM_RMS       # RMS norms, or layer norms with biases
    embed_scale: float = 1.0

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def carries_state(self) -> bool:
        kinds = (_lib.MIXER_LINEAR_ATTENTION, _lib.MIXER_STATE_SPACE, _lib.MIXER_DELTA_RULE, _lib.MIXER_LIGHTNING,
                 _lib.MIXER_MATRIX_MEMORY)
        return any(m is not None and m.mixer in kinds for c in self.layers for m in (c, c.beside))

    def expands_keys(self, c: LayerSpec) -> bool:
        """Does this layer's prefill expand keys and values (csrc/layer_stack.cu, can_expand)?"""
        return (self.torch_dtype == torch.bfloat16 and c.head_dim <= 128 and c.value_dim <= 128
                and c.score_scale > 0 and c.heads <= 65535)


def _uniform(qk_norm: bool, fused_residual: bool, attention_bias: bool = False, moe: bool = False) -> Callable:
    def read(c: dict, shapes: Optional[dict] = None) -> ModelConfig:
        heads = c["num_attention_heads"]
        return ModelConfig(
            c["num_hidden_layers"], c["hidden_size"], heads, c.get("num_key_value_heads", heads),
            c.get("head_dim") or c["hidden_size"] // heads, c["intermediate_size"], c["vocab_size"],
            c.get("rms_norm_eps", 1e-6), c.get("rope_theta", 10000.0), c.get("max_position_embeddings", 4096),
            bool(c.get("tie_word_embeddings", False)), qk_norm, fused_residual, c.get("hidden_act", "silu"),
            c.get("num_experts", 0) if moe else 0, c.get("num_experts_per_tok", 0) if moe else 0,
            c.get("moe_intermediate_size", 0) if moe else 0, bool(c.get("norm_topk_prob", True)), attention_bias)
    return read


def read_rapizen(c: dict, shapes: Optional[dict] = None) -> StackConfig:
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


def read_dilalix(c: dict, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, entry in enumerate(c["layers"]):
        m = entry["mixer"]
        spec = LayerSpec(m["heads"], m["dim"], m["vdim"])
        if entry["type"] == "attention":
            rot, mask = m.get("rot") or {}, m.get("mask") or {}
            spec.mixer, spec.kv_heads, spec.score_scale = _lib.MIXER_WINDOW_ATTENTION, m["kv_heads"], float(m["scale"])
            spec.rotary_dim, spec.rope_base = rot.get("dims", 0), float(rot.get("base", 1.0))
            spec.window, spec.keep_first = min(mask.get("size", NO_WINDOW), NO_WINDOW), mask.get("keep_first", 0)
            spec.value_mix = bool(m.get("v_mix", False))
        elif entry["type"] == "gla":
            spec.mixer, spec.decay_tau = _lib.MIXER_LINEAR_ATTENTION, float(m["tau"])
            name = f"l{i}.mix.a1"
            if not shapes or name not in shapes:
                raise ValueError(f"layer {i}: the rank of the decay is that of tensor {name}, which is not there")
            spec.decay_rank = shapes[name][0]
        else:
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
        ff = entry.get("mlp")
        if ff is not None:
            if ff["kind"] == "dense":
                spec.mlp, spec.intermediate, spec.epilogue = _lib.MLP_DENSE, ff["ff"], _lib.EPILOGUE_GELU_ERF
            elif ff["kind"] == "moe":
                r, groups, shared = ff["router"], ff["router"].get("groups") or {}, ff.get("shared")
                spec.mlp, spec.epilogue = _lib.MLP_SCORED_MOE, _lib.EPILOGUE_CLAMPED_SWIGLU
                spec.intermediate, spec.act_limit = ff["expert"]["ff"], float(ff["expert"]["limit"])
                spec.num_experts, spec.experts_per_tok, spec.router_scale = r["experts"], r["top"], float(r.get("scale", 1.0))
                spec.router_groups, spec.router_keep = groups.get("count", 1), groups.get("keep", groups.get("count", 1))
                if shared:
                    spec.shared_intermediate, spec.shared_act_limit = shared["ff"], float(shared["limit"])
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {ff['kind']!r}")
        layers.append(spec)
    return StackConfig(c["width"], c["vocab"], float(c["norm"]["eps"]), layers, norm_output=_lib.NORM_OUTPUT)


def _set_rotation(spec: LayerSpec, rot: dict) -> None:
    spec.rotary_dim, spec.rope_base = rot["dims"], float(rot["base"])
    s = rot.get("scaling")
    if s:
        spec.rope_factor, spec.rope_low, spec.rope_high = float(s["factor"]), float(s["low"]), float(s["high"])
        spec.rope_original = float(s["original"])


def _biased_attention(m: dict) -> LayerSpec:
    """Grouped-query attention with projection biases and a sink, without norms on queries and keys."""
    spec = LayerSpec(m["heads"], m["dim"], m["vdim"], score_scale=float(m["scale"]), mixer=_lib.MIXER_WINDOW_ATTENTION,
                     kv_heads=m["kv_heads"], head_norm=_lib.HEAD_NORM_NONE, qkv_bias=True, sink=True)
    _set_rotation(spec, m["rot"])
    return spec


def _state_space(m: dict) -> LayerSpec:
    return LayerSpec(m["heads"], m["state"], m["vdim"], mixer=_lib.MIXER_STATE_SPACE, kv_heads=m["groups"],
                     conv_taps=m["conv"], norm_groups=m["norm_groups"])


def _delta_rule(m: dict) -> LayerSpec:
    return LayerSpec(m["heads"], m["dim"], m["vdim"], mixer=_lib.MIXER_DELTA_RULE, kv_heads=m["kv_heads"],
                     conv_taps=m["conv"])


def read_saluzen(c: dict, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, entry in enumerate(c["layers"]):
        m = entry["mixer"]
        if entry["type"] == "parallel":
            spec = _biased_attention(m["left"])
            spec.sink_learned = False
            spec.beside, spec.join = _state_space(m["right"]), _lib.JOIN_NORMED
        elif entry["type"] == "parallel_2":
            spec = _biased_attention(m["left"])
            spec.chunk, spec.gate, spec.out_scale = m["left"]["mask"]["size"], _lib.GATE_HEAD, float(m["left_scale"])
            spec.beside, spec.join = _delta_rule(m["right"]), _lib.JOIN_SUM
            spec.beside.out_scale = float(m["right_scale"])
        elif entry["type"] == "latent_attention":
            spec = LayerSpec(m["heads"], m["dim"] + m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]))
            _set_rotation(spec, {**m["rot"], "dims": m["rot_dim"]})
            if m.get("kv_from") is not None:
                spec.kv_from = m["kv_from"]
        else:
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
        ff = entry.get("mlp")
        if ff is not None:
            if ff["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {ff['kind']!r}")
            spec.mlp, spec.intermediate, spec.epilogue = _lib.MLP_DENSE, ff["ff"], _lib.EPILOGUE_SWIGLU
        layers.append(spec)
    return StackConfig(c["width"], c["vocab"], float(c["norm"]["eps"]), layers, norm_output=_lib.NORM_BOTH)


def _talking_attention(m: dict) -> LayerSpec:
    rot, mask = m.get("rot") or {}, m.get("mask") or {}
    spec = LayerSpec(m["heads"], m["dim"], m["vdim"], score_scale=float(m["scale"]), mixer=_lib.MIXER_WINDOW_ATTENTION,
                     kv_heads=m["kv_heads"], head_norm=_lib.HEAD_NORM_UNIT, value_rotary=True, head_mix=True)
    spec.window = min(mask.get("size", NO_WINDOW), NO_WINDOW)
    spec.rotary_dim, spec.rope_base = rot.get("dims", 0), float(rot.get("base", 1.0))
    if rot.get("scaling"):
        spec.rope_factor = float(rot["scaling"]["factor"])
    if m.get("kv_from") is not None:
        spec.kv_from = m["kv_from"]
    return spec


def read_retotar(c: dict, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, entry in enumerate(c["layers"]):
        m = entry["mixer"]
        if entry["type"] == "attention":
            spec = _talking_attention(m)
        elif entry["type"] == "lightning":
            if len(m["decay"]) != m["heads"]:
                raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
            spec = LayerSpec(m["heads"], m["dim"], m["vdim"], mixer=_lib.MIXER_LIGHTNING, kv_heads=m["heads"], norm_groups=1,
                             decays=tuple(map(float, m["decay"])))
        elif entry["type"] == "mlstm":
            spec = LayerSpec(m["heads"], m["dim"], m["vdim"], mixer=_lib.MIXER_MATRIX_MEMORY, kv_heads=m["heads"],
                             norm_groups=m["heads"], gate_cap=float(m["gate_cap"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
        ff = entry.get("mlp")
        if ff is not None:
            if ff["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {ff['kind']!r}")
            r, groups = ff["router"], ff["router"].get("groups") or {}
            spec.mlp, spec.intermediate, spec.epilogue = _lib.MLP_SCORED_MOE, ff["expert"]["ff"], _lib.EPILOGUE_SWIGLU
            spec.score, spec.num_experts, spec.identity_experts = _lib.SCORE_SOFTMAX, r["experts"], r.get("identity", 0)
            spec.experts_per_tok = r["top"]
            spec.router_groups, spec.router_keep = groups.get("count", 1), groups.get("keep", groups.get("count", 1))
        layers.append(spec)
    return StackConfig(c["width"], c["vocab"], float(c["norm"]["eps"]), layers, norm_output=_lib.NORM_BOTH,
                       norm_kind=_lib.NORM_LAYER, embed_scale=float((c.get("embedding") or {}).get("scale", 1.0)))


REGISTRY: dict[str, Callable] = {
    "LlamaForCausalLM": _uniform(qk_norm=False, fused_residual=False),
    "Qwen2ForCausalLM": _uniform(qk_norm=False, fused_residual=False, attention_bias=True),
    "Qwen3ForCausalLM": _uniform(qk_norm=True, fused_residual=True),
    "Qwen3MoeForCausalLM": _uniform(qk_norm=True, fused_residual=True, moe=True),
    "Rapizen": read_rapizen,
    "Dilalix": read_dilalix,
    "Saluzen": read_saluzen,
    "Retotar": read_retotar,
}


def architecture_of(raw: dict) -> str:
    names = raw.get("architectures") or [raw.get("architecture")]
    if names[0] not in REGISTRY:
        raise ValueError(f"unknown architecture {names[0]!r}; known: {', '.join(sorted(REGISTRY))}")
    return names[0]


def read_config(directory, dtype: str = "bfloat16"):
    """The configuration in ``directory/config.json``, to be run in ``dtype``."""
    from .weights import tensor_shapes

    raw = json.loads((Path(directory) / "config.json").read_text())
    cfg = REGISTRY[architecture_of(raw)](raw, tensor_shapes(directory))
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
