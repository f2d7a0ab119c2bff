"""ctypes binding of ``libb200_token_loop.so`` (the C ABI in ``include/b200_token_loop.h``).

The binding is deliberately thin: every Python-visible operator in this package
ends in exactly one of the calls declared here, and there is no fallback of any
kind — if the shared library is missing the import fails with instructions to
build it.
"""
from __future__ import annotations

import ctypes
import os
from ctypes import c_char_p, c_float, c_int, c_int32, c_int64, c_void_p, POINTER
from pathlib import Path

PKG_DIR = Path(__file__).resolve().parent
LIB_PATH = PKG_DIR / "lib" / "libb200_token_loop.so"

B200_OK = 0
ERROR_NAMES = {
    1: "B200_ERR_INVALID_ARGUMENT",
    2: "B200_ERR_CUDA",
    3: "B200_ERR_TIMEOUT",
    4: "B200_ERR_UNSUPPORTED",
    5: "B200_ERR_STATE",
}

EPILOGUE_NONE = 0
EPILOGUE_SWIGLU = 1
EPILOGUE_GEGLU = 2
EPILOGUE_RELU2 = 4
EPILOGUE_GELU_ERF = 5
EPILOGUE_CLAMPED_SWIGLU = 6
EPILOGUE_F32 = 7

DTYPE_BF16, DTYPE_F32 = 0, 1
MIXER_LATENT_ATTENTION, MIXER_WINDOW_ATTENTION, MIXER_LINEAR_ATTENTION, MIXER_STATE_SPACE, MIXER_DELTA_RULE = 0, 1, 2, 3, 4
MIXER_LIGHTNING, MIXER_MATRIX_MEMORY = 5, 6
RULE_STATE_SPACE, RULE_DELTA, RULE_LIGHTNING, RULE_MATRIX_MEMORY = 0, 1, 2, 3
HEAD_NORM_NONE, HEAD_NORM_WEIGHTED, HEAD_NORM_UNIT = 0, 1, 2
GATE_NONE, GATE_ELEMENT, GATE_HEAD = 0, 1, 2
JOIN_SUM, JOIN_NORMED = 0, 1
NORM_INPUT, NORM_OUTPUT, NORM_BOTH = 0, 1, 2
NORM_RMS, NORM_LAYER = 0, 1
SCORE_SIGMOID, SCORE_SOFTMAX = 0, 1
MLP_NONE, MLP_DENSE, MLP_TABLE_MOE, MLP_SCORED_MOE = 0, 1, 2, 3


def epilogue_is_gated(epilogue: int) -> bool:
    """Does the activation take two stacked halves (gate, up)?"""
    return epilogue not in (EPILOGUE_NONE, EPILOGUE_RELU2, EPILOGUE_GELU_ERF, EPILOGUE_F32)


class B200Error(RuntimeError):
    """Raised when a C-ABI call returns a non-zero status (the reference raises c10::Error)."""

    def __init__(self, code: int, message: str):
        super().__init__(f"{ERROR_NAMES.get(code, code)}: {message}")
        self.code = code


_P = c_void_p
_I = c_int
_L = c_int64
_F = c_float

# name -> (restype, argtypes).  Every symbol include/b200_token_loop.h declares is listed.
PROTOTYPES: dict[str, tuple] = {
    "b200_last_error": (c_char_p, []),
    "b200_abi_version": (_I, []),
    "b200_read_device_status": (_I, [POINTER(c_int32), _P]),
    "b200_rmsnorm": (_I, [_P, _P, _P, _I, _I, _F, _P]),
    "b200_fused_add_rmsnorm": (_I, [_P, _P, _P, _I, _I, _F, _P]),
    "b200_qk_rmsnorm_strided": (_I, [_P, _P, _P, _P, _I, _I, _I, _I, _L, _L, _L, _L, _F, _P]),
    "b200_rope_neox_inplace": (_I, [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _L, _L, _L, _L, _P]),
    "b200_store_kv": (_I, [_P, _P, _P, _P, _P, _I, _I, _I, _L, _L, _L, _P]),
    "b200_qknorm_rope_store": (_I, [_P, _P, _P, _P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _L, _F, _I, _P]),
    "b200_silu_and_mul": (_I, [_P, _P, _I, _I, _P]),
    "b200_gelu_and_mul": (_I, [_P, _P, _I, _I, _P]),
    "b200_embedding": (_I, [_P, _P, _P, _I, _I, _I, _P]),
    "b200_gather_int32_2d": (_I, [_P, _P, _L, _L, _L, _P, _P, _L, _P]),
    "b200_write_token_pool": (_I, [_P, _L, _L, _L, _P, _P, _P, _L, _P]),
    "b200_linear": (_I, [_P, _P, _P, _P, _I, _I, _I, _L, _I, _P]),
    "b200_moe_workspace_bytes": (_L, [_I, _I, _I, _I, _I]),
    "b200_moe_route": (_I, [_P, _P, _P, _P, _I, _I, _I, _I, _P]),
    "b200_moe_forward": (_I, [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _P, _L, _P]),
    "b200_moe_forward_local": (_I, [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P, _L, _P]),
    "b200_attention_decode_workspace_bytes": (_L, [_I, _I, _I, _I]),
    "b200_attention_decode": (_I, [_P, _P, _L, _L, _P, _P, _L, _P, _L, _P, _P, _I, _I, _I, _I, _I, _F, _P, _L, _P]),
    "b200_attention_decode_noalloc": (_I, [_P, _P, _L, _L, _P, _P, _L, _P, _L, _P, _P, _I, _I, _I, _I, _I, _F, _P]),
    "b200_attention_decode_noalloc_status": (_I, [POINTER(c_int32), _P]),
    "b200_attention_prefill": (_I, [_P, _P, _L, _L, _P, _P, _L, _P, _L, _P, _P, _P, _I, _I, _I, _I, _I, _I, _F, _P]),
    "b200_argmax": (_I, [_P, _P, _I, _I, _L, _P]),
    "b200_sample": (_I, [_P, _P, _I, _I, _L, _P, _P, _P, _P, ctypes.c_uint64, _P, _P]),
    "b200_sample_from_probs": (_I, [_P, _P, _I, _I, _P, _I, _P, _F, _P, _P]),
    "b200_comm_create": (_I, [_I, _I, _L, POINTER(c_void_p)]),
    "b200_comm_handle_bytes": (_I, []),
    "b200_comm_export": (_I, [_P, _P]),
    "b200_comm_connect": (_I, [_P, _P]),
    "b200_comm_buffer": (c_void_p, [_P, _I]),
    "b200_comm_destroy": (_I, [_P]),
    "b200_comm_set_wait_limit_ns": (_I, [_P, ctypes.c_uint64]),
    "b200_comm_connect_loopback": (_I, [_P]),
    "b200_comm_loopback_announce": (_I, [_P, ctypes.c_uint32, _P]),
    "b200_engine_comm": (c_void_p, [_P]),
    "b200_decode_chain_grid": (_I, []),
    "b200_allreduce": (_I, [_P, _I, _P, _I, _I, _P]),
    "b200_allreduce_fused_add_rmsnorm": (_I, [_P, _I, _P, _P, _P, _I, _I, _F, _I, _P]),
    "b200_comm_region_bytes": (c_int64, [c_int64]),
    "b200_comm_create_on": (_I, [_I, _I, c_int64, _P, POINTER(c_void_p)]),
    "b200_comm_connect_pointers": (_I, [_P, _P, _P]),
    "b200_comm_uses_multicast": (_I, [_P]),
    "b200_engine_comm_region_bytes": (c_int64, [_P]),
    "b200_engine_comm_attach": (_I, [_P, _P, _P, _P]),
    "b200_engine_comm_export": (_I, [_P, _P]),
    "b200_engine_comm_connect": (_I, [_P, _P]),
    "b200_latent_attention_workspace_bytes": (_L, [_I, _I, _I]),
    "b200_latent_attention": (_I, [_P, _P, _P, _L, _P, _L, _P, _P, _I, _I, _I, _I, _F, _I, _I, _P, _L, _P]),
    "b200_latent_attention_part": (_I, [_P, _P, _P, _L, _P, _L, _P, _P, _I, _I, _I, _I, _I, _F, _I, _I, _P, _L, _P]),
    "b200_rotate_pairs": (_I, [_P, _I, _I, _I, _I, _P, _P, _P, _I, _I, _P]),
    "b200_residual_pair_norm": (_I, [_P, _P, _P, _P, _P, _P, _F, _P, _P, _I, _I, _I, _F, _I, _P]),
    "b200_recurrence": (_I, [_P, _I, _P]),
    "b200_recurrence_scratch": (_I, [_I, _I, _I, _I, _I, _I, _I, _I, POINTER(c_int64)]),
    "b200_residual_norm": (_I, [_P, _P, _I, _P, _P, _P, _I, _L, _F, _I, _P, _F, _F, _I, _I, _I, _F, _I, _P]),
    "b200_table_route": (_I, [_P, _P, _P, _P, _P, _I, _I, _I, _I, _P]),
    "b200_linear_heads": (_I, [_P, _P, _P, _I, _I, _I, _I, _P]),
    "b200_linear_f32": (_I, [_P, _P, _P, _I, _I, _I, _I, _P, _P, _I, _P]),
    "b200_linear_act": (_I, [_P, _P, _P, _I, _I, _I, _I, _F, _I, _P]),
    "b200_residual_post_norm": (_I, [_P, _P, _P, _P, _P, _I, _L, _P, _I, _P, _P, _I, _I, _I, _F, _I, _P]),
    "b200_residual_layer_norm": (_I, [_P, _P, _P, _P, _P, _I, _L, _P, _F, _I, _P, _P, _P, _P, _I, _I, _I, _F, _I, _P]),
    "b200_score_route": (_I, [_P, _P, _P, _P, _P, _P, _P, _I, _P, _L, _I, _I, _I, _I, _I, _F, _I, _I, _P, _P]),
    "b200_head_mix_scratch_bytes": (_L, [_I, _I, _I, _I, _I]),
    "b200_head_mix_workspace_bytes": (_L, [_I, _I, _I]),
    "b200_recurrence_memory_bytes": (_L, [_I, _I]),
    "b200_head_prepare": (_I, [_P, _I, _P]),
    "b200_window_attention": (_I, [_P, _I, _P]),
    "b200_linear_attention": (_I, [_P, _I, _P]),
    "b200_pad_width": (_I, [_I]),
    "b200_pad_head_dim": (_I, [_I]),
    "b200_pad_latent": (_I, [_I]),
    "b200_latent_rope_at": (_I, [_I]),
    "b200_engine_create_stack": (_I, [_P, _P, _P, POINTER(c_void_p)]),
    "b200_engine_token_logits": (_I, [_P, _P, _I, _P]),
    "b200_engine_trace_residual": (_I, [_P, _P]),
    "b200_engine_create": (_I, [_P, _P, POINTER(c_void_p)]),
    "b200_engine_destroy": (_I, [_P]),
    "b200_engine_tensor": (_I, [_P, c_char_p, _I, POINTER(c_void_p), POINTER(c_int64)]),
    "b200_engine_load": (_I, [_P, c_char_p, _I, _P, _L]),
    "b200_engine_write_table": (_I, [_P, _I, _P, _P, _P, _L]),
    "b200_engine_capture_graphs": (_I, [_P, _P, _I]),
    "b200_engine_step": (_I, [_P, _P, _P]),
    "b200_engine_synchronize": (_I, [_P]),
    "b200_engine_set_eos_token": (_I, [_P, c_int32]),
    "b200_engine_result_slots": (_I, []),
    "b200_engine_step_async": (_I, [_P, _P, _P, POINTER(c_int64)]),
    "b200_engine_wait": (_I, [_P, c_int64, POINTER(c_void_p), POINTER(c_void_p)]),
    "b200_engine_read_logits": (_I, [_P, _P, _I]),
    "b200_engine_stream": (c_void_p, [_P]),
    "b200_engine_last_step_ms": (_I, [_P, POINTER(c_float)]),
    "b200_engine_set_profiling": (_I, [_P, _I]),
    "b200_engine_read_profile_allreduce": (_I, [_P, POINTER(c_float), POINTER(c_int32)]),
    "b200_engine_read_profile": (_I, [_P, POINTER(c_float), POINTER(c_int32), POINTER(c_int32)]),
}


class ModelConfigStruct(ctypes.Structure):
    """b200_model_config."""
    _fields_ = [
        ("num_layers", c_int32), ("hidden_size", c_int32), ("num_qo_heads", c_int32),
        ("num_kv_heads", c_int32), ("head_dim", c_int32), ("intermediate_size", c_int32),
        ("vocab_size", c_int32), ("rms_norm_eps", c_float), ("rope_theta", c_float),
        ("max_position", c_int32), ("tie_word_embeddings", c_int32), ("qk_norm", c_int32),
        ("fused_residual", c_int32), ("attention_bias", c_int32), ("hidden_act", c_int32),
        ("num_experts", c_int32), ("num_experts_per_tok", c_int32),
        ("moe_intermediate_size", c_int32), ("norm_topk_prob", c_int32),
    ]


class LayerConfigStruct(ctypes.Structure):
    """b200_layer_config."""
    _fields_ = [
        ("mixer", c_int32), ("heads", c_int32), ("head_dim", c_int32), ("value_dim", c_int32),
        ("q_rank", c_int32), ("kv_rank", c_int32), ("score_scale", c_float), ("mlp", c_int32),
        ("intermediate", c_int32), ("epilogue", c_int32), ("num_experts", c_int32),
        ("experts_per_tok", c_int32), ("kv_heads", c_int32), ("window", c_int32), ("keep_first", c_int32),
        ("rotary_dim", c_int32), ("rope_base", ctypes.c_double), ("value_mix", c_int32),
        ("decay_rank", c_int32), ("decay_tau", c_float), ("router_groups", c_int32), ("router_keep", c_int32),
        ("router_scale", c_float), ("shared_intermediate", c_int32), ("act_limit", c_float),
        ("shared_act_limit", c_float), ("head_norm", c_int32), ("gate", c_int32), ("qkv_bias", c_int32),
        ("sink", c_int32), ("chunk", c_int32), ("rope_factor", ctypes.c_double), ("rope_low", ctypes.c_double),
        ("rope_high", ctypes.c_double), ("rope_original", ctypes.c_double), ("kv_from", c_int32),
        ("conv_taps", c_int32), ("norm_groups", c_int32), ("beside", c_int32), ("join", c_int32), ("out_scale", c_float),
        ("value_rotary", c_int32), ("head_mix", c_int32), ("gate_cap", c_float), ("score", c_int32),
        ("identity_experts", c_int32),
    ]


class HeadPrepareArgs(ctypes.Structure):
    """b200_head_prepare_args."""
    _fields_ = [
        ("joint", _P), ("joint_ld", _L), ("tokens", c_int32), ("heads", c_int32), ("kv_heads", c_int32),
        ("dim", c_int32), ("padded_dim", c_int32), ("padded_value_dim", c_int32), ("q_norm", _P), ("k_norm", _P),
        ("eps", c_float), ("rotary_dim", c_int32), ("max_pos", c_int32), ("cos_table", _P), ("sin_table", _P),
        ("positions", _P), ("out_loc", _P), ("k_cache", _P), ("v_cache", _P), ("num_slots", _L), ("mix", c_int32),
        ("lambda_", _P), ("first_values", _P), ("unit_norm", c_int32), ("value_rotary", c_int32), ("value_cos", _P),
        ("value_sin", _P),
    ]


class WindowAttentionArgs(ctypes.Structure):
    """b200_window_attention_args."""
    _fields_ = [
        ("out", _P), ("q", _P), ("q_stride", _L), ("k_cache", _P), ("v_cache", _P), ("num_slots", _L),
        ("page_table", _P), ("page_table_stride", _L), ("table_idx", _P), ("seq_lens", _P), ("qo_indptr", _P),
        ("row_table", _P), ("row_len", _P), ("tokens", c_int32), ("batch", c_int32), ("max_extend", c_int32),
        ("decode", c_int32), ("plain", c_int32), ("heads", c_int32), ("kv_heads", c_int32), ("padded_dim", c_int32),
        ("padded_value_dim", c_int32), ("page_size", c_int32), ("scale", c_float), ("window", c_int32),
        ("keep_first", c_int32), ("gate", _P), ("gate_stride", _L), ("workspace", _P), ("workspace_bytes", _L),
        ("chunk", c_int32), ("sinks", _P), ("gate_per_head", c_int32), ("out_scale", c_float), ("out_stride", _L),
        ("head_mix", _P), ("value_rotary", c_int32), ("max_pos", c_int32), ("value_cos", _P), ("value_sin", _P),
        ("positions", _P), ("score_bound", c_float), ("mix_scratch", _P),
    ]


class LinearAttentionArgs(ctypes.Structure):
    """b200_linear_attention_args."""
    _fields_ = [
        ("out", _P), ("joint", _P), ("joint_ld", _L), ("tokens", c_int32), ("batch", c_int32), ("decode", c_int32),
        ("plain", c_int32), ("table_idx", _P), ("cached", _P), ("qo_indptr", _P), ("state", _P), ("heads", c_int32),
        ("dim", c_int32), ("padded_dim", c_int32), ("value_dim", c_int32), ("padded_value_dim", c_int32),
        ("rank", c_int32), ("up_ld", c_int32), ("up", _P), ("bias", _P), ("norm", _P), ("tau", c_float),
        ("eps", c_float), ("q_scale", c_float),
    ]


class RecurrenceArgs(ctypes.Structure):
    """b200_recurrence_args."""
    _fields_ = [
        ("out", _P), ("out_ld", _L), ("joint", _P), ("joint_ld", _L), ("rule", c_int32), ("tokens", c_int32),
        ("batch", c_int32), ("max_extend", c_int32), ("decode", c_int32), ("plain", c_int32), ("table_idx", _P),
        ("cached", _P), ("qo_indptr", _P), ("state", _P), ("conv_state", _P), ("heads", c_int32), ("kv_heads", c_int32),
        ("dim", c_int32), ("padded_dim", c_int32), ("value_dim", c_int32), ("padded_value_dim", c_int32),
        ("taps", c_int32), ("norm_groups", c_int32), ("conv", _P), ("conv_bias", _P), ("decay_log", _P),
        ("step_bias", _P), ("skip", _P), ("norm", _P), ("eps", c_float), ("out_scale", c_float), ("mixed", _P),
        ("steps", _P), ("units", _P), ("chunks", _P), ("gate_cap", c_float), ("memory", _P),
    ]


class StackConfigStruct(ctypes.Structure):
    """b200_stack_config."""
    _fields_ = [
        ("num_layers", c_int32), ("layers", POINTER(LayerConfigStruct)), ("dtype", c_int32),
        ("norm_offset", c_float), ("logit_scale", c_float), ("norm_output", c_int32), ("num_beside", c_int32),
        ("beside", POINTER(LayerConfigStruct)), ("norm_kind", c_int32), ("embed_scale", c_float),
    ]


class EngineConfigStruct(ctypes.Structure):
    """b200_engine_config."""
    _fields_ = [
        ("page_size", c_int32), ("num_pages", c_int32), ("max_running_req", c_int32),
        ("max_seq_len", c_int32), ("max_extend_tokens", c_int32), ("tp_rank", c_int32),
        ("tp_size", c_int32), ("expert_parallel", c_int32),
    ]


class StepStruct(ctypes.Structure):
    """b200_step."""
    _fields_ = [
        ("phase", c_int32), ("num_reqs", c_int32), ("num_padded_reqs", c_int32),
        ("table_idx", c_void_p), ("cached_lens", c_void_p), ("extend_lens", c_void_p),
        ("write_pos", c_void_p), ("temperatures", c_void_p), ("top_k", c_void_p),
        ("top_p", c_void_p), ("seeds", c_void_p), ("step_index", ctypes.c_uint64),
    ]

_lib = None


def load() -> ctypes.CDLL:
    """Load the shared library (once) and attach the prototypes."""
    global _lib
    if _lib is not None:
        return _lib
    path = LIB_PATH
    if not path.exists():
        raise ImportError(
            f"{path} is missing: build it with `python -c 'import __graft_entry__ as g; g.build()'` "
            "(nvcc, sm_100a).  There is no fallback path."
        )
    lib = ctypes.CDLL(str(path))
    for name, (restype, argtypes) in PROTOTYPES.items():
        fn = getattr(lib, name)
        fn.restype = restype
        fn.argtypes = argtypes
    _lib = lib
    return lib


def check(code: int) -> None:
    if code != B200_OK:
        msg = load().b200_last_error()
        raise B200Error(code, msg.decode() if msg else "")


def call(name: str, *args) -> None:
    """Call an int-returning entry point and raise B200Error on a non-zero status."""
    check(getattr(load(), name)(*args))
