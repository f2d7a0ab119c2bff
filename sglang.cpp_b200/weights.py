"""Checkpoint loading: safetensors shards -> the packed layouts the engine holds.

Restates the host side of the reference's loader (src/models/weight_loader.cc): the safetensors
header walk (:357-420), the name normalisation (:195-211), the merge of q/k/v into ``qkv_proj`` and
of gate/up into ``gate_up_proj`` (:27-41, 62-120) and the stacking of per-expert tensors into
``[E, ...]`` blocks (:43, 236-258).  Sharding for tensor / expert parallelism is done afterwards by
``tp.shard_layer`` when the engine uploads (``Engine.load_weights``).  Pure torch / numpy, no CUDA.

Not restated: the FP8 block-quantised checkpoints the reference dequantises at load (:213-234);
only BF16 / F16 / F32 and I32 (index tables) tensors are accepted.

Models whose layers are listed one by one (``models.StackConfig``) have a packing of their own,
``pack_layer_stack``: the layouts of ``b200_engine_create_stack``, zero-padded.
"""
from __future__ import annotations

import json
import math
import re
import struct
from pathlib import Path

import numpy as np
import torch

_DTYPES = {"BF16": (torch.bfloat16, 2), "F16": (torch.float16, 2), "F32": (torch.float32, 4), "I32": (torch.int32, 4)}
_EXPERT = re.compile(r"^(.*\.experts)\.(\d+)\.(.+)$")


def read_safetensors(path) -> dict:
    """name -> tensor for one ``.safetensors`` file (8-byte little-endian header length, a JSON
    header of dtype / shape / data_offsets, then the raw little-endian data).  The tensors are
    views of a read-only memory map."""
    path = Path(path)
    with open(path, "rb") as f:
        (hlen,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(hlen))
    data = np.memmap(path, dtype=np.uint8, mode="r", offset=8 + hlen)
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        if info["dtype"] not in _DTYPES:
            raise ValueError(f"Unsupported safetensors dtype: {info['dtype']} ({name})")
        dtype, width = _DTYPES[info["dtype"]]
        lo, hi = info["data_offsets"]
        shape = tuple(info["shape"])
        n = int(np.prod(shape)) if shape else 1
        if hi - lo != n * width:
            raise ValueError(f"{name}: {hi - lo} bytes for shape {shape} of {info['dtype']}")
        buf = np.frombuffer(data[lo:hi], dtype=np.uint8)
        out[name] = torch.frombuffer(bytearray(buf.tobytes()), dtype=dtype).reshape(shape)
    return out


def tensor_shapes(directory) -> dict:
    """name -> shape of every tensor in the ``.safetensors`` files of a directory (headers only)."""
    shapes = {}
    for path in sorted(Path(directory).glob("*.safetensors")):
        with open(path, "rb") as f:
            (hlen,) = struct.unpack("<Q", f.read(8))
            header = json.loads(f.read(hlen))
        shapes.update({k: tuple(v["shape"]) for k, v in header.items() if k != "__metadata__"})
    return shapes


def write_safetensors(path, tensors: dict) -> None:
    """The inverse of read_safetensors (tests and tools; the same dtypes)."""
    names = {v[0]: k for k, v in _DTYPES.items()}
    header, blobs, off = {}, [], 0
    for name, t in tensors.items():
        t = t.contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(header, separators=(",", ":")).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)))
        f.write(h)
        for b in blobs:
            f.write(b)


def normalize_weight_name(name: str) -> str:
    """src/models/weight_loader.cc:195-200."""
    return name[len("language_model."):] if name.startswith("language_model.") else name


def pack_checkpoint(cfg, tensors: dict) -> dict:
    """Hugging Face parameter names -> {"embed", "lm_head", "final_norm", "layers": [...]} with
    qkv = cat(q, k, v), gate_up = cat(gate, up) and experts stacked, all cast to bf16 (the dtype
    the reference's ``model.to(device, dtype)`` ends with, weight_loader.cc:542)."""
    t = {normalize_weight_name(k): v for k, v in tensors.items()}
    bf = lambda x: x.to(torch.bfloat16).contiguous()

    def need(name):
        if name not in t:
            raise KeyError(f"checkpoint has no tensor {name}")
        return t[name]

    w = {"embed": bf(need("model.embed_tokens.weight")), "final_norm": bf(need("model.norm.weight")), "layers": []}
    w["lm_head"] = w["embed"] if cfg.tie_word_embeddings or "lm_head.weight" not in t else bf(t["lm_head.weight"])
    for i in range(cfg.num_layers):
        p = f"model.layers.{i}."
        a = p + "self_attn."
        L = {"qkv": bf(torch.cat([need(a + "q_proj.weight"), need(a + "k_proj.weight"), need(a + "v_proj.weight")], 0)),
             "o": bf(need(a + "o_proj.weight")),
             "input_norm": bf(need(p + "input_layernorm.weight")),
             "post_norm": bf(need(p + "post_attention_layernorm.weight"))}
        if cfg.attention_bias:
            L["qkv_bias"] = bf(torch.cat([need(a + "q_proj.bias"), need(a + "k_proj.bias"), need(a + "v_proj.bias")], 0))
        if cfg.qk_norm:
            L["q_norm"] = bf(need(a + "q_norm.weight"))
            L["k_norm"] = bf(need(a + "k_norm.weight"))
        m = p + "mlp."
        if cfg.num_experts > 0:
            L["router"] = bf(need(m + "gate.weight"))
            gu, dn = [], []
            for e in range(cfg.num_experts):
                x = f"{m}experts.{e}."
                gu.append(torch.cat([need(x + "gate_proj.weight"), need(x + "up_proj.weight")], 0))
                dn.append(need(x + "down_proj.weight"))
            L["experts_gate_up"] = bf(torch.stack(gu, 0))
            L["experts_down"] = bf(torch.stack(dn, 0))
        else:
            L["gate_up"] = bf(torch.cat([need(m + "gate_proj.weight"), need(m + "up_proj.weight")], 0))
            L["down"] = bf(need(m + "down_proj.weight"))
        w["layers"].append(L)
    _check_shapes(cfg, w)
    return w


def unpack_checkpoint(cfg, w: dict) -> dict:
    """Packed layouts -> Hugging Face parameter names (the inverse of pack_checkpoint)."""
    d = cfg.head_dim
    qd, kd = cfg.num_qo_heads * d, cfg.num_kv_heads * d
    out = {"model.embed_tokens.weight": w["embed"], "model.norm.weight": w["final_norm"]}
    if not cfg.tie_word_embeddings:
        out["lm_head.weight"] = w["lm_head"]
    for i, L in enumerate(w["layers"]):
        p = f"model.layers.{i}."
        a = p + "self_attn."
        out[a + "q_proj.weight"], out[a + "k_proj.weight"], out[a + "v_proj.weight"] = (
            L["qkv"][:qd], L["qkv"][qd:qd + kd], L["qkv"][qd + kd:])
        out[a + "o_proj.weight"] = L["o"]
        if "qkv_bias" in L:
            b = L["qkv_bias"]
            out[a + "q_proj.bias"], out[a + "k_proj.bias"], out[a + "v_proj.bias"] = b[:qd], b[qd:qd + kd], b[qd + kd:]
        if "q_norm" in L:
            out[a + "q_norm.weight"], out[a + "k_norm.weight"] = L["q_norm"], L["k_norm"]
        out[p + "input_layernorm.weight"] = L["input_norm"]
        out[p + "post_attention_layernorm.weight"] = L["post_norm"]
        m = p + "mlp."
        if "experts_gate_up" in L:
            ie = cfg.moe_intermediate_size
            out[m + "gate.weight"] = L["router"]
            for e in range(cfg.num_experts):
                x = f"{m}experts.{e}."
                out[x + "gate_proj.weight"] = L["experts_gate_up"][e, :ie]
                out[x + "up_proj.weight"] = L["experts_gate_up"][e, ie:]
                out[x + "down_proj.weight"] = L["experts_down"][e]
        else:
            I = cfg.intermediate_size
            out[m + "gate_proj.weight"], out[m + "up_proj.weight"] = L["gate_up"][:I], L["gate_up"][I:]
            out[m + "down_proj.weight"] = L["down"]
    return out


def pack_layer_stack(cfg, tensors: dict) -> dict:
    """Parameter names of the layer-stack designs -> the padded layouts of ``b200_engine_create_stack``, in
    the dtype the model runs in.  Every tensor is checked against the shape its layer's description asks for."""
    from ._lib import (GATE_ELEMENT, GATE_HEAD, HEAD_NORM_WEIGHTED, JOIN_NORMED, MIXER_DELTA_RULE, MIXER_LATENT_ATTENTION,
                       MIXER_LIGHTNING, MIXER_LINEAR_ATTENTION, MIXER_MATRIX_MEMORY, MIXER_STATE_SPACE, MIXER_WINDOW_ATTENTION,
                       MLP_DENSE, MLP_NONE, MLP_SCORED_MOE, NORM_BOTH, NORM_LAYER, SCORE_SOFTMAX, epilogue_is_gated, load)

    lib = load()
    width, head, latent = lib.b200_pad_width, lib.b200_pad_head_dim, lib.b200_pad_latent
    D, V = cfg.hidden_size, cfg.vocab_size
    hp = width(D)

    def need(name, *shape, dtype=None):
        if name not in tensors:
            raise KeyError(f"checkpoint has no tensor {name}")
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name} has shape {tuple(t.shape)}, expected {shape}")
        return t.to(dtype or cfg.torch_dtype)

    def pad(t, *shape):
        out = torch.zeros(shape, dtype=t.dtype)
        out[tuple(slice(0, n) for n in t.shape)] = t
        return out

    def norm(name, to):
        """A norm's weight, and under layer norms its bias."""
        out = {to: pad(need(name, D), hp)}
        if cfg.norm_kind == NORM_LAYER:
            out[to + "_bias"] = pad(need(name + ".b", D), hp)
        return out

    w = {"embed": pad(need("embed", V, D), width(V), hp), **norm("final.norm", "final_norm"), "layers": []}
    if not cfg.tie_word_embeddings:
        w["lm_head"] = pad(need("head", V, D), width(V), hp)
    def rows(name, n, to, k=D, kp=hp):
        """One matrix [n, k], padded to [to, kp]."""
        return pad(need(name, n, k), to, kp)

    def head_rows(name, heads, n, to, k=D, kp=hp):
        """A matrix of `heads` blocks of n rows, every block padded to `to` rows."""
        return pad(need(name, heads * n, k).view(heads, n, k), heads, to, kp).reshape(heads * to, kp)

    def latent_attention(m, c):
        H, dr, dv, qr, kr = c.heads, c.rotary_dim, c.value_dim, c.q_rank, c.kv_rank
        d, at = c.head_dim - dr, lib.b200_latent_rope_at(kr) if dr else kr
        dp, vp, qp, rp, op = head(d + dr), head(dv), width(qr), latent(at + dr), latent(kr)
        # A head's rotated dimensions come first.  Keys take them from the latent as they are, so that one matrix per
        # head turns a latent into its whole key.
        uk = torch.zeros(H, dp, rp, dtype=cfg.torch_dtype)
        uk[:, dr:dr + d, :kr] = need(m + "uk", H * d, kr).view(H, d, kr)
        uk[:, range(dr), range(at, at + dr)] = 1
        uq = need(m + "uq", H * (d + dr), qr).view(H, d + dr, qr)
        L = {"down_qkv": rows(m + "dq", qr, qp), "q_latent_norm": pad(need(m + "dq.norm", qr), qp),
             "uq": pad(torch.cat([uq[:, d:], uq[:, :d]], 1), H, dp, qp), "uk_absorb": uk.transpose(1, 2).contiguous(),
             "uv": pad(need(m + "uv", H * dv, kr).view(H, dv, kr), H, vp, op)}
        if c.kv_from < 0:
            dkv, down = need(m + "dkv", kr + dr, D), torch.zeros(rp, hp, dtype=cfg.torch_dtype)
            down[:kr, :D], down[at:at + dr, :D] = dkv[:kr], dkv[kr:]
            L["down_qkv"] = torch.cat([L["down_qkv"], down])
            L["kv_latent_norm"] = pad(need(m + "dkv.norm", kr), rp)
        if cfg.expands_keys(c):
            L["uk"] = uk
        return L, vp

    # The mixers below return (rows of the input projection, their bias or None, other tensors, padded value dimension).
    def window_attention(m, c):
        H, G, d, dv = c.heads, c.kv_heads, c.head_dim, c.value_dim
        dp, vp = head(d), head(dv)
        parts = [("q", H, d, dp), ("k", G, d, dp), ("v", G, dv, vp)][:3 if c.kv_from < 0 else 1]
        joint = [head_rows(m + name, n, k, kp) for name, n, k, kp in parts]
        if c.gate == GATE_ELEMENT:
            joint.append(head_rows(m + "g", H, dv, vp))
        elif c.gate == GATE_HEAD:
            joint.append(rows(m + "g", H, width(H)))
        joint, L, bias = torch.cat(joint), {}, None
        if c.qkv_bias:
            bias = torch.cat([pad(need(f"{m}{name}.b", n * k).view(n, k), n, kp).flatten() for name, n, k, kp in parts])
            bias = pad(bias, len(joint))
        if c.head_norm == HEAD_NORM_WEIGHTED:
            L.update(q_head_norm=pad(need(m + "q.norm", d), dp), k_head_norm=pad(need(m + "k.norm", d), dp))
        if c.head_mix or c.value_rotary:
            L["head_mix"] = need(m + "talk", H, H, dtype=torch.float32) if c.head_mix else torch.eye(H)
        if c.value_mix:
            L["value_mix"] = need(m + "vmix", dtype=torch.float32).reshape(1)
        if c.sink:
            L["sinks"] = need(m + "sink", H, dtype=torch.float32) if c.sink_learned else torch.zeros(H)
        return joint, bias, L, vp

    def linear_attention(m, c):
        H, d, dv, r = c.heads, c.head_dim, c.value_dim, c.decay_rank
        dp, vp = width(d), width(dv)
        joint = torch.cat([head_rows(m + "q", H, d, dp), head_rows(m + "k", H, d, dp), head_rows(m + "v", H, dv, vp),
                           head_rows(m + "g", H, dv, vp), rows(m + "a1", r, width(r))])
        L = {"decay_up": head_rows(m + "a2", H, d, dp, r, -(-r // 16) * 16),
             "decay_bias": pad(need(m + "a2.b", H * d, dtype=torch.float32).view(H, d), H, dp),
             "head_norm": pad(need(m + "norm", dv), vp)}
        return joint, None, L, vp

    def by_head(t, heads, n, to):
        """The first dimension as `heads` blocks of n, each padded to `to`."""
        return pad(t.reshape(heads, n, *t.shape[1:]), heads, to, *t.shape[1:]).flatten(0, 1)

    def state_space(m, c):
        H, G, N, dv, taps = c.heads, c.kv_heads, c.head_dim, c.value_dim, c.conv_taps
        dp, vp, inner = width(N), width(dv), H * dv
        f32 = dict(dtype=torch.float32)
        blocks = [(H, dv, vp), (G, N, dp), (G, N, dp)]              # x, B, C: the convolution's channels
        split = [n * k for n, k, _ in blocks]
        z, xbc, dt = need(m + "in", 2 * inner + 2 * G * N + H, D).split([inner, sum(split), H])
        joint = torch.cat([by_head(z, H, dv, vp)] + [by_head(t, *b) for t, b in zip(xbc.split(split), blocks)] + [pad(dt, width(H), D)])
        conv = [by_head(t, *b) for t, b in zip(need(m + "conv", sum(split), taps, **f32).split(split), blocks)]
        bias = [by_head(t, *b) for t, b in zip(need(m + "conv.b", sum(split), **f32).split(split), blocks)]
        L = {"conv": torch.cat(conv).T.contiguous(), "conv_bias": torch.cat(bias), "decay_log": need(m + "A_log", H, **f32),
             "step_bias": need(m + "dt_bias", H, **f32), "skip": need(m + "D", H, **f32),
             "head_norm": by_head(need(m + "norm", inner), H, dv, vp)}
        return pad(joint, len(joint), hp), None, L, vp

    def delta_rule(m, c):
        H, G, d, dv, taps = c.heads, c.kv_heads, c.head_dim, c.value_dim, c.conv_taps
        dp, vp = width(d), width(dv)
        f32 = dict(dtype=torch.float32)
        blocks = {"v": (H, dv, vp), "k": (G, d, dp), "q": (G, d, dp)}
        steps = torch.cat([need(m + "a", H, D), need(m + "b", H, D)])
        joint = torch.cat([head_rows(m + "g", H, dv, vp)] + [head_rows(m + n, *b) for n, b in blocks.items()] +
                          [pad(steps, width(2 * H), hp)])
        conv = torch.cat([by_head(need(f"{m}{n}.conv", b[0] * b[1], taps, **f32), *b) for n, b in blocks.items()])
        L = {"conv": conv.T.contiguous(), "conv_bias": torch.zeros(len(conv)), "decay_log": need(m + "A_log", H, **f32),
             "step_bias": need(m + "dt_bias", H, **f32), "head_norm": pad(need(m + "norm", dv), vp)}
        return joint, None, L, vp

    def head_channels(m, c, vp):
        """Gate, values, keys and queries of a recurrence whose heads all have their own."""
        H, d, dv, dp = c.heads, c.head_dim, c.value_dim, width(c.head_dim)
        return [head_rows(m + name, H, n, to) for name, n, to in (("g", dv, vp), ("v", dv, vp), ("k", d, dp), ("q", d, dp))]

    def lightning(m, c):
        H, dv, vp = c.heads, c.value_dim, width(c.value_dim)
        # (a decay of 0 as one that leaves nothing in fp32)
        decay = torch.tensor([max(math.log(g), -250.0) if g > 0 else -250.0 for g in c.decays])
        L = {"decay_log": decay, "head_norm": by_head(need(m + "norm", H * dv), H, dv, vp)}
        return torch.cat(head_channels(m, c, vp)), None, L, vp

    def matrix_memory(m, c):
        H, dv, vp = c.heads, c.value_dim, width(c.value_dim)
        gates = torch.cat([need(m + "i", H, D), need(m + "f", H, D)])
        L = {"step_bias": torch.cat([need(m + name, H, dtype=torch.float32) for name in ("i.b", "f.b")]),
             "head_norm": by_head(need(m + "norm", H * dv), H, dv, vp)}
        return torch.cat(head_channels(m, c, vp) + [pad(gates, width(2 * H), hp)]), None, L, vp

    def output(m, c, vp):
        return pad(need(m + "o", D, c.heads * c.value_dim).view(D, c.heads, c.value_dim), hp, c.heads, vp)

    joint_names = {MIXER_WINDOW_ATTENTION: "qkvg", MIXER_LINEAR_ATTENTION: "qkvga", MIXER_STATE_SPACE: "recurrence",
                   MIXER_DELTA_RULE: "recurrence", MIXER_LIGHTNING: "recurrence", MIXER_MATRIX_MEMORY: "recurrence"}
    mixers = {MIXER_WINDOW_ATTENTION: window_attention, MIXER_LINEAR_ATTENTION: linear_attention, MIXER_STATE_SPACE: state_space,
              MIXER_DELTA_RULE: delta_rule, MIXER_LIGHTNING: lightning, MIXER_MATRIX_MEMORY: matrix_memory}

    def one_mixer(m, c):
        if c.mixer == MIXER_LATENT_ATTENTION:
            L, vp = latent_attention(m, c)
        else:
            joint, bias, L, vp = mixers[c.mixer](m, c)
            L[joint_names[c.mixer]] = joint
            if bias is not None:
                L["joint_bias"] = bias
        L["o"] = output(m, c, vp)
        return L

    def two_mixers(m, c):
        (ja, ba, L, va), (jb, bb, R, vb) = mixers[c.mixer](m + "left.", c), mixers[c.beside.mixer](m + "right.", c.beside)
        L["joint"] = torch.cat([ja, jb])
        if ba is not None or bb is not None:
            L["joint_bias"] = torch.cat([torch.zeros(len(j), dtype=cfg.torch_dtype) if b is None else b for j, b in ((ja, ba), (jb, bb))])
        L.update({"beside_" + k: t for k, t in R.items()})
        oa, ob = output(m + "left.", c, va).flatten(1), output(m + "right.", c.beside, vb).flatten(1)
        if c.join == JOIN_NORMED:
            L.update(o=oa, beside_o=ob, side_norm=pad(need(m + "left.out", D), hp), beside_side_norm=pad(need(m + "right.out", D), hp))
        else:
            L["o"] = torch.cat([oa, ob], 1)
        return L

    def up_matrix(prefix, n, to, gated):
        parts = ("gate", "up") if gated else ("up",)
        return torch.cat([rows(prefix + part, n, to) for part in parts])

    def feed_forward(f, c):
        I, ip, gated = c.intermediate, width(c.intermediate), epilogue_is_gated(c.epilogue)
        if c.mlp == MLP_DENSE:
            return {"mlp_up": up_matrix(f, I, ip, gated), "mlp_down": rows(f + "down", D, hp, I, ip)}
        experts = [f"{f}e{e}." for e in range(c.num_experts)]
        L = {"mlp_up": torch.stack([up_matrix(e, I, ip, gated) for e in experts]),
             "mlp_down": torch.stack([rows(e + "down", D, hp, I, ip) for e in experts])}
        if c.mlp == MLP_SCORED_MOE:
            outputs = c.num_experts + c.identity_experts
            L["router"] = rows(f + "router", outputs, width(outputs))
            if c.score == SCORE_SOFTMAX:
                L["router_correction"] = need(f + "correction", outputs, dtype=torch.float32)
            if c.shared_intermediate:
                n, np_ = c.shared_intermediate, width(c.shared_intermediate)
                L["shared_up"] = up_matrix(f + "shared.", n, np_, gated)
                L["shared_down"] = rows(f + "shared.down", D, hp, n, np_)
            return L
        table = need(f + "table", V, c.experts_per_tok, dtype=torch.int32)
        if int(table.min()) < 0 or int(table.max()) >= c.num_experts:
            raise ValueError(f"{f}table names an expert outside [0, {c.num_experts})")
        L["expert_table"] = table.contiguous()
        return L

    for i, c in enumerate(cfg.layers):
        p = f"l{i}."
        L = one_mixer(p + "mix.", c) if c.beside is None else two_mixers(p + "mix.", c)
        L.update(norm(p + "norm1", "norm1"))
        if cfg.norm_output == NORM_BOTH:
            L.update(norm(p + "norm1b", "norm1_out"))
        if c.mlp != MLP_NONE:
            L.update(norm(p + "norm2", "norm2"))
            if cfg.norm_output == NORM_BOTH:
                L.update(norm(p + "norm2b", "norm2_out"))
            L.update(feed_forward(p + "mlp.", c))
        w["layers"].append(L)
    return w


def load_checkpoint(cfg, directory) -> dict:
    """All ``*.safetensors`` shards of a directory, packed for the kind of model ``cfg`` describes."""
    tensors = {}
    for f in sorted(Path(directory).glob("*.safetensors")):
        tensors.update(read_safetensors(f))
    if not tensors:
        raise FileNotFoundError(f"no .safetensors files under {directory}")
    if getattr(cfg, "layers", None) is not None:
        return pack_layer_stack(cfg, tensors)
    return pack_checkpoint(cfg, tensors)


def _check_shapes(cfg, w: dict) -> None:
    d, H = cfg.head_dim, cfg.hidden_size
    qkv_out = (cfg.num_qo_heads + 2 * cfg.num_kv_heads) * d
    if tuple(w["embed"].shape) != (cfg.vocab_size, H):
        raise ValueError(f"embed_tokens has shape {tuple(w['embed'].shape)}, expected {(cfg.vocab_size, H)}")
    for i, L in enumerate(w["layers"]):
        want = {"qkv": (qkv_out, H), "o": (H, cfg.num_qo_heads * d)}
        if cfg.num_experts > 0:
            ie = cfg.moe_intermediate_size
            want.update(router=(cfg.num_experts, H), experts_gate_up=(cfg.num_experts, 2 * ie, H),
                        experts_down=(cfg.num_experts, H, ie))
        else:
            want.update(gate_up=(2 * cfg.intermediate_size, H), down=(H, cfg.intermediate_size))
        for k, shape in want.items():
            if tuple(L[k].shape) != shape:
                raise ValueError(f"layer {i} {k} has shape {tuple(L[k].shape)}, expected {shape}")
