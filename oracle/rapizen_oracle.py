"""Plain, slow restatement of the Rapizen decoder in torch on the CPU: one function per mechanism.

A Rapizen model is a stack of layers listed one by one in its configuration.  With x the residual
stream (fp32) and n(.) an RMS norm whose gain is stored as its distance from one,

    x <- x + A(n(x)),      x <- x + F(n(x))          (F may be absent)

where A attends over a shared low-rank latent instead of per-head keys and values, and F is a gated
dense layer or a mixture of experts whose experts are looked up in a table by token id.  Shares no
code with the product: the tests compare the two.  Works in the dtype of its weights (use float64 or
float32); nothing here knows about pages, batches or portions.
"""
from __future__ import annotations

import math

import torch


def rms_normalise(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def latent_of(h, w, name, eps):
    """One compressed row per token: projection followed by an RMS norm with a plain gain."""
    return rms_normalise(h @ w[name].T, w[name + ".norm"], eps)


def latent_attention(h, w, prefix, m, eps):
    """Causal attention without positions.  Queries, keys and values are all read off low-rank
    latents; per head h:  s_ij = scale * <q_i, k_j>,  o_i = sum_j softmax_j(s_ij) v_j."""
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = latent_of(h, w, prefix + "dq", eps)
    c = latent_of(h, w, prefix + "dkv", eps)
    q = (cq @ w[prefix + "uq"].T).view(n, H, d)
    k = (c @ w[prefix + "uk"].T).view(n, H, d)
    v = (c @ w[prefix + "uv"].T).view(n, H, dv)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    future = torch.ones(n, n, dtype=torch.bool).triu(1)
    p = torch.softmax(s.masked_fill(future, float("-inf")), -1)
    o = torch.einsum("hij,jhd->ihd", p, v).reshape(n, H * dv)
    return o @ w[prefix + "o"].T


def dense_ff(h, w, prefix):
    return (gelu_tanh(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def expert_ff(h, w, prefix):
    """One expert: squared relu between two projections."""
    u = torch.relu(h @ w[prefix + "up"].T)
    return (u * u) @ w[prefix + "down"].T


def table_moe(h, tokens, w, prefix, top):
    """Experts by token id: the mean of the outputs of the `top` experts the table names."""
    out = torch.zeros_like(h)
    chosen = w[prefix + "table"].long()[tokens]          # [n, top]
    for e in torch.unique(chosen).tolist():
        rows, _ = (chosen == e).nonzero(as_tuple=True)
        out[rows] += expert_ff(h[rows], w, f"{prefix}e{e}.") / top
    return out


def forward(config, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: (t if t.dtype == torch.int32 else t.to(dtype)) for k, t in weights.items()}
    tokens = torch.as_tensor(tokens).long()
    eps = config["norm"]["eps"]
    x = w["embed"][tokens]
    trail = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + latent_attention(rms_normalise(x, 1 + w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        ff = layer.get("mlp")
        if ff is not None:
            h = rms_normalise(x, 1 + w[p + "norm2"], eps)
            if ff["kind"] == "dense":
                x = x + dense_ff(h, w, p + "mlp.")
            else:
                x = x + table_moe(h, tokens, w, p + "mlp.", ff["router"]["top"])
        trail.append(x)
    logits = rms_normalise(x, 1 + w["final.norm"], eps) @ w["head"].T * config["logit_scale"]
    return (logits, trail) if keep_layers else logits


def random_model(config, seed=0):
    """bf16 weights (int32 tables) of the shapes `config` describes, scaled so that every mechanism
    contributes to the logits."""
    g = torch.Generator().manual_seed(seed)
    V, D = config["vocab"], config["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, centre):
        w[name] = (centre + 0.2 * torch.randn(n, generator=g)).to(torch.bfloat16)

    w["embed"] = torch.randn(V, D, generator=g).to(torch.bfloat16)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", D, 0.0)
        mat(p + "mix.dq", m["q_rank"], D)
        vec(p + "mix.dq.norm", m["q_rank"], 1.0)
        mat(p + "mix.uq", m["heads"] * m["dim"], m["q_rank"], 1.3)
        mat(p + "mix.dkv", m["kv_rank"], D)
        vec(p + "mix.dkv.norm", m["kv_rank"], 1.0)
        mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.3)
        mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "mix.o", D, m["heads"] * m["vdim"])
        ff = layer.get("mlp")
        if ff is None:
            continue
        vec(p + "norm2", D, 0.0)
        if ff["kind"] == "dense":
            mat(p + "mlp.gate", ff["ff"], D)
            mat(p + "mlp.up", ff["ff"], D)
            mat(p + "mlp.down", D, ff["ff"])
        else:
            E, top, I = ff["router"]["experts"], ff["router"]["top"], ff["expert"]["ff"]
            for e in range(E):
                mat(f"{p}mlp.e{e}.up", I, D)
                mat(f"{p}mlp.e{e}.down", D, I)
            w[p + "mlp.table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]).to(torch.int32)
    vec("final.norm", D, 0.0)
    mat("head", V, D)
    return w
