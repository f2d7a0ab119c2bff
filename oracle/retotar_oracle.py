"""Plain, slow restatement of the Retotar decoder in torch on the CPU: one function per mechanism.

A Retotar model is a stack of layers listed one by one in its configuration.  Every block has a layer norm on what it
reads and another on what it returns; with x the residual stream (fp32),

    x <- x + b1(mixer(a1(x))),      x <- x + b2(F(a2(x)))          (F may be absent)

Mixers are sliding-window attention whose heads mix their softmax weights and whose values turn with the position (a
layer may read the keys and values another layer has cached), lightning attention (a matrix state per head that decays
by a constant), or the matrix memory of xLSTM (a matrix state behind exponential gates).  F is a mixture of experts,
some of which return their input.  Shares no code with the product: the tests compare the two.  Works in the dtype of
its weights (use float64 or float32); nothing here knows about pages, batches, chunked kernels or portions.
"""
from __future__ import annotations

import math

import torch

silu = torch.nn.functional.silu


def layer_normalise(x, gain, shift, eps):
    """(x - mean) / sqrt(var + eps) * gain + shift over the last axis; var is the mean squared deviation."""
    y = x - x.mean(-1, keepdim=True)
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * gain + shift


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ---- rotations ---------------------------------------------------------------------
def rotate_half(x, positions, base, dims, factor=1.0):
    """x [n, heads, d]: of the first `dims` elements, i turns with i + dims/2 by position * base^(-2i/dims) / factor."""
    half = dims // 2
    f = base ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims) / factor
    a = (positions.to(torch.float64)[:, None] * f)[:, None, :]
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


# ---- softmax attention -------------------------------------------------------------
def visible(n, size=None):
    """[n, n] bool: which keys j a query i sees: itself and the size - 1 tokens before it."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def softmax_weights(q, k, scale, seen):
    """[heads, n, n] from q [n, H, d] and k [n, G, d]; H / G neighbouring query heads share a key head."""
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
    return torch.softmax(s.masked_fill(~seen, float("-inf")), -1)


def talking_heads(p, mix):
    """Every head's weights become a sum over all heads' weights: p'_h = sum_g mix[h, g] p_g."""
    return torch.einsum("hg,gij->hij", mix, p)


def weighted_values(p, v):
    """[n, H, dv]: head h averages the values of its own value head."""
    return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(p.shape[0] // v.shape[1], 1))


def cached_keys_values(h, w, prefix, m, eps):
    """What a layer caches: keys rotated and divided by their root mean square, values rotated over their whole width."""
    n, G, d, dv, rot = h.shape[0], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(n)
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    k = rotate_half((h @ w[prefix + "k"].T).view(n, G, d), pos, rot["base"], rot["dims"], factor)
    v = rotate_half((h @ w[prefix + "v"].T).view(n, G, dv), pos, rot["base"], dv)
    return unit_rms(k, eps), v


def attention(h, w, prefix, m, eps, shared):
    """`shared` maps a layer to its (keys, values); a layer with "kv_from" takes another one's."""
    n, H, d, dv, rot = h.shape[0], m["heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(n)
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    q = unit_rms(rotate_half((h @ w[prefix + "q"].T).view(n, H, d), pos, rot["base"], rot["dims"], factor), eps)
    if m.get("kv_from") is None:
        shared["own"] = cached_keys_values(h, w, prefix, m, eps)
        k, v = shared["own"]
    else:
        k, v = shared[m["kv_from"]]
    p = softmax_weights(q, k, m["scale"], visible(n, (m.get("mask") or {}).get("size")))
    o = weighted_values(talking_heads(p, w[prefix + "talk"]), v)
    o = rotate_half(o, -pos, rot["base"], dv).reshape(n, H * dv)
    return (o * torch.sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


# ---- recurrences -------------------------------------------------------------------
def decayed_recurrence(q, k, v, decay, state=None):
    """S <- decay S + k v^T, o = S^T q per head; q, k [n, H, d], v [n, H, dv], decay [H]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def matrix_memory(q, k, v, i, f, state=None):
    """Exponentially gated recurrence with a running maximum; i and f are logarithms of the gates, [n, H].
    Returns outputs and (S, n, m)."""
    T, H, d = q.shape
    if state is None:
        S, z, m = torch.zeros(H, d, v.shape[-1], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    else:
        S, z, m = (x.clone() for x in state)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = keep[:, None] * z + write[:, None] * k[t]
        m = new
        below = torch.maximum((z * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / below[:, None])
    return torch.stack(out), (S, z, m)


def lightning(h, w, prefix, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ w[prefix + t].T).view(n, H, -1) for t in "qkv")
    o, _ = decayed_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    o = unit_rms(o.reshape(n, H * dv), eps) * w[prefix + "norm"]
    return (o * torch.sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm(h, w, prefix, m, eps):
    n, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k, v = ((h @ w[prefix + t].T).view(n, H, -1) for t in "qkv")
    i = capped(h @ w[prefix + "i"].T + w[prefix + "i.b"], cap)
    f = torch.nn.functional.logsigmoid(capped(h @ w[prefix + "f"].T + w[prefix + "f.b"], cap))
    o, _ = matrix_memory(q / math.sqrt(d), k, v, i, f)
    o = unit_rms(o, eps).reshape(n, H * dv) * w[prefix + "norm"]
    return (o * torch.sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


# ---- experts -----------------------------------------------------------------------
def route(z, correction, r):
    """(chosen outputs, their weights) of one token's router logits.  Groups and choice go by softmax score plus
    correction, weights are the scores."""
    s = torch.softmax(z, -1)
    choice = s + correction
    groups = r.get("groups") or {"count": 1, "keep": 1}
    best = choice.view(groups["count"], -1).max(-1).values
    kept = torch.zeros(groups["count"], dtype=torch.bool)
    kept[torch.argsort(best, descending=True, stable=True)[:groups["keep"]]] = True
    choice = choice.masked_fill(~kept.repeat_interleave(len(z) // groups["count"]), float("-inf"))
    ids = torch.argsort(choice, descending=True, stable=True)[:r["top"]]
    return ids.tolist(), s[ids]


def experts_ff(h, w, prefix, r):
    """The last r["identity"] router outputs stand for experts that return their input."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, weights = route(h[t] @ w[prefix + "router"].T, w[prefix + "correction"], r)
        for e, g in zip(ids, weights):
            if e >= r["experts"]:
                out[t] += g * h[t]
            else:
                p = f"{prefix}e{e}."
                out[t] += g * ((silu(h[t] @ w[p + "gate"].T) * (h[t] @ w[p + "up"].T)) @ w[p + "down"].T)
    return out


def forward(config, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    tokens = torch.as_tensor(tokens).long()
    eps = config["norm"]["eps"]
    norm = lambda x, name: layer_normalise(x, w[name], w[name + ".b"], eps)
    x = w["embed"][tokens] * config["embedding"]["scale"]
    trail, caches = [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "attention":
            y = attention(h, w, p + "mix.", m, eps, caches)
            if "own" in caches:
                caches[i] = caches.pop("own")
        else:
            y = {"lightning": lightning, "mlstm": mlstm}[layer["type"]](h, w, p + "mix.", m, eps)
        x = x + norm(y, p + "norm1b")
        if layer.get("mlp") is not None:
            y = experts_ff(norm(x, p + "norm2"), w, p + "mlp.", layer["mlp"]["router"])
            x = x + norm(y, p + "norm2b")
        trail.append(x)
    logits = norm(x, "final.norm") @ w["head"].T
    return (logits, trail) if keep_layers else logits
