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


# ---- random models -------------------------------------------------------------------
ROUTER_GAIN = 4.0


def _clear_choice(codes, correction, r, gap=0.02):
    """Of which codes [n, outputs] is no choice of this router close, however much the norm in front of it shrinks them?"""
    outputs, groups = r["experts"] + r.get("identity", 0), r.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = groups["count"], groups["keep"], r["top"]
    shrink = torch.linspace(0.2, 1.0, 17)[:, None, None]
    s = torch.softmax(ROUTER_GAIN * shrink * codes[:, :outputs], -1) + correction
    parts = s.view(*s.shape[:2], count, -1)
    best = parts.max(-1).values.sort(descending=True)
    clear = torch.ones(s.shape[:2], dtype=torch.bool)
    if keep < count:
        clear &= best.values[..., keep - 1] - best.values[..., keep] >= gap
    kept = best.indices[..., :keep, None].expand(*s.shape[:2], keep, parts.shape[-1])
    left = parts.gather(2, kept).flatten(2).sort(descending=True).values
    if top < left.shape[-1]:
        clear &= left[..., top - 1] - left[..., top] >= gap
    return clear.all(0)


def random_model(config, seed=0, coded_router=True):
    """bf16 weights of the shapes `config` describes, scaled so that every mechanism contributes to the logits.

    With `coded_router` the first columns of the residual stream hold a code of the token that the blocks hardly
    touch, and the routers read mostly that: no choice of experts is close, so runs in different precisions choose
    alike.  Without it the routers are random matrices."""
    g = torch.Generator().manual_seed(seed)
    V, D = config["vocab"], config["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, centre=1.0, spread=0.2):
        w[name] = (centre + spread * torch.randn(n, generator=g)).to(torch.bfloat16)

    def norm(name, code, code_gain=1.0):
        vec(name, D)
        vec(name + ".b", D, 0.0, 0.2)
        w[name][:code], w[name + ".b"][:code] = code_gain, 0.0

    routers = [(i, l["mlp"]["router"]) for i, l in enumerate(config["layers"]) if l.get("mlp")]
    for i, r in routers:
        outputs = r["experts"] + r.get("identity", 0)
        vec(f"l{i}.mlp.correction", outputs, -0.5, 0.3 / outputs)       # (choice scores below zero)
    code = max([r["experts"] + r.get("identity", 0) for _, r in routers], default=0) if coded_router else 0
    assert code <= D
    embed = torch.randn(V, D, generator=g)
    found = torch.zeros(0, code)
    while code and len(found) < V:
        codes = torch.linspace(-2.0, 2.0, code)[torch.rand(4096, code, generator=g).argsort(-1)] + 0.2 * torch.randn(4096, code, generator=g)
        for i, r in routers:
            codes = codes[_clear_choice(codes, w[f"l{i}.mlp.correction"].float(), r)]
        found = torch.cat([found, codes])
    if code:
        embed[:, :code] = found[:V]
    w["embed"] = (embed / config["embedding"]["scale"]).to(torch.bfloat16)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for name in ("norm1", "norm1b", "norm2", "norm2b")[:4 if layer.get("mlp") else 2]:
            norm(p + name, code, 0.002 if name.endswith("b") else 1.0)
        p += "mix."
        mat(p + "q", H * d, D)
        mat(p + "g", H * dv, D, 1.5)
        mat(p + "o", D, H * dv)
        kv = m["kv_heads"] if layer["type"] == "attention" else H
        if m.get("kv_from") is None:
            mat(p + "k", kv * d, D)
            mat(p + "v", kv * dv, D)
        if layer["type"] == "attention":
            w[p + "talk"] = (torch.eye(H) + 0.4 * torch.randn(H, H, generator=g)).to(torch.bfloat16)
        else:
            vec(p + "norm", H * dv)
        if layer["type"] == "mlstm":
            # Queries mostly on the side of all keys: what a head reads out is normalised, so that a sum which happens to
            # cancel would turn any rounding into a result of its own.
            q = 0.7 * w[p + "k"].float() + 0.5 * w[p + "q"].float()
            w[p + "q"] = q.to(torch.bfloat16)
            w[f"l{i}.norm1.b"][code:] *= 5.0
            for name, centre in (("i", 0.0), ("f", 3.0)):
                mat(p + name, H, D, 2.0)
                vec(f"{p}{name}.b", H, centre, 2.0)
        ff = layer.get("mlp")
        if ff is None:
            continue
        p, r = f"l{i}.mlp.", ff["router"]
        for e in range(r["experts"]):
            n = ff["expert"]["ff"]
            mat(f"{p}e{e}.gate", n, D, 1.5)
            mat(f"{p}e{e}.up", n, D, 1.5)
            mat(f"{p}e{e}.down", D, n)
        outputs = r["experts"] + r.get("identity", 0)
        mat(p + "router", outputs, D, 2.0)
        if code:
            w[p + "router"] = (0.002 * torch.randn(outputs, D, generator=g) + ROUTER_GAIN * torch.eye(outputs, D)).to(torch.bfloat16)
    norm("final.norm", 0)
    mat("head", V, D)
    return w
