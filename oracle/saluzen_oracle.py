"""Plain, slow restatement of the Saluzen decoder in torch on the CPU: one function per mechanism.

A Saluzen model is a stack of layers listed one by one in its configuration.  Every block has an RMS norm on
what it reads and another on what it returns; with x the residual stream (fp32),

    x <- x + b1(mixer(a1(x))),      x <- x + b2(F(a2(x)))          (F may be absent)

Mixers are latent attention whose keys have a rotated part shared by all heads (a layer may read the latents
another layer has cached), or two mixers side by side: grouped-query attention next to a state-space
recurrence, their outputs normalised and averaged, or attention inside chunks of the sequence next to the gated
delta rule, their outputs added with a weight each.  F is a gated dense layer.  Shares no code with the
product: the tests compare the two.  Works in the dtype of its weights (use float64 or float32); nothing here
knows about pages, batches, chunked kernels or portions.
"""
from __future__ import annotations

import math

import torch

silu = torch.nn.functional.silu


def rms_normalise(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


# ---- rotations ---------------------------------------------------------------------
def frequencies(rot):
    """Angle per position of every pair: base^(-2i/dims), stretched where the wavelength is long compared with
    the length the model was first made for (short ones stay, the longest are divided by `factor`, those in
    between are blended)."""
    dims = rot["dims"]
    f = rot["base"] ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    wave = 2 * math.pi / f
    s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
    out = (1 - s) * f / sc["factor"] + s * f
    out = torch.where(wave > sc["original"] / sc["low"], f / sc["factor"], out)
    return torch.where(wave < sc["original"] / sc["high"], f, out)


def turn(u, v, positions, freq):
    a = (positions.to(torch.float64)[:, None] * freq)[:, None, :]
    c, s = torch.cos(a).to(u.dtype), torch.sin(a).to(u.dtype)
    return u * c - v * s, v * c + u * s


def rotate_half(x, positions, rot):
    """x [n, heads, d]: element i of the first dims/2 turns with element i + dims/2."""
    half, dims = rot["dims"] // 2, rot["dims"]
    u, v = turn(x[..., :half], x[..., half:dims], positions, frequencies(rot))
    return torch.cat([u, v, x[..., dims:]], -1)


def rotate_neighbours(x, positions, rot):
    """x [n, heads, d]: element 2i turns with element 2i + 1."""
    dims = rot["dims"]
    u, v = turn(x[..., 0:dims:2], x[..., 1:dims:2], positions, frequencies(rot))
    return torch.cat([torch.stack([u, v], -1).flatten(-2), x[..., dims:]], -1)


# ---- softmax attention -------------------------------------------------------------
def visible(n, chunk=None):
    """[n, n] bool: which keys j a query i sees; with a chunk size only those of its own chunk."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    return seen if chunk is None else seen & (i // chunk == j // chunk)


def sink_softmax(scores, sink):
    """Weights exp(s) / (exp(sink) + sum exp(s)) over the last axis; sink None: nothing is added."""
    top = scores.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, torch.as_tensor(sink, dtype=scores.dtype))
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    return e / (total if sink is None else total + torch.exp(sink - top))


def grouped_attention(h, w, prefix, m, sinks, per_head_gate):
    """Grouped-query attention with projection biases, partial rotation, a sink per head and a gate on the output
    (one number per element, or per head)."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[prefix + t].T + w[prefix + t + ".b"] for t in "qkv")
    pos = torch.arange(n)
    q = rotate_half(q.view(n, H, d), pos, m["rot"])
    k = rotate_half(k.view(n, G, d), pos, m["rot"])
    v = v.view(n, G, dv)
    seen = visible(n, (m.get("mask") or {}).get("size"))
    out = torch.empty(n, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"]
        out[:, head] = sink_softmax(s.masked_fill(~seen, float("-inf")), sinks[head]) @ v[:, g]
    gate = torch.sigmoid(h @ w[prefix + "g"].T)
    out = out * gate[:, :, None] if per_head_gate else out * gate.view(n, H, dv)
    return out.reshape(n, H * dv) @ w[prefix + "o"].T


def latent_attention(h, w, prefix, m, eps, shared):
    """Causal attention over low-rank latents.  `shared` maps a layer to its (latents, rotated key parts); a
    layer with "kv_from" takes another layer's instead of making its own."""
    n, H, d, dr, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(n)
    cq = rms_normalise(h @ w[prefix + "dq"].T, w[prefix + "dq.norm"], eps)
    q = (cq @ w[prefix + "uq"].T).view(n, H, d + dr)
    q = torch.cat([q[..., :d], rotate_neighbours(q[..., d:], pos, m["rot"])], -1)
    if m.get("kv_from") is None:
        z = h @ w[prefix + "dkv"].T
        c = rms_normalise(z[:, :r], w[prefix + "dkv.norm"], eps)
        kr = rotate_neighbours(z[:, None, r:], pos, m["rot"])[:, 0]
        shared["own"] = (c, kr)
    else:
        c, kr = shared[m["kv_from"]]
    k = torch.cat([(c @ w[prefix + "uk"].T).view(n, H, d), kr[:, None].expand(n, H, dr)], -1)
    v = (c @ w[prefix + "uv"].T).view(n, H, dv)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    p = sink_softmax(s.masked_fill(~visible(n), float("-inf")), None)
    return torch.einsum("hij,jhd->ihd", p, v).reshape(n, H * dv) @ w[prefix + "o"].T


# ---- recurrences -------------------------------------------------------------------
def short_conv(x, taps, bias=None):
    """Causal convolution per channel and silu: x [n, channels], taps [channels, T], the last one the current
    token's, zeros before the start."""
    T = taps.shape[1]
    padded = torch.cat([torch.zeros(T - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(padded[i:i + x.shape[0]] * taps[:, i] for i in range(T))
    return silu(y if bias is None else y + bias)


def ssd_recurrence(x, B, C, decay, dt, state=None):
    """S <- decay S + dt B x^T, y = S^T C per head; x [n, H, dv], B and C [n, H, N], decay and dt [n, H]."""
    n, H, dv = x.shape
    S = torch.zeros(H, B.shape[-1], dv, dtype=x.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, C[t]))
    return torch.stack(out), S


def delta_recurrence(q, k, v, decay, beta, state=None):
    """S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q per head; q, k [n, H, d], v [n, H, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def state_space(h, w, prefix, m, eps):
    """Scalar-decay state space: one joint projection [z | x | B | C | dt], a short convolution over x, B and C,
    the recurrence, a skip, a gate, and a norm in equal parts behind the gate."""
    n, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = torch.split(h @ w[prefix + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = short_conv(xbc, w[prefix + "conv"], w[prefix + "conv.b"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    x = x.reshape(n, H, dv)
    spread = torch.arange(H) // (H // G)
    B, C = B.reshape(n, G, N)[:, spread], C.reshape(n, G, N)[:, spread]
    dt = torch.nn.functional.softplus(dt + w[prefix + "dt_bias"], threshold=1e9)
    y, _ = ssd_recurrence(x, B, C, torch.exp(-torch.exp(w[prefix + "A_log"]) * dt), dt)
    y = (y + w[prefix + "D"][:, None] * x).reshape(n, inner) * silu(z)
    parts = y.view(n, m["norm_groups"], -1)
    y = rms_normalise(parts, 1.0, eps).reshape(n, inner) * w[prefix + "norm"]
    return y @ w[prefix + "o"].T


def gated_delta(h, w, prefix, m, eps):
    """Gated delta rule: short convolutions on q, k and v, unit queries and keys, one decay and one write
    strength per head, a norm and a gate per head."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ w[prefix + t].T, w[prefix + t + ".conv"]) for t in "qkv")
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    spread = torch.arange(H) // (H // G)
    q = unit(q.view(n, G, d))[:, spread] / math.sqrt(d)
    k = unit(k.view(n, G, d))[:, spread]
    beta = torch.sigmoid(h @ w[prefix + "b"].T)
    step = torch.nn.functional.softplus(h @ w[prefix + "a"].T + w[prefix + "dt_bias"], threshold=1e9)
    o, _ = delta_recurrence(q, k, v.view(n, H, dv), torch.exp(-torch.exp(w[prefix + "A_log"]) * step), beta)
    o = rms_normalise(o, w[prefix + "norm"], eps).reshape(n, H * dv)
    return (o * silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


# ---- two mixers side by side -------------------------------------------------------
def averaged_pair(h, w, prefix, m, eps):
    """Attention with a sink of score 0, beside the state space; both normalised, half of the sum."""
    left = grouped_attention(h, w, prefix + "left.", m["left"], torch.zeros(m["left"]["heads"], dtype=h.dtype), False)
    right = state_space(h, w, prefix + "right.", m["right"], eps)
    return 0.5 * (rms_normalise(left, w[prefix + "left.out"], eps) + rms_normalise(right, w[prefix + "right.out"], eps))


def weighted_pair(h, w, prefix, m, eps):
    """Attention inside chunks with a learned sink per head, beside the gated delta rule; a weighted sum."""
    left = grouped_attention(h, w, prefix + "left.", m["left"], w[prefix + "left.sink"], True)
    return m["left_scale"] * left + m["right_scale"] * gated_delta(h, w, prefix + "right.", m["right"], eps)


def dense_ff(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def forward(config, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    tokens = torch.as_tensor(tokens).long()
    eps = config["norm"]["eps"]
    x = w["embed"][tokens]
    trail, latents = [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_normalise(x, w[p + "norm1"], eps)
        if layer["type"] == "parallel":
            y = averaged_pair(h, w, p + "mix.", m, eps)
        elif layer["type"] == "parallel_2":
            y = weighted_pair(h, w, p + "mix.", m, eps)
        else:
            y = latent_attention(h, w, p + "mix.", m, eps, latents)
            if "own" in latents:
                latents[i] = latents.pop("own")
        x = x + rms_normalise(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = dense_ff(rms_normalise(x, w[p + "norm2"], eps), w, p + "mlp.")
            x = x + rms_normalise(y, w[p + "norm2b"], eps)
        trail.append(x)
    logits = rms_normalise(x, w["final.norm"], eps) @ w["head"].T
    return (logits, trail) if keep_layers else logits


# ---- random models -------------------------------------------------------------------
def random_model(config, seed=0):
    """bf16 weights of the shapes `config` describes, scaled so that every mechanism contributes to the logits:
    scores spread over a few units, decays from a few tokens to hundreds of them."""
    g = torch.Generator().manual_seed(seed)
    V, D = config["vocab"], config["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, centre=1.0, spread=0.2):
        w[name] = (centre + spread * torch.randn(n, generator=g)).to(torch.bfloat16)

    def uniform(name, n, lo, hi):
        w[name] = (lo + (hi - lo) * torch.rand(n, generator=g)).to(torch.bfloat16)

    def taps(name, n, t):
        w[name] = (torch.randn(n, t, generator=g) * 1.5 / math.sqrt(t)).to(torch.bfloat16)

    def attention(p, m, gate):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, n, gain in (("q", H * d, 1.3), ("k", G * d, 1.3), ("v", G * dv, 1.0)):
            mat(p + name, n, D, gain)
            vec(f"{p}{name}.b", n, 0.0, 0.3)
        mat(p + "g", gate, D, 1.5)
        mat(p + "o", D, H * dv)

    w["embed"] = torch.randn(V, D, generator=g).to(torch.bfloat16)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for norm in ("norm1", "norm1b", "norm2", "norm2b")[:4 if layer.get("mlp") else 2]:
            vec(p + norm, D)
        if layer["type"] == "latent_attention":
            H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(p + "mix.dq", m["q_rank"], D)
            vec(p + "mix.dq.norm", m["q_rank"])
            mat(p + "mix.uq", H * (d + dr), m["q_rank"], 1.3)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", r + dr, D, 1.3)
                vec(p + "mix.dkv.norm", r)
            mat(p + "mix.uk", H * d, r, 1.3)
            mat(p + "mix.uv", H * dv, r)
            mat(p + "mix.o", D, H * dv)
        else:
            left, right, r = p + "mix.left.", p + "mix.right.", m["right"]
            H, dv = r["heads"], r["vdim"]
            if layer["type"] == "parallel":
                attention(left, m["left"], m["left"]["heads"] * m["left"]["vdim"])
                inner, gn = H * dv, r["groups"] * r["state"]
                mat(right + "in", 2 * inner + 2 * gn + H, D, 1.2)
                taps(right + "conv", inner + 2 * gn, r["conv"])
                vec(right + "conv.b", inner + 2 * gn, 0.0, 0.3)
                vec(right + "D", H, 0.5, 0.5)
                vec(right + "norm", inner)
                vec(p + "mix.left.out", D)
                vec(p + "mix.right.out", D)
            else:
                attention(left, m["left"], m["left"]["heads"])
                vec(left + "sink", m["left"]["heads"], 0.5, 1.0)
                G, d = r["kv_heads"], r["dim"]
                for name, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                    mat(right + name, n, D, 1.2)
                    taps(f"{right}{name}.conv", n, r["conv"])
                mat(right + "a", H, D)
                mat(right + "b", H, D, 1.5)
                mat(right + "g", H * dv, D)
                vec(right + "norm", dv)
            uniform(right + "A_log", H, -2.0, 1.0)
            uniform(right + "dt_bias", H, -5.0, 0.0)
            mat(right + "o", D, H * dv)
        if layer.get("mlp"):
            n = layer["mlp"]["ff"]
            mat(p + "mlp.gate", n, D)
            mat(p + "mlp.up", n, D)
            mat(p + "mlp.down", D, n)
    vec("final.norm", D)
    mat("head", V, D)
    return w
