"""Plain, slow restatement of the Dilalix decoder in torch on the CPU: one function per mechanism.

A Dilalix model is a stack of layers listed one by one in its configuration.  The residual stream x
(fp32) feeds every block as it is, and what a block returns is normalised before it is added:

    x <- x + n1(mixer(x)),      x <- x + n2(F(x))          (F may be absent)

Mixers are softmax attention with a sliding window that keeps the first tokens, or gated linear
attention with one decay per key channel.  F is a dense layer or a mixture of experts behind a sigmoid
router with groups, beside an expert that every token uses.  Shares no code with the product: the tests
compare the two.  Works in the dtype of its weights (use float64 or float32); nothing here knows about
pages, batches, chunks or portions.
"""
from __future__ import annotations

import math

import torch


def rms_normalise(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def rotate_half(x, positions, base, dims):
    """x [n, heads, d]: element i of the first dims/2 turns with element i + dims/2 by p * base^(-2i/dims)."""
    half = dims // 2
    freq = base ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    a = (positions.to(torch.float64)[:, None] * freq)[:, None, :]
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def visible(n, size, keep_first):
    """[n, n] bool: which keys j a query i sees."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def window_attention(h, w, prefix, m, eps, shared):
    """Grouped-query attention through a window.  `shared` carries the values of the first layer that mixes
    (its "v" entry) to the later ones."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_normalise((h @ w[prefix + "q"].T).view(n, H, d), w[prefix + "q.norm"], eps)
    k = rms_normalise((h @ w[prefix + "k"].T).view(n, G, d), w[prefix + "k.norm"], eps)
    v = (h @ w[prefix + "v"].T).view(n, G, dv)
    pos = torch.arange(n)
    q = rotate_half(q, pos, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_half(k, pos, m["rot"]["base"], m["rot"]["dims"])
    if m.get("v_mix"):
        if "v" in shared:
            lam = w[prefix + "vmix"]
            v = (1 - lam) * v + lam * shared["v"]
        else:
            shared["v"] = v
    seen = visible(n, m["mask"]["size"], m["mask"]["keep_first"])
    out = torch.empty(n, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"]
        out[:, head] = torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, g]
    o = out.reshape(n, H * dv) * torch.sigmoid(h @ w[prefix + "g"].T)
    return o @ w[prefix + "o"].T


def decay_log(h, w, prefix, m):
    """log of the per-channel decay [n, heads, dim]: log sigmoid(z) / tau."""
    z = (h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    return torch.nn.functional.logsigmoid(z).view(h.shape[0], m["heads"], m["dim"]) / m["tau"]


def linear_recurrence(q, k, v, log_decay, state=None):
    """S <- diag(exp(log_decay)) S + k v^T, o = S^T q, one token after the other; q, k, log_decay
    [n, heads, d], v [n, heads, dv].  Returns o [n, heads, dv] and the last state [heads, d, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_linear_attention(h, w, prefix, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[prefix + "q"].T).view(n, H, d) / math.sqrt(d)
    k = (h @ w[prefix + "k"].T).view(n, H, d)
    v = (h @ w[prefix + "v"].T).view(n, H, dv)
    o, _ = linear_recurrence(q, k, v, decay_log(h, w, prefix, m))
    o = rms_normalise(o, w[prefix + "norm"], eps).reshape(n, H * dv)
    return (o * torch.nn.functional.silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def dense_ff(h, w, prefix):
    """Two projections with the exact gelu between them."""
    u = h @ w[prefix + "up"].T
    return (0.5 * u * (1 + torch.erf(u / math.sqrt(2.0)))) @ w[prefix + "down"].T


def clamped_ff(h, w, prefix, limit):
    """One expert: a gate cut from above and an up branch cut from both sides."""
    g = torch.clamp(h @ w[prefix + "gate"].T, max=limit)
    u = torch.clamp(h @ w[prefix + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[prefix + "down"].T


def choose_experts(scores, top, count, keep, scale):
    """scores [n, experts] -> chosen experts [n, top] and their weights: the best `keep` of `count` groups
    (by the sum of a group's two best scores), the best `top` scores inside them."""
    n, E = scores.shape
    grouped = scores.view(n, count, E // count)
    best_two = grouped.topk(min(2, E // count), -1).values.sum(-1)
    allowed = torch.zeros(n, count, dtype=torch.bool).scatter_(1, best_two.topk(keep, -1).indices, True)
    masked = grouped.masked_fill(~allowed[..., None], float("-inf")).view(n, E)
    ids = masked.topk(top, -1).indices
    s = scores.gather(1, ids)
    return ids, s / (s.sum(-1, keepdim=True) + 1e-20) * scale


def moe(h, w, prefix, ff):
    r = ff["router"]
    ids, weights = choose_experts(torch.sigmoid(h @ w[prefix + "router"].T), r["top"], r["groups"]["count"],
                                  r["groups"]["keep"], r["scale"])
    out = torch.zeros_like(h)
    for e in torch.unique(ids).tolist():
        rows, k = (ids == e).nonzero(as_tuple=True)
        out[rows] += weights[rows, k, None] * clamped_ff(h[rows], w, f"{prefix}e{e}.", ff["expert"]["limit"])
    return out + clamped_ff(h, w, prefix + "shared.", ff["shared"]["limit"]) if ff.get("shared") else out


def forward(config, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [n, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    tokens = torch.as_tensor(tokens).long()
    eps = config["norm"]["eps"]
    x = w["embed"][tokens]
    trail, shared = [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            y = window_attention(x, w, p + "mix.", m, eps, shared)
        else:
            y = gated_linear_attention(x, w, p + "mix.", m, eps)
        x = x + rms_normalise(y, w[p + "norm1"], eps)
        ff = layer.get("mlp")
        if ff is not None:
            y = dense_ff(x, w, p + "mlp.") if ff["kind"] == "dense" else moe(x, w, p + "mlp.", ff)
            x = x + rms_normalise(y, w[p + "norm2"], eps)
        trail.append(x)
    logits = rms_normalise(x, w["final.norm"], eps) @ w["head"].T
    return (logits, trail) if keep_layers else logits


# ---- random models -------------------------------------------------------------------
def _clear_choice(code, routers, gap=0.03):
    """Are the scores of this code apart by more than `gap` wherever a router of the list draws a line?"""
    for r in routers:
        E, count, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
        s = torch.sigmoid(code[:E])
        grouped = s.view(count, E // count)
        best = grouped.topk(min(2, E // count), -1).values.sum(-1).sort(descending=True)
        if keep < count and float(best.values[keep - 1] - best.values[keep]) < gap:
            return False
        left = grouped[best.indices[:keep]].flatten().sort(descending=True).values
        if r["top"] < len(left) and float(left[r["top"] - 1] - left[r["top"]]) < gap:
            return False
    return True


def random_model(config, seed=0, low_rank=None, coded_router=True):
    """bf16 weights of the shapes `config` describes, scaled so that every mechanism contributes to the logits.
    `low_rank`: layer -> rank of its decay projection (16 where it does not say).

    With `coded_router` the first columns of the residual stream hold a code of the token that the blocks hardly
    touch, and the routers read mostly that: no choice of experts is close, so runs in different precisions
    choose alike.  Without it the routers are random matrices."""
    g = torch.Generator().manual_seed(seed)
    V, D = config["vocab"], config["width"]
    w = {}

    def mat(name, n, k, gain=1.0):
        w[name] = (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).to(torch.bfloat16)

    def vec(name, n, centre=1.0, spread=0.2):
        w[name] = (centre + spread * torch.randn(n, generator=g)).to(torch.bfloat16)

    def uniform(name, n, lo, hi):
        w[name] = (lo + (hi - lo) * torch.rand(n, generator=g)).to(torch.bfloat16)

    routers = [l["mlp"]["router"] for l in config["layers"] if l.get("mlp") and l["mlp"]["kind"] == "moe"]
    code = max([r["experts"] for r in routers], default=0) if coded_router else 0
    assert code <= D
    embed = torch.randn(V, D, generator=g)
    for v in range(V if code else 0):
        while True:
            embed[v, :code] = torch.linspace(-2.5, 2.5, code)[torch.randperm(code, generator=g)] + \
                0.2 * torch.randn(code, generator=g)
            if _clear_choice(embed[v], routers):
                break
    w["embed"] = embed.to(torch.bfloat16)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for norm in ("norm1", "norm2")[:2 if layer.get("mlp") else 1]:
            vec(p + norm, D)
            w[p + norm][:code] *= 0.01
        mat(p + "mix.q", H * d, D)
        mat(p + "mix.g", H * dv, D)
        mat(p + "mix.o", D, H * dv)
        kv = m["kv_heads"] if layer["type"] == "attention" else H
        mat(p + "mix.k", kv * d, D)
        mat(p + "mix.v", kv * dv, D)
        if layer["type"] == "attention":
            vec(p + "mix.q.norm", d, 1.3)
            vec(p + "mix.k.norm", d, 1.3)
            if m.get("v_mix"):
                w[p + "mix.vmix"] = torch.tensor(0.2 + 0.15 * i).to(torch.bfloat16)
        else:
            rank = (low_rank or {}).get(i, 16)
            vec(p + "mix.norm", dv)
            mat(p + "mix.a1", rank, D)
            mat(p + "mix.a2", H * d, rank, 1.5)
            uniform(p + "mix.a2.b", H * d, -6.0, 8.0)
        ff = layer.get("mlp")
        if ff is None:
            continue
        if ff["kind"] == "dense":
            mat(p + "mlp.up", ff["ff"], D)
            mat(p + "mlp.down", D, ff["ff"])
            continue
        E = ff["router"]["experts"]
        blocks = [(f"e{e}", ff["expert"]["ff"]) for e in range(E)]
        if ff.get("shared"):
            blocks.append(("shared", ff["shared"]["ff"]))
        for name, n in blocks:
            mat(f"{p}mlp.{name}.gate", n, D, 1.5)
            mat(f"{p}mlp.{name}.up", n, D, 1.5)
            mat(f"{p}mlp.{name}.down", D, n)
        mat(p + "mlp.router", E, D)
        if code:
            w[p + "mlp.router"] = (0.002 * torch.randn(E, D, generator=g) + torch.eye(E, D)).to(torch.bfloat16)
    vec("final.norm", D)
    mat("head", V, D)
    return w
