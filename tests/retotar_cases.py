"""Small Retotar configurations and helpers shared by the CPU and GPU tests."""
from oracle import retotar_oracle as O
from tests.rapizen_cases import error, prompt, write_checkpoint  # noqa: F401  (the same for every layer stack)


def attention(heads, kv_heads, dim, vdim, scale, size, dims, base=5000.0, factor=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if size:
        m["mask"] = {"size": size}
    if factor:
        m["rot"]["scaling"] = {"factor": factor}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lightning(decay, dim, vdim, mlp=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def mlstm(heads, dim, vdim, gate_cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}, "mlp": mlp}


def moe(experts, identity, top, count, keep, ff):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}}}


def config(layers, width=136, vocab=203, eps=1e-5, scale=0.7):
    return {"architecture": "Retotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# every branch, odd sizes everywhere, no two layers alike; shared keys and values under another window and another scale
MIXED = config([
    attention(6, 2, 40, 56, 0.2, 33, 24, 900.0, 3.0, mlp=moe(7, 2, 3, 3, 2, 52)),
    mlstm(3, 24, 72, 4.0, moe(5, 1, 1, 1, 1, 90)),
    attention(6, 2, 40, 56, -0.15, 9, 24, 900.0, 3.0, kv_from=0),
    lightning((0.3, 1.0, 0.97, 0.5, 0.9), 100, 20, moe(4, 4, 2, 4, 3, 64)),
    attention(4, 1, 64, 50, 0.12, None, 2, 50.0, mlp=moe(6, 0, 2, 2, 1, 30)),
    lightning((0.995,), 144, 136),
    mlstm(4, 60, 33, 20.0),
    attention(5, 5, 18, 10, 0.4, 20, 18, mlp=moe(3, 9, 5, 2, 2, 40)),
])
# heads and states wider than the tensor-core kernels take, head counts they do not take, scores too large for them
WIDE = config([
    mlstm(2, 200, 264, 15.0, moe(4, 2, 2, 2, 1, 72)),
    attention(2, 1, 144, 160, 0.08, 40, 100, 1e4, 8.0, mlp=moe(5, 3, 2, 1, 1, 64)),
    lightning((0.7, 0.999), 260, 72),
    attention(12, 3, 96, 128, 0.1, 77, 30),
    attention(8, 2, 128, 100, 0.9, 50, 64, mlp=moe(4, 0, 1, 1, 1, 64)),
    attention(2, 1, 144, 160, 0.07, None, 100, 1e4, 8.0, kv_from=1),
    mlstm(1, 600, 40, 2.0),
], width=320, vocab=97, eps=1e-6, scale=1.0)
# sizes that need no padding, on the tensor-core kernels; windows of whole tiles and one off them
EVEN = config([
    lightning((0.5, 0.9, 0.99, 0.9995), 128, 128, moe(8, 4, 3, 3, 2, 128)),
    attention(8, 2, 128, 128, 0.0884, 128, 128, 1e6, 2.0, mlp=moe(10, 2, 2, 2, 1, 64)),
    mlstm(4, 128, 128, 15.0),
    attention(8, 2, 128, 128, 0.0884, 65, 128, 1e6, 2.0, kv_from=1, mlp=moe(12, 0, 4, 4, 2, 64)),
    attention(16, 1, 128, 128, 0.0884, 200, 64),
    lightning((0.8, 0.98, 0.3, 0.6, 0.95, 0.999), 64, 64),
    attention(32, 8, 128, 128, 0.0884, 100, 32, 1e4),
    mlstm(6, 64, 64, 8.0, moe(6, 6, 4, 4, 3, 64)),
    attention(4, 4, 128, 128, 0.12, None, 128, 1e4),
    attention(32, 4, 128, 128, 0.0884, 129, 128, 1e4),
], width=256, vocab=510, eps=1e-6, scale=0.25)

CONFIGS = {"mixed": MIXED, "wide": WIDE, "even": EVEN}

_models = {}


def model(name, seed=11):
    """(configuration, weights) of a named case; random weights are drawn once."""
    if name not in _models:
        _models[name] = O.random_model(CONFIGS[name], seed)
    return CONFIGS[name], _models[name]


def shapes_of(weights):
    return {k: tuple(t.shape) for k, t in weights.items()}
