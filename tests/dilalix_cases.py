"""Small Dilalix configurations and helpers shared by the CPU and GPU tests."""
from oracle import dilalix_oracle as O
from tests.rapizen_cases import error, prompt, write_checkpoint  # noqa: F401  (the same for every layer stack)


def attention(heads, kv_heads, dim, vdim, scale, size, keep_first, dims, base=5000.0, v_mix=False, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
                      "mask": {"size": size, "keep_first": keep_first}, "rot": {"base": base, "dims": dims}}}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, count, keep, scale, ff, limit, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale},
            "expert": {"ff": ff, "limit": limit}, "shared": shared and {"ff": shared[0], "limit": shared[1]}}


def config(layers, width=136, vocab=203, eps=1e-5):
    return {"architecture": "Dilalix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


# every branch, odd sizes everywhere, no two layers alike
MIXED = config([
    attention(6, 2, 40, 56, 0.2, 33, 3, 24, v_mix=True, mlp=moe(12, 3, 4, 2, 1.7, 52, 0.8, (80, 1.3))),
    gla(3, 24, 72, 8.0),
    attention(5, 5, 64, 24, 0.15, 9, 0, 64, base=100.0, mlp=dense(90)),
    gla(5, 100, 20, 1.0, moe(6, 1, 1, 1, 1.0, 200, 3.0)),
    attention(4, 2, 128, 56, 0.09, 64, 70, 2, v_mix=True, mlp=moe(8, 3, 8, 3, 2.2, 64, 1.0, (40, 0.6))),
    gla(1, 144, 136, 16.0, dense(50)),
])
# heads of more than 128 and head counts that the tensor-core kernels do not take; no expert groups to drop
WIDE = config([
    gla(2, 200, 264, 4.0, dense(320)),
    attention(2, 1, 144, 160, 0.08, 40, 5, 100, mlp=moe(10, 2, 2, 2, 1.5, 72, 2.0, (72, 2.0))),
    attention(3, 3, 128, 128, 0.09, 77, 1, 128, v_mix=True, mlp=dense(64)),
    attention(12, 3, 96, 128, 0.1, 20, 2, 30, v_mix=True),
], width=320, vocab=97, eps=1e-6)
# sizes that need no padding; windows of whole tiles and one off them
EVEN = config([
    gla(4, 128, 128, 16.0, dense(512)),
    attention(8, 2, 128, 128, 0.0884, 128, 4, 128, base=1e6, v_mix=True, mlp=moe(16, 4, 4, 2, 2.5, 128, 7.0, (128, 7.0))),
    gla(6, 64, 64, 8.0, moe(16, 2, 2, 1, 1.0, 64, 1.0, (256, 4.0))),
    attention(8, 2, 128, 128, 0.0884, 65, 130, 64, base=1e4, v_mix=True, mlp=dense(256)),
    attention(16, 1, 128, 128, 0.0884, 200, 0, 128, mlp=dense(64)),
], width=256, vocab=512, eps=1e-6)

CONFIGS = {"mixed": MIXED, "wide": WIDE, "even": EVEN}
RANKS = {"mixed": {1: 10, 3: 33, 5: 70}, "wide": {0: 5}, "even": {2: 24}}

_models = {}


def model(name, seed=11):
    """(configuration, weights) of a named case; random weights are drawn once."""
    if name not in _models:
        _models[name] = O.random_model(CONFIGS[name], seed, RANKS[name])
    return CONFIGS[name], _models[name]


def shapes_of(weights):
    return {k: tuple(t.shape) for k, t in weights.items()}
