"""Small Saluzen configurations and helpers shared by the CPU and GPU tests."""
from oracle import saluzen_oracle as O
from tests.rapizen_cases import error, prompt, write_checkpoint  # noqa: F401  (the same for every layer stack)


def attention(heads, kv_heads, dim, vdim, scale, dims, base=5000.0, scaling=None, size=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if size:
        m["mask"] = {"size": size}
    return m


def state_space(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": ff and {"kind": "dense", "ff": ff}}


def parallel_2(left, right, left_scale, right_scale, ff=None):
    return {"type": "parallel_2", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"left": left, "left_scale": left_scale, "right": right, "right_scale": right_scale}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=3000.0, kv_from=None, ff=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": ff and {"kind": "dense", "ff": ff}}


def config(layers, width=136, vocab=203, eps=1e-5):
    return {"architecture": "Saluzen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


# every branch, odd sizes everywhere, no two layers alike
MIXED = config([
    latent(5, 40, 12, 56, 72, 83, 0.14, ff=100),
    parallel(attention(6, 2, 40, 56, 0.16, 24, 900.0, (3.0, 1.5, 5.0, 60)), state_space(6, 20, 24, 3, 5, 4), 90),
    parallel_2(attention(6, 3, 36, 24, 0.2, 36, size=33), delta(6, 3, 24, 40, 2), 0.6, 1.4),
    latent(3, 24, 12, 128, 130, 83, 0.2, kv_from=0),
    parallel(attention(5, 5, 64, 24, 0.12, 2), state_space(5, 72, 100, 1, 1, 3)),
    latent(18, 16, 30, 16, 64, 64, 0.18, base=50.0, ff=64),
    parallel_2(attention(4, 1, 128, 72, 0.1, 64, size=7), delta(3, 1, 100, 20, 9), 1.3, -0.7, 52),
    latent(7, 52, 30, 33, 40, 64, 0.13, base=50.0, kv_from=5, ff=70),
])
# heads and states wider than the tensor-core kernels take, latents wider than they take
WIDE = config([
    parallel_2(attention(2, 1, 144, 160, 0.08, 100, size=50), delta(2, 2, 200, 264, 4), 0.9, 0.9, 320),
    latent(3, 100, 60, 136, 40, 600, 0.09, ff=72),
    parallel(attention(3, 3, 160, 24, 0.08, 160, 1e4, (8.0, 1.0, 4.0, 300)), state_space(4, 136, 260, 2, 3, 1), 64),
    latent(2, 150, 60, 40, 96, 600, 0.07, kv_from=1),
], width=320, vocab=97, eps=1e-6)
# sizes that need no padding, on the tensor-core kernels; chunks of whole tiles and one off them
EVEN = config([
    parallel(attention(8, 2, 128, 128, 0.0884, 128, 1e6, (8.0, 1.0, 4.0, 64)), state_space(8, 64, 128, 1, 4, 1), 512),
    latent(16, 64, 64, 128, 192, 512, 0.0884, base=1e4, ff=256),
    parallel_2(attention(8, 2, 128, 128, 0.0884, 64, size=128), delta(4, 2, 128, 128, 4), 0.7, 1.2, 256),
    latent(40, 96, 32, 128, 128, 96, 0.0884, base=1e4),
    parallel_2(attention(16, 1, 128, 128, 0.0884, 128, size=65), delta(4, 4, 64, 64, 3), 1.0, 1.0),
    latent(8, 64, 64, 128, 64, 512, 0.0884, base=1e4, kv_from=1, ff=64),
    parallel(attention(4, 4, 128, 128, 0.0884, 32), state_space(16, 128, 64, 4, 2, 8)),
], width=256, vocab=512, eps=1e-6)

CONFIGS = {"mixed": MIXED, "wide": WIDE, "even": EVEN}

_models = {}


def model(name, seed=11):
    """(configuration, weights) of a named case; random weights are drawn once."""
    if name not in _models:
        _models[name] = O.random_model(CONFIGS[name], seed)
    return CONFIGS[name], _models[name]


def shapes_of(weights):
    return {k: tuple(t.shape) for k, t in weights.items()}
