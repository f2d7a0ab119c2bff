"""Small Rapizen configurations and helpers shared by the CPU and GPU tests."""
import json

import torch

from oracle import rapizen_oracle as O


def layer(heads, dim, vdim, q_rank, kv_rank, scale, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width=136, vocab=203, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Rapizen", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers}


# every branch, odd sizes everywhere, no two layers alike
MIXED = config([
    layer(5, 40, 56, 72, 80, 0.16, moe(7, 3, 52)),
    layer(3, 96, 32, 48, 200, 0.1, None),
    layer(4, 24, 128, 130, 130, 0.21, dense(90)),
    layer(1, 128, 8, 16, 24, 0.09, moe(5, 1, 200)),
    layer(18, 16, 16, 64, 64, 0.25, moe(3, 3, 64)),
])
# head sizes above 128 (attention never expands) and a latent wider than the tensor-core kernel takes
WIDE = config([
    layer(2, 144, 160, 96, 600, 0.08, dense(320)),
    layer(3, 200, 136, 40, 300, 0.07, moe(4, 2, 72)),
], width=320, vocab=97, eps=1e-6, logit_scale=1.3)
# one layer of each kind, sizes that need no padding
EVEN = config([
    layer(8, 128, 128, 128, 256, 0.0884, dense(512)),
    layer(40, 128, 128, 192, 384, 0.0884, moe(16, 4, 128)),
], width=256, vocab=512, eps=1e-6, logit_scale=1.0)

CONFIGS = {"mixed": MIXED, "wide": WIDE, "even": EVEN}


def write_checkpoint(directory, cfg, weights):
    from sglang_cpp_b200.weights import write_safetensors

    directory.mkdir(parents=True, exist_ok=True)
    (directory / "config.json").write_text(json.dumps(cfg))
    write_safetensors(directory / "model.safetensors", weights)
    return directory


def prompt(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


_models = {}


def model(name, seed=11):
    """(configuration, weights) of a named case; random weights are drawn once."""
    if name not in _models:
        _models[name] = O.random_model(CONFIGS[name], seed)
    return CONFIGS[name], _models[name]


def error(got, want):
    """Largest root-mean-square difference of a row of logits (means taken off), relative to the rms of all."""
    got, want = got.double(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt())
