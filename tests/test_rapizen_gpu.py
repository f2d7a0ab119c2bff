"""Whole Rapizen models through the engine - prompts, portions, mixed batches, decoding, reuse of pages,
generation and the commands - against the plain oracle.  fp32 runs are held to fp32 rounding, bf16 runs to a
few bf16 steps of the logits' spread."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from oracle import rapizen_oracle as O
from tests import rapizen_cases as C

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


def engine_of(name, dtype, pages=16, page_size=64, live=4, max_extend=1024, weights=None):
    from sglang_cpp_b200.engine import Engine, EngineConfig
    from sglang_cpp_b200.host_batch import HostBatcher
    from sglang_cpp_b200.models import read_rapizen
    from sglang_cpp_b200.weights import pack_layer_stack

    cfg, w = C.model(name)
    mc = read_rapizen(cfg)
    mc.torch_dtype = getattr(torch, dtype)
    e = Engine(mc, EngineConfig(page_size, pages, live, pages * page_size, max_extend))
    e.load_weights(pack_layer_stack(mc, weights or w))
    return e, HostBatcher(e, pages, page_size, live, enable_prefix_cache=False)


def run(e, hb, req, ids, portions):
    """Feed `ids` in the given portions; logits at every position."""
    out, at = [], 0
    for n in portions:
        hb.extend([req], [ids[at:at + n]]).synchronize()
        out.append(e.token_logits(range(n)))
        at += n
    assert at == len(ids)
    return torch.cat(out)


def cut(n, size):
    return [size] * (n // size) + ([n % size] if n % size else [])


_want = {}


def oracle(name, ids):
    key = (name, tuple(ids))
    if key not in _want:
        _want[key] = O.forward(*C.model(name), ids)
    return _want[key]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_whole_prompts_layer_by_layer(pkg, name, dtype):
    cfg, w = C.model(name)
    ids = C.prompt(cfg, 150, 2)
    want, trail = O.forward(cfg, w, ids, keep_layers=True)
    e, hb = engine_of(name, dtype)
    trace = e.trace_residual(len(ids))
    got = run(e, hb, hb.open_request(200), ids, [len(ids)])
    for l, x in enumerate(trail):
        rms = float(x.pow(2).mean().sqrt())
        worst = float((trace[l].double() - x).pow(2).mean(-1).sqrt().max()) / rms
        assert worst < LIMIT[dtype] / 2, f"layer {l}: {worst}"
    assert C.error(got, want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(C.CONFIGS))
@pytest.mark.parametrize("size", [1, 2, 3, 31, 33, 64, 65])
def test_portions_equal_the_whole(pkg, name, dtype, size):
    ids = C.prompt(C.CONFIGS[name], 140, 3)
    e, hb = engine_of(name, dtype)
    if size == 1:
        e.capture_graphs([1])
    got = run(e, hb, hb.open_request(200), ids, [7] + cut(133, size))
    assert C.error(got, oracle(name, ids)) < LIMIT[dtype]


@pytest.mark.parametrize("expand_min", ["0", "100000"])
def test_both_forms_of_prefill_attention_agree(pkg, monkeypatch, expand_min):
    """Keys and values expanded for every portion, or never."""
    monkeypatch.setenv("B200_LATENT_EXPAND_MIN", expand_min)
    ids = C.prompt(C.MIXED, 140, 3)
    e, hb = engine_of("mixed", "bfloat16")
    got = run(e, hb, hb.open_request(200), ids, [40, 1, 2, 60, 3, 34])
    assert C.error(got, oracle("mixed", ids)) < LIMIT["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "even"])
@pytest.mark.parametrize("page_size", [1, 16, 64])
def test_mixed_batches_equal_each_request_alone(pkg, name, dtype, page_size):
    """Long portions, short portions and single tokens of four unequal requests in the same steps; one of
    them is left out now and then, rows and pages of finished ones are used by the next."""
    cfg = C.CONFIGS[name]
    e, hb = engine_of(name, dtype, pages=768 // page_size, page_size=page_size)
    e.capture_graphs([1, 2, 4])
    prompts = [C.prompt(cfg, n, 20 + n) for n in (170, 9, 120, 66, 130, 5, 71, 1)]
    rng = np.random.default_rng(page_size)
    waiting, live, got = list(range(len(prompts))), {}, {i: [] for i in range(len(prompts))}
    steps = 0
    while waiting or live:
        while waiting and len(live) < 4:
            i = waiting.pop(0)
            live[i] = hb.open_request(len(prompts[i]))
        order = [i for i in live if rng.random() < 0.8] or list(live)
        rng.shuffle(order)
        portions = []
        for i in order:
            left = len(prompts[i]) - live[i].cached_len
            portions.append(min(left, int(rng.choice([1, 1, 2, 5, 17, 40, 90]))))
        take = [prompts[i][live[i].cached_len:live[i].cached_len + n] for i, n in zip(order, portions)]
        hb.extend([live[i] for i in order], take).synchronize()
        logits = e.token_logits(range(sum(portions)))
        for i, part in zip(order, logits.split(portions)):
            got[i].append(part)
        for i in [i for i in order if live[i].cached_len == len(prompts[i])]:
            hb.release(live.pop(i))
        steps += 1
    assert len(hb.cache_manager.free_pages) == 768 // page_size
    for i, p in enumerate(prompts):
        assert C.error(torch.cat(got[i]), oracle(name, p)) < LIMIT[dtype], f"request {i} after {steps} steps"


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_that_held_something_else(pkg, dtype):
    """A pool of three pages used up by one request after the other, in a different page order each time."""
    e, hb = engine_of("mixed", dtype, pages=3)
    for k, n in enumerate((192, 70, 129, 65, 192)):
        ids = C.prompt(C.MIXED, n, 40 + k)
        a = hb.open_request(192)
        got = run(e, hb, a, ids, [n - 3, 1, 2])
        assert C.error(got, oracle("mixed", ids)) < LIMIT[dtype]
        hb.cache_manager.free_pages.reverse()
        hb.release(a)


def pointed(name, far, extra=0):
    """Weights of `name` where, in layer 0, the token at the end of the prompt attends to the token at `far`
    with nearly all its weight, so that losing that one key changes everything behind it."""
    cfg, w = C.model(name)
    w = dict(w)
    m = cfg["layers"][0]["mixer"]
    H, d = m["heads"], m["dim"]
    ids = C.prompt(cfg, 140 + extra, 5)
    ask, mark = cfg["vocab"] - 1, cfg["vocab"] - 2
    ids = [t % (cfg["vocab"] - 2) for t in ids]
    ids[far], ids[-1] = mark, ask
    n1 = lambda tok: O.rms_normalise(w["embed"][tok].double(), 1 + w["l0.norm1"].double(), cfg["norm"]["eps"])
    eps = cfg["norm"]["eps"]
    W = {k: t.double() for k, t in w.items() if k.startswith("l0.mix.")}
    cq = O.latent_of(n1(ask)[None], W, "l0.mix.dq", eps)[0]
    c = O.latent_of(n1(mark)[None], W, "l0.mix.dkv", eps)[0]
    k = (W["l0.mix.uk"] @ c).view(H, d)
    # the asking token's query along the marked token's key, with a score of about 40
    uq = W["l0.mix.uq"].view(H, d, -1)
    for h in range(H):
        q = 40 / m["scale"] * k[h] / (k[h] @ k[h])
        uq[h] += torch.outer(q - uq[h] @ cq, cq) / (cq @ cq)
    w["l0.mix.uq"] = uq.reshape(H * d, -1).bfloat16()
    return cfg, w, ids


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 138])
def test_a_far_key_is_seen_from_a_prompt_and_from_decoding(pkg, dtype, far):
    cfg, w, ids = pointed("mixed", far)
    want = O.forward(cfg, w, ids)[-1:]
    lost = O.forward(cfg, w, ids[:far] + [(ids[far] + 1) % 200] + ids[far + 1:])[-1:]
    assert C.error(lost, want) > 0.2           # the key matters
    for portions in ([140], [139, 1], [100, 38, 2], [64, 64, 12]):
        e, hb = engine_of("mixed", dtype, weights=w)
        got = run(e, hb, hb.open_request(140), ids, portions)[-1:]
        assert C.error(got, want) < 2 * LIMIT[dtype], portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(pkg, dtype):
    ids = C.prompt(C.MIXED, 330, 6)
    e, hb = engine_of("mixed", dtype)
    e.capture_graphs([1])
    got = run(e, hb, hb.open_request(400), ids, [5] + [1] * 325)
    assert C.error(got, oracle("mixed", ids)) < LIMIT[dtype]


def test_padded_decode_graphs(pkg):
    """Three requests on a graph of four rows: the dummy row changes nothing."""
    e, hb = engine_of("even", "bfloat16")
    e.capture_graphs([4])
    prompts = [C.prompt(C.EVEN, n, 60 + n) for n in (40, 3, 70)]
    reqs = [hb.open_request(100) for _ in prompts]
    hb.extend(reqs, [p[:-2] for p in prompts]).synchronize()
    for j in (-2, -1):
        hb.extend(reqs, [[p[j]] for p in prompts]).synchronize()
        got = e.logits(3).float()
        for i, p in enumerate(prompts):
            n = len(p) + j
            assert C.error(got[i:i + 1], oracle("even", p)[n:n + 1]) < LIMIT["bfloat16"]


# ---- generation ------------------------------------------------------------------------
def greedy(name, ids, n):
    cfg, w = C.model(name)
    ids = list(ids)
    for _ in range(n):
        ids.append(int(O.forward(cfg, w, ids)[-1].argmax()))
    return ids[-n:]


@pytest.mark.parametrize("page_size, max_extend", [(16, 1024), (1, 48), (64, 100)])
def test_greedy_generation_through_the_scheduler(pkg, page_size, max_extend):
    """Prompts longer than a prefill step, a prefix that two requests share, more requests than rows."""
    from sglang_cpp_b200.generate import generate

    e, _ = engine_of("mixed", "float32", pages=1024 // page_size, page_size=page_size, live=3, max_extend=max_extend)
    e.capture_graphs([])
    shared = C.prompt(C.MIXED, 40, 70)
    prompts = [shared + [3, 1], C.prompt(C.MIXED, 130, 71), shared + [3, 2], C.prompt(C.MIXED, 1, 72), shared]
    got = generate(e, prompts, 8)
    assert got == [greedy("mixed", p, 8) for p in prompts]
    assert generate(e, prompts[:2], 5, prefix_cache=False) == [g[:5] for g in got[:2]]


def test_sampling(pkg):
    from sglang_cpp_b200.generate import generate

    for dtype in DTYPES:
        e, _ = engine_of("even", dtype)
        p = [C.prompt(C.EVEN, 20, 80)]
        cold = generate(e, p, 6, temperature=1e-5)
        assert cold == generate(e, p, 6) == generate(e, p, 6, temperature=3.0, top_k=1)
        hot = [tuple(generate(e, p, 6, temperature=2.0, seed=s)[0]) for s in range(4)]
        assert len(set(hot)) > 1


# ---- commands ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_command(pkg, tmp_path, dtype):
    cfg, w = C.model("mixed")
    C.write_checkpoint(tmp_path / "m", cfg, w)
    a, b = C.prompt(cfg, 100, 90), C.prompt(cfg, 30, 91)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}, {"id": "a", "tokens": a[70:71], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[71:], "want": [28]}, {"id": "b", "tokens": b[2:], "want": [0, 27]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": a, "want": [99]}], "end": ["c"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                        str(tmp_path / "o"), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                       capture_output=True, text=True, timeout=250)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "o" / "1.f32").exists()
    A, B = oracle("mixed", a), oracle("mixed", b)
    for step, want in ((0, A[[0, 69]]), (2, torch.stack([A[99], B[2], B[29]])), (3, A[99:])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{step}.f32", "<f4")).view(len(want), -1)
        assert C.error(got, want) < 2 * LIMIT[dtype]


def test_generate_command(pkg, tmp_path):
    cfg, w = C.model("mixed")
    C.write_checkpoint(tmp_path / "m", cfg, w)
    prompts = [C.prompt(cfg, 25, 92), C.prompt(cfg, 3, 93)]
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--max-new-tokens", "5", "--num-pages", "64", "--max-seq-len", "100"],
                       input="\n".join(" ".join(map(str, p)) for p in prompts), capture_output=True, text=True,
                       timeout=250, env=dict(os.environ))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [[int(t) for t in x.split()] for x in r.stdout.splitlines()] == [greedy("mixed", p, 5) for p in prompts]
