"""Whole Retotar models through the engine - prompts, portions, mixed batches, decoding, reuse of pages and states,
generation and the commands - against the plain oracle.  fp32 runs are held to fp32 rounding; bf16 runs to about
twice the rounding error seen with each configuration."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from oracle import retotar_oracle as O
from tests import retotar_cases as C

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
FP32_LIMIT = 4e-5
BF16_LIMIT = {"mixed": 0.05, "wide": 0.05, "even": 0.05, "pointing": 0.03, "states": 0.03}


def limit(name, dtype):
    return FP32_LIMIT if dtype == "float32" else BF16_LIMIT[name]


DTYPES = ["float32", "bfloat16"]


def engine_for(cfg, w, dtype, pages=16, page_size=64, live=4, max_extend=1024):
    from sglang_cpp_b200.engine import Engine, EngineConfig
    from sglang_cpp_b200.host_batch import HostBatcher
    from sglang_cpp_b200.models import read_retotar
    from sglang_cpp_b200.weights import pack_layer_stack

    mc = read_retotar(cfg, C.shapes_of(w))
    mc.torch_dtype = getattr(torch, dtype)
    e = Engine(mc, EngineConfig(page_size, pages, live, pages * page_size, max_extend))
    e.load_weights(pack_layer_stack(mc, w))
    return e, HostBatcher(e, pages, page_size, live, enable_prefix_cache=False)


def engine_of(name, dtype, **kw):
    return engine_for(*C.model(name), dtype, **kw)


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
        assert worst < limit(name, dtype), f"layer {l}: {worst}"
    assert C.error(got, want) < limit(name, dtype)


def test_routers_that_read_the_whole_stream(pkg):
    """Random router matrices (in fp32, where no choice of experts is close)."""
    cfg = C.MIXED
    w = O.random_model(cfg, 5, coded_router=False)
    ids = C.prompt(cfg, 90, 7)
    e, hb = engine_for(cfg, w, "float32")
    got = run(e, hb, hb.open_request(200), ids, [60, 1, 29])
    assert C.error(got, O.forward(cfg, w, ids)) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(C.CONFIGS))
@pytest.mark.parametrize("size", [1, 2, 3, 31, 33, 64, 65])
def test_portions_equal_the_whole(pkg, name, dtype, size):
    ids = C.prompt(C.CONFIGS[name], 140, 3)
    e, hb = engine_of(name, dtype)
    if size == 1:
        e.capture_graphs([1])
    got = run(e, hb, hb.open_request(200), ids, [7] + cut(133, size))
    assert C.error(got, oracle(name, ids)) < limit(name, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(C.CONFIGS))
@pytest.mark.parametrize("page_size", [1, 16, 64])
def test_mixed_batches_equal_each_request_alone(pkg, name, dtype, page_size):
    """Long portions, short portions and single tokens of four unequal requests in the same steps; one of
    them is left out now and then, rows, states and pages of finished ones are used by the next."""
    cfg = C.CONFIGS[name]
    e, hb = engine_of(name, dtype, pages=768 // page_size, page_size=page_size)
    e.capture_graphs([1, 2, 4])
    prompts = [C.prompt(cfg, n, 20 + n) for n in (170, 9, 120, 66, 130, 5, 71, 1)]
    rng = np.random.default_rng(page_size)
    waiting, live, got = list(range(len(prompts))), {}, {i: [] for i in range(len(prompts))}
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
    assert len(hb.cache_manager.free_pages) == 768 // page_size
    for i, p in enumerate(prompts):
        assert C.error(torch.cat(got[i]), oracle(name, p)) < limit(name, dtype), f"request {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "even"])
def test_pages_and_states_that_held_something_else(pkg, name, dtype):
    """A pool of three pages and one state used up by one request after the other, in a different page order
    each time."""
    e, hb = engine_of(name, dtype, pages=3, live=1)
    for k, n in enumerate((192, 70, 129, 1, 65, 192)):
        ids = C.prompt(C.CONFIGS[name], n, 240 + k)
        a = hb.open_request(192)
        got = run(e, hb, a, ids, [n - 3, 1, 2] if n > 3 else [n])
        assert C.error(got, oracle(name, ids)) < limit(name, dtype)
        hb.cache_manager.free_pages.reverse()
        hb.release(a)


# ---- keys that stand out ---------------------------------------------------------------
# One attention layer alone.  Column 0 of the embedding marks a token, column 1 lets one ask: the asking token's query
# points at the marked token's key, which takes nearly all the weight wherever it is seen.  Keys rotate in two other
# dimensions only.
def pointing(dim, window, n, spots, asks, seed=8):
    cfg = C.config([C.attention(4, 2, dim, dim, 32 / dim, window, 2)], width=dim, vocab=64, scale=1.0)
    w = O.random_model(cfg, seed)
    ask, mark = 62, 63
    ids = [t % 62 for t in C.prompt(cfg, n, seed)]
    for s in spots:
        ids[s] = mark
    for a in asks:
        ids[a] = ask
    w["embed"][:, :2] = 0
    w["embed"][mark, 0], w["embed"][ask, 1] = 30.0, 30.0
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(dim).bfloat16(), torch.zeros(dim).bfloat16()
    at = 5                                       # the dimension in which key and query meet
    k, q = 0.02 * torch.eye(dim), 0.02 * torch.eye(dim)
    k[at, 0], q[at, 1] = 3.0, 3.0
    w["l0.mix.k"], w["l0.mix.q"] = k.repeat(2, 1).bfloat16(), q.repeat(4, 1).bfloat16()
    return cfg, w, ids


EDGES = [  # (window, spot of the marked token, asking positions)
    (50, 100, (101, 149, 150, 155)),   # seen by the 49 tokens behind it
    (64, 63, (64, 126, 127)),
    (64, 64, (127, 128, 130)),
    (128, 0, (127, 128, 131)),
    (129, 64, (192, 193)),
    (1, 20, (21, 22)),                 # nobody but oneself
    (140, 125, (264, 265, 268)),       # a window over three tiles
    (500, 3, (140, 141)),              # all of them
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 128])
@pytest.mark.parametrize("window, spot, asks", EDGES)
def test_window_edges_show_in_prompts_and_in_decoding(pkg, dtype, dim, window, spot, asks):
    n = max(asks) + 5
    cfg, w, ids = pointing(dim, window, n, [spot], asks)
    want = O.forward(cfg, w, ids)
    # the mark matters exactly where the rule says it is seen
    other = O.forward(cfg, w, ids[:spot] + [5] + ids[spot + 1:])
    for a in asks:
        moved = float((want[a] - other[a]).pow(2).mean().sqrt() / want.std())
        assert (moved > 0.04) if a - spot < window else (moved == 0), (a, moved)
    e, hb = engine_for(cfg, w, dtype)
    e.capture_graphs([1])
    first = min(asks)
    for portions in ([n], [first] + [1] * (n - first), [64, n - 64] if n > 64 else [3, n - 3], cut(n, 7)):
        req = hb.open_request(n)
        got = run(e, hb, req, ids, portions)
        hb.release(req)
        for a in asks:
            assert C.error(got[a:a + 1], want[a:a + 1]) < limit("pointing", dtype), (portions, a)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 128])
def test_far_keys_are_found(pkg, dtype, dim):
    """Without a window: the first token, tokens around page borders and one near the end, asked for from far away.  (What
    a far value turns by depends on the distance.)"""
    n = 420
    e = None
    for spot in (0, 1, 63, 64, 127, 128, 400):
        cfg, w, ids = pointing(dim, None, n, [spot], (n - 2, n - 1))
        want = O.forward(cfg, w, ids)
        other = O.forward(cfg, w, ids[:spot] + [5] + ids[spot + 1:])
        assert float((want[n - 1] - other[n - 1]).pow(2).mean().sqrt() / want.std()) > 0.02
        if e is None:
            e, hb = engine_for(cfg, w, dtype)
            e.capture_graphs([1])
        for portions in ([n], [n - 2, 1, 1], [n - 3, 3], [200, 219, 1]):
            req = hb.open_request(n)
            got = run(e, hb, req, ids, portions)
            hb.release(req)
            assert C.error(got[n - 2:], want[n - 2:]) < limit("pointing", dtype), (spot, portions)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["lightning", "mlstm"])
def test_states_remember_from_far_away(pkg, dtype, kind):
    """Heads that never forget: the first token still moves the logits hundreds of tokens on, from a prompt, from
    portions and from decoding."""
    n = 300
    layer = C.lightning((1.0, 0.9999), 24, 40) if kind == "lightning" else C.mlstm(2, 24, 40, 30.0)
    cfg = C.config([layer], width=64, vocab=64)
    w = O.random_model(cfg, 3)
    ids = [t % 62 for t in C.prompt(cfg, n, 5)]
    ids[2] = 63
    if kind == "mlstm":
        w["l0.mix.f"] = torch.zeros_like(w["l0.mix.f"])
        w["l0.mix.f.b"] = torch.full_like(w["l0.mix.f.b"], 12.0)
    w["embed"][:, 0], w["embed"][63, 0] = 0.0, 30.0
    w["l0.norm1"], w["l0.norm1.b"] = torch.ones(64).bfloat16(), torch.zeros(64).bfloat16()
    for name in "kv" if kind == "lightning" else "i":            # the marked token writes more than all others
        w["l0.mix." + name] = 0.1 * w["l0.mix." + name]
        w["l0.mix." + name][:, 0] = 1.5
    want = O.forward(cfg, w, ids)
    other = O.forward(cfg, w, ids[:2] + [5] + ids[3:])
    assert float((want[n - 1] - other[n - 1]).pow(2).mean().sqrt() / want.std()) > 0.05
    e, hb = engine_for(cfg, w, dtype)
    e.capture_graphs([1])
    for portions in ([n], [n - 2, 1, 1], [1, 2, n - 3], [70, 64, 66, 99, 1]):
        req = hb.open_request(n)
        got = run(e, hb, req, ids, portions)
        hb.release(req)
        assert C.error(got[n - 2:], want[n - 2:]) < limit("states", dtype), portions


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "even"])
def test_long_decoding(pkg, name, dtype):
    """Windows slide over decoded tokens, states run on through hundreds of steps."""
    ids = C.prompt(C.CONFIGS[name], 330, 6)
    e, hb = engine_of(name, dtype)
    e.capture_graphs([1])
    got = run(e, hb, hb.open_request(400), ids, [5] + [1] * 325)
    assert C.error(got, oracle(name, ids)) < limit(name, dtype)


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
            assert C.error(got[i:i + 1], oracle("even", p)[n:n + 1]) < limit("even", "bfloat16")


# ---- generation ------------------------------------------------------------------------
def greedy(name, ids, n):
    cfg, w = C.model(name)
    ids = list(ids)
    for _ in range(n):
        ids.append(int(O.forward(cfg, w, ids)[-1].argmax()))
    return ids[-n:]


@pytest.mark.parametrize("page_size, max_extend", [(16, 1024), (1, 48), (64, 100)])
def test_greedy_generation_through_the_scheduler(pkg, page_size, max_extend):
    """Prompts longer than a prefill step, a prefix that two requests share (its state is not in the pages, so
    it is computed twice), more requests than rows."""
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
    A, B = oracle("mixed", a), oracle("mixed", b)
    for step, want in ((0, A[[0, 69]]), (2, torch.stack([A[99], B[2], B[29]])), (3, A[99:])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{step}.f32", "<f4")).view(len(want), -1)
        assert C.error(got, want) < limit("mixed", dtype)


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
