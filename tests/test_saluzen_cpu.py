"""Saluzen without a GPU: the oracle's own consistency, the registry and weight packing."""
import copy
import math

import pytest
import torch

from oracle import saluzen_oracle as O
from tests import saluzen_cases as C

F64 = torch.float64


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# ---- the oracle -----------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_oracle_is_causal_and_its_decode_equals_its_prefill(name):
    cfg, w = C.model(name)
    ids = C.prompt(cfg, 40, 1)
    full = O.forward(cfg, w, ids)
    for n in (1, 2, 35):
        torch.testing.assert_close(O.forward(cfg, w, ids[:n]), full[:n])
    other = ids[:30] + [(t + 1) % cfg["vocab"] for t in ids[30:]]
    torch.testing.assert_close(O.forward(cfg, w, other)[:30], full[:30])


def test_oracle_chunks_in_words():
    """Chunks of 4: token 9 is in the chunk 8 .. 11."""
    seen = O.visible(12, 4)
    assert seen[9].nonzero().flatten().tolist() == [8, 9]
    assert seen[8].nonzero().flatten().tolist() == [8]
    assert seen[7].nonzero().flatten().tolist() == [4, 5, 6, 7]
    assert O.visible(5)[3].nonzero().flatten().tolist() == [0, 1, 2, 3]


def test_oracle_sinks_take_their_share():
    s = torch.tensor([[1.0, -2.0, 0.5]], dtype=F64)
    e = torch.exp(s)
    torch.testing.assert_close(O.sink_softmax(s, torch.tensor(0.0)), e / (1 + e.sum()))
    torch.testing.assert_close(O.sink_softmax(s, torch.tensor(50.0, dtype=F64)), e / (math.exp(50.0) + e.sum()))
    torch.testing.assert_close(O.sink_softmax(s, None), torch.softmax(s, -1))
    assert float(O.sink_softmax(torch.full((1, 2), -500.0, dtype=F64), torch.tensor(0.0)).sum()) < 1e-200


def test_oracle_frequencies_are_stretched_by_wavelength():
    rot = {"base": 10000.0, "dims": 64}
    plain = O.frequencies(rot)
    f = O.frequencies({**rot, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 128}})
    wave = 2 * math.pi / plain
    short, long = wave < 32, wave > 128
    between = ~short & ~long
    assert bool(short.any()) and bool(long.any()) and bool(between.any())
    torch.testing.assert_close(f[short], plain[short])
    torch.testing.assert_close(f[long], plain[long] / 8)
    assert bool((f[between] < plain[between]).all() and (f[between] > plain[between] / 8).all())


def test_oracle_rotations_depend_on_distances_only():
    for turn in (O.rotate_half, O.rotate_neighbours):
        rot = {"base": 100.0, "dims": 6}
        q, k = rand(1, 1, 8), rand(1, 1, 8, seed=1)
        dot = lambda i, j: (turn(q, torch.tensor([i]), rot) * turn(k, torch.tensor([j]), rot)).sum()
        torch.testing.assert_close(dot(9, 4), dot(105, 100))
        torch.testing.assert_close(turn(q, torch.tensor([7]), rot)[..., 6:], q[..., 6:])
    e = torch.zeros(1, 1, 8, dtype=F64)
    e[..., 0] = 1
    assert O.rotate_half(e, torch.tensor([1]), rot).nonzero()[:, 2].tolist() == [0, 3]
    assert O.rotate_neighbours(e, torch.tensor([1]), rot).nonzero()[:, 2].tolist() == [0, 1]


def test_oracle_convolution_in_words():
    x, taps, bias = rand(6, 2), rand(2, 3, seed=1), rand(2, seed=2)
    got = O.short_conv(x, taps, bias)
    y = x[4] * taps[:, 2] + x[3] * taps[:, 1] + x[2] * taps[:, 0] + bias
    torch.testing.assert_close(got[4], y * torch.sigmoid(y))
    y = x[0] * taps[:, 2] + bias
    torch.testing.assert_close(got[0], y * torch.sigmoid(y))


def test_oracle_recurrences_continue_from_their_state():
    q, k, v = rand(9, 2, 5), rand(9, 2, 5, seed=1), rand(9, 2, 3, seed=2)
    g, b = torch.sigmoid(rand(9, 2, seed=3)), torch.sigmoid(rand(9, 2, seed=4))
    for step in (lambda s, S: O.ssd_recurrence(v[s], k[s], q[s], g[s], b[s], S), lambda s, S: O.delta_recurrence(q[s], k[s], v[s], g[s], b[s], S)):
        whole, last = step(slice(0, 9), None)
        a, mid = step(slice(0, 4), None)
        c, end = step(slice(4, 9), mid)
        torch.testing.assert_close(torch.cat([a, c]), whole)
        torch.testing.assert_close(end, last)


def test_oracle_state_space_equals_its_sum_over_the_past():
    x, B, Cc = rand(7, 1, 3), rand(7, 1, 4, seed=1), rand(7, 1, 4, seed=2)
    g, dt = torch.sigmoid(rand(7, 1, seed=3)), torch.rand(7, 1, dtype=F64)
    got, _ = O.ssd_recurrence(x, B, Cc, g, dt)
    for t in range(7):
        want = sum(g[s + 1:t + 1].prod() * dt[s] * (B[s, 0] @ Cc[t, 0]) * x[s, 0] for s in range(t + 1))
        torch.testing.assert_close(got[t, 0], want)


def test_oracle_delta_rule_replaces_what_a_key_held():
    """With unit keys, full strength and no decay the state answers a key with the last value written to it."""
    k = torch.zeros(3, 1, 4, dtype=F64)
    k[0, 0, 1] = k[1, 0, 2] = k[2, 0, 1] = 1
    v, one = rand(3, 1, 2), torch.ones(3, 1, dtype=F64)
    q = k[[0, 0, 2]]
    o, S = O.delta_recurrence(q, k, v, one, one)
    torch.testing.assert_close(o[:, 0], v[[0, 0, 2], 0])       # token 1 asks for what token 0 wrote
    torch.testing.assert_close(S[0, 2], v[1, 0])
    o, _ = O.delta_recurrence(q, k, v, one, 0.5 * one)
    torch.testing.assert_close(o[2, 0], 0.5 * (0.5 * v[0, 0]) + 0.5 * v[2, 0])


# ---- registry and weights ----------------------------------------------------------
def test_registry_reads_every_layer(pkg, tmp_path):
    from sglang_cpp_b200 import _lib
    from sglang_cpp_b200.models import StackConfig, read_config

    C.write_checkpoint(tmp_path, *C.model("mixed"))
    cfg = read_config(tmp_path)
    assert isinstance(cfg, StackConfig) and (cfg.num_layers, cfg.hidden_size, cfg.vocab_size) == (8, 136, 203)
    assert cfg.norm_output == _lib.NORM_BOTH and cfg.norm_offset == 0.0 and cfg.rms_norm_eps == 1e-5 and cfg.carries_state
    a, b, c, d, e, f, g, h = cfg.layers
    assert (a.mixer, a.heads, a.head_dim, a.rotary_dim, a.value_dim) == (_lib.MIXER_LATENT_ATTENTION, 5, 52, 12, 56)
    assert (a.q_rank, a.kv_rank, a.score_scale, a.rope_base, a.kv_from, a.beside) == (72, 83, 0.14, 3000.0, -1, None)
    assert (a.mlp, a.intermediate, a.epilogue) == (_lib.MLP_DENSE, 100, _lib.EPILOGUE_SWIGLU)
    assert (d.kv_from, d.mlp, h.kv_from) == (0, _lib.MLP_NONE, 5)
    assert (b.mixer, b.heads, b.kv_heads, b.head_dim, b.value_dim) == (_lib.MIXER_WINDOW_ATTENTION, 6, 2, 40, 56)
    assert (b.rotary_dim, b.rope_base, b.rope_factor, b.rope_low, b.rope_high, b.rope_original) == (24, 900.0, 3.0, 1.5, 5.0, 60.0)
    assert (b.head_norm, b.qkv_bias, b.sink, b.sink_learned, b.gate, b.chunk) == (False, True, True, False, _lib.GATE_ELEMENT, 0)
    assert (b.join, b.out_scale, b.beside.mixer, b.beside.out_scale) == (_lib.JOIN_NORMED, 1.0, _lib.MIXER_STATE_SPACE, 1.0)
    r = b.beside
    assert (r.heads, r.kv_heads, r.head_dim, r.value_dim, r.conv_taps, r.norm_groups) == (6, 3, 24, 20, 5, 4)
    assert (c.chunk, c.gate, c.sink_learned, c.out_scale, c.join) == (33, _lib.GATE_HEAD, True, 0.6, _lib.JOIN_SUM)
    r = c.beside
    assert (r.mixer, r.heads, r.kv_heads, r.head_dim, r.value_dim, r.conv_taps, r.out_scale) == (
        _lib.MIXER_DELTA_RULE, 6, 3, 24, 40, 2, 1.4)
    assert g.beside.out_scale == -0.7 and e.rope_factor == 0.0
    s = c.as_struct()
    assert (s.chunk, s.gate, s.qkv_bias, s.head_norm, s.beside, s.kv_from) == (33, _lib.GATE_HEAD, 1, 0, -1, -1)
    assert s.out_scale == pytest.approx(0.6) and b.as_struct().rope_original == 60.0
    assert read_config(tmp_path, "float32").torch_dtype == torch.float32


def test_models_without_a_recurrence_carry_no_state(pkg):
    from sglang_cpp_b200.models import read_saluzen

    assert not read_saluzen(C.config([C.latent(2, 8, 4, 8, 16, 16, 0.3)])).carries_state
    assert read_saluzen(C.config([C.parallel_2(C.attention(2, 1, 8, 8, 0.3, 8, size=4), C.delta(1, 1, 8, 8, 2), 1, 1)])).carries_state


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][1].update(type="parallel_3"), "layer 1: unknown mixer"),
    (lambda c: c["layers"][0].update(mlp={"kind": "moe"}), "layer 0: unknown feed-forward"),
])
def test_registry_refuses_what_it_does_not_know(pkg, change, text):
    from sglang_cpp_b200.models import read_saluzen

    cfg = copy.deepcopy(C.MIXED)
    change(cfg)
    with pytest.raises(ValueError, match=text):
        read_saluzen(cfg)


def test_packing_keeps_every_number_and_pads_with_zeros(pkg, tmp_path):
    from sglang_cpp_b200.models import read_config
    from sglang_cpp_b200.weights import load_checkpoint

    cfg, w = C.model("mixed")
    C.write_checkpoint(tmp_path, cfg, w)
    P = load_checkpoint(read_config(tmp_path, "float32"), tmp_path)
    D, hp = cfg["width"], 192
    f = lambda name: w[name].float()
    total = lambda t: float(t.double().abs().sum())
    same = torch.testing.assert_close

    L = P["layers"][0]                       # latents of 83, 12 rotated dimensions from column 88 on
    assert L["down_qkv"].shape == (128 + 128, hp)
    same(L["down_qkv"][128:211, :D], f("l0.mix.dkv")[:83])
    same(L["down_qkv"][216:228, :D], f("l0.mix.dkv")[83:])
    same(L["uq"][:, :12, :72], f("l0.mix.uq").view(5, 52, 72)[:, 40:])
    same(L["uq"][:, 12:52, :72], f("l0.mix.uq").view(5, 52, 72)[:, :40])
    same(L["uk_absorb"][:, :83, 12:52], f("l0.mix.uk").view(5, 40, 83).transpose(1, 2))
    same(L["uk_absorb"][:, 88:100, :12], torch.eye(12).expand(5, 12, 12))
    assert total(L["uk_absorb"]) == pytest.approx(total(w["l0.mix.uk"]) + 5 * 12)
    assert L["uv"].shape == (5, 128, 128) and total(L["kv_latent_norm"]) == pytest.approx(total(w["l0.mix.dkv.norm"]))
    assert "kv_latent_norm" not in P["layers"][3] and P["layers"][3]["down_qkv"].shape == (192, hp)

    L = P["layers"][1]                       # left 6 over 2 heads of 40 / 56; right 6 heads of 20, 3 groups of 24
    left, right = (6 + 2) * 128 + 2 * 128 + 6 * 128, 2 * 6 * 64 + 2 * 3 * 64 + 64
    assert L["joint"].shape == (left + right, hp) and L["joint_bias"].shape == (left + right,)
    same(L["joint_bias"][768:1024].view(2, 128)[:, :40], f("l1.mix.left.k.b").view(2, 40))
    assert total(L["joint_bias"]) == pytest.approx(sum(total(w[f"l1.mix.left.{n}.b"]) for n in "qkv"), rel=1e-6)
    R, src = L["joint"][left:], f("l1.mix.right.in")
    same(R[:384].view(6, 64, hp)[:, :20, :D], src[:120].view(6, 20, D))                       # gate
    same(R[384:768].view(6, 64, hp)[:, :20, :D], src[120:240].view(6, 20, D))                 # values
    same(R[768:960].view(3, 64, hp)[:, :24, :D], src[240:312].view(3, 24, D))                 # keys
    same(R[960:1152].view(3, 64, hp)[:, :24, :D], src[312:384].view(3, 24, D))                # queries
    same(R[1152:1158, :D], src[384:])                                                         # steps
    assert total(R) == pytest.approx(total(src))
    assert L["beside_conv"].shape == (5, 384 + 384)
    same(L["beside_conv"].T[384:576].view(3, 64, 5)[:, :24], f("l1.mix.right.conv")[120:192].view(3, 24, 5))
    same(L["beside_head_norm"].view(6, 64)[:, :20], f("l1.mix.right.norm").view(6, 20))
    same(L["sinks"], torch.zeros(6))
    assert L["o"].shape == (hp, 6 * 128) and L["beside_o"].shape == (hp, 6 * 64)
    same(L["side_norm"][:D], f("l1.mix.left.out"))
    same(L["norm1_out"][:D], f("l1.norm1b"))
    same(L["norm2_out"][:D], f("l1.norm2b"))

    L = P["layers"][2]                       # left 6 over 3 heads of 36 / 24; right 6 over 3 heads of 24 / 40
    left = (6 + 3) * 128 + 3 * 128 + 64
    same(L["joint"][left - 64:left - 58, :D], f("l2.mix.left.g"))
    R = L["joint"][left:]
    same(R[768:960].view(3, 64, hp)[:, :24, :D], f("l2.mix.right.k").view(3, 24, D))
    same(R[1152:1158, :D], f("l2.mix.right.a"))
    same(R[1158:1164, :D], f("l2.mix.right.b"))
    same(L["beside_conv"].T[576:768].view(3, 64, 2)[:, :24], f("l2.mix.right.q.conv").view(3, 24, 2))
    same(L["sinks"], f("l2.mix.left.sink"))
    assert L["o"].shape == (hp, 6 * 128 + 6 * 64) and "beside_o" not in L and "norm2" not in L
    same(L["o"][:D, 768:].view(D, 6, 64)[..., :40], f("l2.mix.right.o").view(D, 6, 40))


@pytest.mark.parametrize("change, err", [
    (lambda w: w.pop("l2.mix.left.sink"), KeyError),
    (lambda w: w.pop("l1.mix.right.out"), KeyError),
    (lambda w: w.pop("l0.norm2b"), KeyError),
    (lambda w: w.update({"l1.mix.right.in": w["l1.mix.right.in"][:-1]}), ValueError),
    (lambda w: w.update({"l2.mix.right.k.conv": w["l2.mix.right.k.conv"][:, 1:]}), ValueError),
    (lambda w: w.update({"l0.mix.dkv": w["l0.mix.dkv"][:-1]}), ValueError),
])
def test_packing_checks_names_and_shapes(pkg, change, err):
    from sglang_cpp_b200.models import read_saluzen
    from sglang_cpp_b200.weights import pack_layer_stack

    cfg, w = C.model("mixed")
    w = dict(w)
    change(w)
    with pytest.raises(err):
        pack_layer_stack(read_saluzen(cfg, C.shapes_of(w)), w)
