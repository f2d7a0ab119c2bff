"""Retotar without a GPU: the oracle's own consistency, the registry and weight packing."""
import copy
import math

import pytest
import torch

from oracle import retotar_oracle as O
from tests import retotar_cases as C

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


def test_oracle_window_in_words():
    """A window of 3: token 9 sees 7, 8 and itself."""
    seen = O.visible(12, 3)
    assert seen[9].nonzero().flatten().tolist() == [7, 8, 9]
    assert seen[1].nonzero().flatten().tolist() == [0, 1]
    assert O.visible(5)[3].nonzero().flatten().tolist() == [0, 1, 2, 3]


def test_oracle_layer_norm_equals_torchs():
    x, w, b = rand(4, 9), rand(9, seed=1), rand(9, seed=2)
    torch.testing.assert_close(O.layer_normalise(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (9,), w, b, 1e-3))


def test_oracle_rotations_depend_on_distances_only():
    q, k = rand(1, 1, 8), rand(1, 1, 8, seed=1)
    turn = lambda x, p, f=1.0: O.rotate_half(x, torch.tensor([p]), 100.0, 6, f)
    dot = lambda i, j: (turn(q, i) * turn(k, j)).sum()
    torch.testing.assert_close(dot(9, 4), dot(105, 100))
    torch.testing.assert_close(turn(q, 7)[..., 6:], q[..., 6:])
    torch.testing.assert_close(turn(q, 12, 4.0), turn(q, 3))
    e = torch.zeros(1, 1, 8, dtype=F64)
    e[..., 0] = 1
    assert turn(e, 1).nonzero()[:, 2].tolist() == [0, 3]


def test_oracle_turned_values_depend_on_distances_only():
    """What a query gets from a value is the value turned by their distance, wherever the two are."""
    v = rand(1, 1, 6)
    turn = lambda x, p: O.rotate_half(x, torch.tensor([p]), 50.0, 6)
    torch.testing.assert_close(turn(turn(v, 9), -11), turn(turn(v, 109), -111))
    torch.testing.assert_close(turn(turn(v, 5), -5), v)


def test_oracle_heads_mix_before_they_meet_the_values():
    p, v = torch.softmax(rand(4, 3, 5), -1), rand(5, 2, 7, seed=1)
    mix = rand(4, 4, seed=2)
    got = O.weighted_values(O.talking_heads(p, mix), v)
    want = sum(mix[3, g] * (p[g, 1] @ v[:, 1]) for g in range(4))      # head 3 has the second value head
    torch.testing.assert_close(got[1, 3], want)
    torch.testing.assert_close(O.talking_heads(p, torch.eye(4, dtype=F64)), p)


def test_oracle_recurrences_continue_from_their_state():
    q, k, v = rand(9, 2, 5), rand(9, 2, 5, seed=1), rand(9, 2, 3, seed=2)
    i, f = 3 * rand(9, 2, seed=3), -torch.rand(9, 2, dtype=F64)
    decay = torch.tensor([0.9, 0.2], dtype=F64)
    for step in (lambda s, S: O.decayed_recurrence(q[s], k[s], v[s], decay, S), lambda s, S: O.matrix_memory(q[s], k[s], v[s], i[s], f[s], S)):
        whole, last = step(slice(0, 9), None)
        a, mid = step(slice(0, 4), None)
        b, end = step(slice(4, 9), mid)
        torch.testing.assert_close(torch.cat([a, b]), whole)
        torch.testing.assert_close(end, last)


def test_oracle_matrix_memory_equals_its_sum_over_the_past():
    """Without the running maximum: sums with weights exp(i_s + f_s+1 + .. + f_t), and a denominator that is at least 1."""
    q, k, v = rand(7, 1, 4), rand(7, 1, 4, seed=1), rand(7, 1, 3, seed=2)
    i, f = rand(7, 1, seed=3), -torch.rand(7, 1, dtype=F64)
    got, (_, _, m) = O.matrix_memory(q, k, v, i, f)
    for t in range(7):
        w = [torch.exp(i[s, 0] + f[s + 1:t + 1, 0].sum()) * (q[t, 0] @ k[s, 0]) for s in range(t + 1)]
        num, den = sum(w[s] * v[s, 0] for s in range(t + 1)), sum(w)
        torch.testing.assert_close(got[t, 0], num / max(abs(den), 1.0), rtol=1e-4, atol=1e-4)
    assert float(m) >= float(f.sum())                                   # (the maximum starts at 0)


def test_oracle_lightning_equals_its_sum_over_the_past():
    q, k, v = rand(6, 1, 4), rand(6, 1, 4, seed=1), rand(6, 1, 3, seed=2)
    got, _ = O.decayed_recurrence(q, k, v, torch.tensor([0.7], dtype=F64))
    want = sum(0.7 ** (5 - s) * (k[s, 0] @ q[5, 0]) * v[s, 0] for s in range(6))
    torch.testing.assert_close(got[5, 0], want)


def test_oracle_routing_in_words():
    r = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    z = torch.log(torch.tensor([0.30, 0.02, 0.25, 0.2, 0.13, 0.10], dtype=F64))
    none = torch.zeros(6, dtype=F64)
    ids, weights = O.route(z, none, r)
    assert ids == [0, 1]                                               # the pair that holds the best, not the best two
    torch.testing.assert_close(weights, torch.tensor([0.30, 0.02], dtype=F64))
    lift = none.clone()
    lift[5] = 0.5                                                      # (of the choice alone)
    ids, weights = O.route(z, lift, r)
    assert ids == [5, 4]
    torch.testing.assert_close(weights, torch.tensor([0.10, 0.13], dtype=F64))
    ids, _ = O.route(z, none - 5.0, {**r, "groups": {"count": 3, "keep": 2}})
    assert ids == [0, 2]                                               # scores below zero still beat what is out


def test_oracle_identity_experts_return_their_input():
    r = {"experts": 1, "identity": 1, "top": 1, "groups": {"count": 1, "keep": 1}}
    h = rand(3, 4)
    w = {"router": torch.zeros(2, 4, dtype=F64), "correction": torch.tensor([0.0, 1.0], dtype=F64)}
    torch.testing.assert_close(O.experts_ff(h, w, "", r), 0.5 * h)


def test_random_models_leave_no_choice_close():
    cfg, w = C.model("mixed")
    ids = C.prompt(cfg, 30, 4)
    a = O.forward(cfg, w, ids, torch.float64)
    b = O.forward(cfg, w, ids, torch.float32)
    assert float((a - b).abs().max()) < 1e-3


# ---- registry and weights ----------------------------------------------------------
def test_registry_reads_every_layer(pkg, tmp_path):
    from sglang_cpp_b200 import _lib
    from sglang_cpp_b200.models import NO_WINDOW, StackConfig, read_config

    C.write_checkpoint(tmp_path, *C.model("mixed"))
    cfg = read_config(tmp_path)
    assert isinstance(cfg, StackConfig) and (cfg.num_layers, cfg.hidden_size, cfg.vocab_size) == (8, 136, 203)
    assert (cfg.norm_output, cfg.norm_kind, cfg.embed_scale, cfg.rms_norm_eps) == (_lib.NORM_BOTH, _lib.NORM_LAYER, 0.7, 1e-5)
    assert cfg.carries_state
    a, b, c, d, e, f, g, h = cfg.layers
    assert (a.mixer, a.heads, a.kv_heads, a.head_dim, a.value_dim, a.score_scale) == (_lib.MIXER_WINDOW_ATTENTION, 6, 2, 40, 56, 0.2)
    assert (a.window, a.rotary_dim, a.rope_base, a.rope_factor, a.rope_original) == (33, 24, 900.0, 3.0, 0.0)
    assert (a.head_norm, a.value_rotary, a.head_mix, a.gate, a.kv_from) == (_lib.HEAD_NORM_UNIT, True, True, _lib.GATE_ELEMENT, -1)
    assert (c.kv_from, c.window, c.score_scale, c.mlp) == (0, 9, -0.15, _lib.MLP_NONE)
    assert (e.window, e.rope_factor) == (NO_WINDOW, 0.0)
    assert (a.mlp, a.intermediate, a.epilogue, a.score) == (_lib.MLP_SCORED_MOE, 52, _lib.EPILOGUE_SWIGLU, _lib.SCORE_SOFTMAX)
    assert (a.num_experts, a.identity_experts, a.experts_per_tok, a.router_groups, a.router_keep, a.shared_intermediate) == (7, 2, 3, 3, 2, 0)
    assert e.identity_experts == 0
    assert (b.mixer, b.heads, b.kv_heads, b.head_dim, b.value_dim, b.gate_cap, b.norm_groups) == (
        _lib.MIXER_MATRIX_MEMORY, 3, 3, 24, 72, 4.0, 3)
    assert (d.mixer, d.heads, d.norm_groups, d.decays) == (_lib.MIXER_LIGHTNING, 5, 1, (0.3, 1.0, 0.97, 0.5, 0.9))
    s = c.as_struct()
    assert (s.kv_from, s.value_rotary, s.head_mix, s.head_norm, s.window) == (0, 1, 1, 2, 9)
    s = b.as_struct()
    assert (s.mixer, s.gate_cap, s.identity_experts, s.score) == (6, 4.0, 1, 1)
    assert read_config(tmp_path, "float32").torch_dtype == torch.float32


def test_models_without_a_recurrence_carry_no_state(pkg):
    from sglang_cpp_b200.models import read_retotar

    assert not read_retotar(C.config([C.attention(2, 1, 8, 8, 0.3, 4, 8)])).carries_state
    assert read_retotar(C.config([C.lightning((0.5,), 8, 8)])).carries_state
    assert read_retotar(C.config([C.mlstm(1, 8, 8, 3.0)])).carries_state


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][1].update(type="gru"), "layer 1: unknown mixer"),
    (lambda c: c["layers"][0].update(mlp={"kind": "dense"}), "layer 0: unknown feed-forward"),
    (lambda c: c["layers"][3]["mixer"]["decay"].pop(), "layer 3: 4 decays for 5 heads"),
])
def test_registry_refuses_what_it_does_not_know(pkg, change, text):
    from sglang_cpp_b200.models import read_retotar

    cfg = copy.deepcopy(C.MIXED)
    change(cfg)
    with pytest.raises(ValueError, match=text):
        read_retotar(cfg)


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
    same(P["final_norm_bias"][:D], f("final.norm.b"))

    L = P["layers"][0]                       # 6 over 2 heads of 40 / 56
    assert L["qkvg"].shape == ((6 + 2) * 128 + 2 * 128 + 6 * 128, hp)
    same(L["qkvg"][768:1024].view(2, 128, hp)[:, :40, :D], f("l0.mix.k").view(2, 40, D))
    same(L["qkvg"][1280:].view(6, 128, hp)[:, :56, :D], f("l0.mix.g").view(6, 56, D))
    assert total(L["qkvg"]) == pytest.approx(sum(total(w[f"l0.mix.{n}"]) for n in "qkvg"))
    same(L["head_mix"], f("l0.mix.talk"))
    for to, name in (("norm1", "norm1"), ("norm1_out", "norm1b"), ("norm2", "norm2"), ("norm2_out", "norm2b")):
        same(L[to][:D], f("l0." + name))
        same(L[to + "_bias"][:D], f(f"l0.{name}.b"))
        assert total(L[to + "_bias"]) == pytest.approx(total(w[f"l0.{name}.b"]))
    assert L["router"].shape == (64, hp) and L["mlp_up"].shape == (7, 128, hp)
    same(L["router"][:9, :D], f("l0.mlp.router"))
    same(L["router_correction"], f("l0.mlp.correction"))
    assert "q_head_norm" not in L

    L = P["layers"][1]                       # 3 heads of 24 / 72
    R = L["recurrence"]
    assert R.shape == (2 * 3 * 128 + 2 * 3 * 64 + 64, hp)
    same(R[:384].view(3, 128, hp)[:, :72, :D], f("l1.mix.g").view(3, 72, D))
    same(R[384:768].view(3, 128, hp)[:, :72, :D], f("l1.mix.v").view(3, 72, D))
    same(R[768:960].view(3, 64, hp)[:, :24, :D], f("l1.mix.k").view(3, 24, D))
    same(R[960:1152].view(3, 64, hp)[:, :24, :D], f("l1.mix.q").view(3, 24, D))
    same(R[1152:1155, :D], f("l1.mix.i"))
    same(R[1155:1158, :D], f("l1.mix.f"))
    assert total(R) == pytest.approx(sum(total(w[f"l1.mix.{n}"]) for n in "gvkqif"))
    same(L["step_bias"], torch.cat([f("l1.mix.i.b"), f("l1.mix.f.b")]))
    same(L["head_norm"].view(3, 128)[:, :72].float(), f("l1.mix.norm").view(3, 72))

    L = P["layers"][2]                       # keys and values of layer 0
    assert L["qkvg"].shape == (6 * 128 + 6 * 128, hp)
    same(L["qkvg"][768:].view(6, 128, hp)[:, :56, :D], f("l2.mix.g").view(6, 56, D))

    L = P["layers"][3]
    assert L["recurrence"].shape == (2 * 5 * 64 + 2 * 5 * 128, hp) and "step_bias" not in L
    same(L["decay_log"], torch.tensor([math.log(x) for x in (0.3, 1.0, 0.97, 0.5, 0.9)]))


@pytest.mark.parametrize("change, err", [
    (lambda w: w.pop("l0.mix.talk"), KeyError),
    (lambda w: w.pop("l0.norm2b.b"), KeyError),
    (lambda w: w.pop("l1.mix.f.b"), KeyError),
    (lambda w: w.update({"l0.mlp.correction": w["l0.mlp.correction"][:-1]}), ValueError),
    (lambda w: w.update({"l1.mix.norm": w["l1.mix.norm"][:-1]}), ValueError),
    (lambda w: w.update({"l3.mix.v": w["l3.mix.v"][:-1]}), ValueError),
])
def test_packing_checks_names_and_shapes(pkg, change, err):
    from sglang_cpp_b200.models import read_retotar
    from sglang_cpp_b200.weights import pack_layer_stack

    cfg, w = C.model("mixed")
    w = dict(w)
    change(w)
    with pytest.raises(err):
        pack_layer_stack(read_retotar(cfg, C.shapes_of(w)), w)
