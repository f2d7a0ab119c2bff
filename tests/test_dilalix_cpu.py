"""Dilalix without a GPU: the oracle's own consistency, the registry, weight packing and request bookkeeping."""
import copy
import json

import pytest
import torch

from oracle import dilalix_oracle as O
from tests import dilalix_cases as C


# ---- the oracle -----------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_oracle_is_causal_and_its_decode_equals_its_prefill(name):
    cfg, w = C.model(name)
    ids = C.prompt(cfg, 60, 1)
    full = O.forward(cfg, w, ids)
    for n in (1, 2, 35, 59):
        torch.testing.assert_close(O.forward(cfg, w, ids[:n]), full[:n])
    other = ids[:40] + [(t + 1) % cfg["vocab"] for t in ids[40:]]
    torch.testing.assert_close(O.forward(cfg, w, other)[:40], full[:40])


def test_oracle_window_in_words():
    """Query 10 through a window of 4 that keeps 2: itself and three before it, and the first two."""
    assert O.visible(12, 4, 2)[10].nonzero().flatten().tolist() == [0, 1, 7, 8, 9, 10]
    assert O.visible(12, 4, 2)[1].nonzero().flatten().tolist() == [0, 1]
    assert O.visible(12, 1, 0)[5].nonzero().flatten().tolist() == [5]
    assert O.visible(6, 100, 0)[5].tolist() == [True] * 6


def test_oracle_recurrence_equals_its_sum_over_the_past():
    """o_t = sum_s (q_t . prod of decays . k_s) v_s, and a state handed on continues it."""
    g = torch.Generator().manual_seed(0)
    n, H, d, dv = 9, 2, 5, 3
    q, k, v = (torch.randn(n, H, m, generator=g, dtype=torch.float64) for m in (d, d, dv))
    ld = -torch.rand(n, H, d, generator=g, dtype=torch.float64)
    got, last = O.linear_recurrence(q, k, v, ld)
    b = ld.cumsum(0)
    for t in range(n):
        want = sum(((q[t] * k[s] * torch.exp(b[t] - b[s])).sum(-1, keepdim=True) * v[s]) for s in range(t + 1))
        torch.testing.assert_close(got[t], want)
    a, mid = O.linear_recurrence(q[:4], k[:4], v[:4], ld[:4])
    b, end = O.linear_recurrence(q[4:], k[4:], v[4:], ld[4:], mid)
    torch.testing.assert_close(torch.cat([a, b]), got)
    torch.testing.assert_close(end, last)


def test_oracle_groups_count_for_their_two_best():
    """Group 0 has the single best expert, group 1 the best pair; with one group kept the pair wins."""
    s = torch.tensor([[0.9, 0.1, 0.2, 0.6, 0.7, 0.1]])
    ids, weights = O.choose_experts(s, 2, 2, 1, 3.0)
    assert sorted(ids[0].tolist()) == [3, 4]
    torch.testing.assert_close(weights.sum(), torch.tensor(3.0))
    torch.testing.assert_close(weights[0], s[0][ids[0]] / 1.3 * 3)
    ids, _ = O.choose_experts(s, 2, 2, 2, 3.0)
    assert sorted(ids[0].tolist()) == [0, 4]
    ids, _ = O.choose_experts(s, 1, 6, 2, 1.0)      # groups of one expert
    assert ids[0].tolist() == [0]


def test_oracle_experts_clamp_one_side_of_the_gate_and_both_of_the_other():
    eye = torch.eye(1, dtype=torch.float64)
    w = {"e.gate": eye, "e.up": eye, "e.down": eye}
    for x, (g, u) in {5.0: (2.0, 2.0), -5.0: (-5.0, -2.0), 0.5: (0.5, 0.5)}.items():
        g, u = torch.tensor(g, dtype=torch.float64), torch.tensor(u, dtype=torch.float64)
        got = O.clamped_ff(torch.full((1, 1), x, dtype=torch.float64), w, "e.", 2.0)
        torch.testing.assert_close(got[0, 0], g * torch.sigmoid(1.702 * g) * (u + 1))


# ---- registry and weights ----------------------------------------------------------
def test_registry_reads_every_layer(pkg, tmp_path):
    from sglang_cpp_b200 import _lib
    from sglang_cpp_b200.models import StackConfig, read_config

    C.write_checkpoint(tmp_path, *C.model("mixed"))
    cfg = read_config(tmp_path)
    assert isinstance(cfg, StackConfig) and cfg.num_layers == 6 and cfg.hidden_size == 136 and cfg.vocab_size == 203
    assert cfg.norm_output and cfg.norm_offset == 0.0 and cfg.rms_norm_eps == 1e-5 and cfg.carries_state
    a, b, c, d, e, f = cfg.layers
    assert (a.mixer, a.heads, a.kv_heads, a.head_dim, a.value_dim) == (_lib.MIXER_WINDOW_ATTENTION, 6, 2, 40, 56)
    assert (a.score_scale, a.window, a.keep_first, a.rotary_dim, a.rope_base, a.value_mix) == (0.2, 33, 3, 24, 5000.0, True)
    assert (a.mlp, a.epilogue) == (_lib.MLP_SCORED_MOE, _lib.EPILOGUE_CLAMPED_SWIGLU)
    assert (a.num_experts, a.experts_per_tok, a.router_groups, a.router_keep, a.router_scale) == (12, 3, 4, 2, 1.7)
    assert (a.intermediate, a.act_limit, a.shared_intermediate, a.shared_act_limit) == (52, 0.8, 80, 1.3)
    assert (b.mixer, b.decay_tau, b.decay_rank, b.mlp) == (_lib.MIXER_LINEAR_ATTENTION, 8.0, 10, _lib.MLP_NONE)
    assert (c.mlp, c.epilogue, c.intermediate, c.value_mix) == (_lib.MLP_DENSE, _lib.EPILOGUE_GELU_ERF, 90, False)
    assert d.decay_rank == 33 and d.shared_intermediate == 0 and e.keep_first == 70 and f.decay_rank == 70
    assert read_config(tmp_path, "float32").torch_dtype == torch.float32
    s = a.as_struct()
    assert (s.kv_heads, s.window, s.value_mix, s.router_keep) == (2, 33, 1, 2) and s.rope_base == 5000.0


def test_what_a_configuration_leaves_out_is_off(pkg):
    from sglang_cpp_b200.models import NO_WINDOW, read_dilalix

    m = {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.5}
    cfg = read_dilalix(C.config([{"type": "attention", "mixer": m}]))
    a = cfg.layers[0]
    assert (a.window, a.keep_first, a.rotary_dim, a.value_mix, a.mlp) == (NO_WINDOW, 0, 0, False, 0)
    assert not cfg.carries_state


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][1].update(type="window"), "layer 1: unknown mixer"),
    (lambda c: c["layers"][0].update(mlp={"kind": "other"}), "layer 0: unknown feed-forward"),
])
def test_registry_refuses_what_it_does_not_know(pkg, change, text):
    from sglang_cpp_b200.models import read_dilalix

    cfg = copy.deepcopy(C.MIXED)
    change(cfg)
    with pytest.raises(ValueError, match=text):
        read_dilalix(cfg, C.shapes_of(C.model("mixed")[1]))


def test_the_rank_of_the_decay_comes_from_the_checkpoint(pkg):
    from sglang_cpp_b200.models import read_dilalix

    with pytest.raises(ValueError, match="l1.mix.a1"):
        read_dilalix(C.MIXED)


def test_packing_pads_with_zeros_and_keeps_every_number(pkg, tmp_path):
    from sglang_cpp_b200.models import read_config
    from sglang_cpp_b200.weights import load_checkpoint

    cfg, w = C.model("mixed")
    C.write_checkpoint(tmp_path, cfg, w)
    P = load_checkpoint(read_config(tmp_path, "float32"), tmp_path)
    D, hp = cfg["width"], 192
    f = lambda name: w[name].float()
    L = P["layers"][0]                       # 6 heads over 2, 40 / 56 wide
    assert L["qkvg"].shape == (6 * 128 + 2 * 128 + 2 * 128 + 6 * 128, hp)
    torch.testing.assert_close(L["qkvg"][:768].view(6, 128, hp)[:, :40, :D], f("l0.mix.q").view(6, 40, D))
    torch.testing.assert_close(L["qkvg"][768:1024].view(2, 128, hp)[:, :40, :D], f("l0.mix.k").view(2, 40, D))
    torch.testing.assert_close(L["qkvg"][1024:1280].view(2, 128, hp)[:, :56, :D], f("l0.mix.v").view(2, 56, D))
    torch.testing.assert_close(L["qkvg"][1280:].view(6, 128, hp)[:, :56, :D], f("l0.mix.g").view(6, 56, D))
    assert float(L["qkvg"].double().abs().sum()) == pytest.approx(
        sum(float(w[f"l0.mix.{n}"].double().abs().sum()) for n in "qkvg"))
    assert float(L["value_mix"]) == float(w["l0.mix.vmix"]) and L["value_mix"].dtype == torch.float32
    assert "value_mix" not in P["layers"][2]
    assert L["mlp_up"].shape == (12, 2 * 64, hp) and L["router"].shape == (64, hp) and L["shared_up"].shape == (2 * 128, hp)
    torch.testing.assert_close(L["mlp_up"][11, 64:116, :D], f("l0.mlp.e11.up"))
    torch.testing.assert_close(L["shared_up"][:80, :D], f("l0.mlp.shared.gate"))
    torch.testing.assert_close(L["shared_down"][:D, :80], f("l0.mlp.shared.down"))
    torch.testing.assert_close(L["router"][:12, :D], f("l0.mlp.router"))
    L = P["layers"][1]                       # 3 heads of 24 / 72, rank 10
    assert L["qkvga"].shape == (2 * 3 * 64 + 2 * 3 * 128 + 64, hp) and L["decay_up"].shape == (3 * 64, 16)
    torch.testing.assert_close(L["qkvga"][-64:-54, :D], f("l1.mix.a1"))
    torch.testing.assert_close(L["decay_up"].view(3, 64, 16)[:, :24, :10], f("l1.mix.a2").view(3, 24, 10))
    torch.testing.assert_close(L["decay_bias"][:, :24], f("l1.mix.a2.b").view(3, 24))
    assert "norm2" not in L
    L = P["layers"][2]
    assert L["mlp_up"].shape == (128, hp) and "shared_up" not in P["layers"][3]
    torch.testing.assert_close(L["o"][:D, :, :24], f("l2.mix.o").view(D, 5, 24))


@pytest.mark.parametrize("change, err", [
    (lambda w: w.pop("l0.mix.vmix"), KeyError),
    (lambda w: w.pop("l0.mlp.shared.up"), KeyError),
    (lambda w: w.update({"l1.mix.a2": w["l1.mix.a2"][:, :-1]}), ValueError),
    (lambda w: w.update({"l0.mlp.router": w["l0.mlp.router"][:-1]}), ValueError),
])
def test_packing_checks_names_and_shapes(pkg, change, err):
    from sglang_cpp_b200.models import read_dilalix
    from sglang_cpp_b200.weights import pack_layer_stack

    cfg, w = C.model("mixed")
    w = dict(w)
    change(w)
    with pytest.raises(err):
        pack_layer_stack(read_dilalix(cfg, C.shapes_of(w)), w)


def test_scalars_survive_safetensors(pkg, tmp_path):
    from sglang_cpp_b200.weights import read_safetensors, tensor_shapes, write_safetensors

    t = {"lambda": torch.tensor(0.25).bfloat16(), "w": torch.randn(2, 3).bfloat16()}
    write_safetensors(tmp_path / "x.safetensors", t)
    back = read_safetensors(tmp_path / "x.safetensors")
    assert back["lambda"].shape == () and float(back["lambda"]) == 0.25
    assert tensor_shapes(tmp_path) == {"lambda": (), "w": (2, 3)}


# ---- requests ------------------------------------------------------------------------
class FakeEngine:
    dummy_table_idx = 2
    pt_cols = 256

    def __init__(self, carries_state):
        self.carries_state = carries_state

    def write_page_table(self, *a):
        pass

    def write_token_pool(self, *a):
        pass


@pytest.mark.parametrize("carries_state", [False, True])
def test_prefixes_are_not_shared_between_requests_that_carry_a_state(pkg, carries_state):
    """The pages of a prefix hold its keys and values, but not what its tokens left in a state."""
    from sglang_cpp_b200.host_batch import HostBatcher, HostScheduler

    shared = list(range(64))
    sched = HostScheduler(FakeEngine(carries_state), 16, 16, 2, 256, 512)
    for uid in (0, 1):
        sched.submit(uid, shared + [uid], 2)
        while True:
            batch = sched.next_batch()
            if batch is None:
                break
            sched.finish_batch(batch, [7] * len(batch.reqs))
    assert sched.prefix_hits == (0 if carries_state else 64)
    assert len(sched.cache_manager.free_pages) == (16 if carries_state else 12)
    hb = HostBatcher(FakeEngine(carries_state), 16, 16, 2)
    assert hb.cache_manager.enabled is not carries_state


def test_configuration_files_are_plain_json():
    for cfg in C.CONFIGS.values():
        assert json.loads(json.dumps(cfg)) == cfg
