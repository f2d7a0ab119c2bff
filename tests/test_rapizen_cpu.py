"""Rapizen without a GPU: the oracle's own consistency, the registry, weight packing, request bookkeeping
and the trace replay's step handling."""
import copy
import json

import numpy as np
import pytest
import torch

from oracle import rapizen_oracle as O
from tests import rapizen_cases as C


# ---- the oracle -----------------------------------------------------------------
def test_oracle_is_causal_and_its_decode_equals_its_prefill():
    cfg, w = C.model("mixed")
    ids = C.prompt(cfg, 12, 1)
    full = O.forward(cfg, w, ids)
    for n in (1, 2, 7, 11):
        torch.testing.assert_close(O.forward(cfg, w, ids[:n]), full[:n])
    other = ids[:8] + [(t + 1) % cfg["vocab"] for t in ids[8:]]
    torch.testing.assert_close(O.forward(cfg, w, other)[:8], full[:8])


def test_oracle_attention_equals_its_latent_space_form():
    """q . (U c) == (U^T q) . c and sum p (V c) == V sum p c."""
    cfg, w = C.model("mixed")
    m, eps, p = cfg["layers"][2]["mixer"], 1e-5, "l2.mix."
    w = {k: t.double() for k, t in w.items() if k.startswith(p)}
    h = torch.randn(9, cfg["width"], generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    want = O.latent_attention(h, w, p, m, eps)
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    cq, c = O.latent_of(h, w, p + "dq", eps), O.latent_of(h, w, p + "dkv", eps)
    q = (cq @ w[p + "uq"].T).view(-1, H, d)
    qa = torch.einsum("ihd,hdr->ihr", q, w[p + "uk"].view(H, d, -1))
    s = torch.einsum("ihr,jr->hij", qa, c) * m["scale"]
    s = s.masked_fill(torch.ones(9, 9, dtype=torch.bool).triu(1), float("-inf"))
    o = torch.einsum("hij,jr->ihr", torch.softmax(s, -1), c)
    o = torch.einsum("ihr,hvr->ihv", o, w[p + "uv"].view(H, dv, -1)).reshape(9, -1)
    torch.testing.assert_close(o @ w[p + "o"].T, want)


def test_oracle_experts_follow_the_table_not_the_activations():
    cfg, w = C.model("mixed")
    top, p = 3, "l0.mlp."
    w64 = {k: (t if t.dtype == torch.int32 else t.double()) for k, t in w.items()}
    h = torch.randn(4, cfg["width"], dtype=torch.float64, generator=torch.Generator().manual_seed(3))
    tok = torch.tensor([5, 9, 5, 0])
    got = O.table_moe(h, tok, w64, p, top)
    for i in range(4):
        want = sum(O.expert_ff(h[i:i + 1], w64, f"{p}e{int(e)}.") for e in w[p + "table"][tok[i]]) / top
        torch.testing.assert_close(got[i:i + 1], want)


# ---- registry and weights ----------------------------------------------------------
def test_registry_reads_every_layer(pkg, tmp_path):
    from sglang_cpp_b200 import _lib
    from sglang_cpp_b200.models import StackConfig, read_config

    (tmp_path / "config.json").write_text(json.dumps(C.MIXED))
    cfg = read_config(tmp_path)
    assert isinstance(cfg, StackConfig) and cfg.num_layers == 5 and cfg.hidden_size == 136
    assert cfg.norm_offset == 1.0 and cfg.logit_scale == 0.7 and cfg.rms_norm_eps == 1e-5
    a, b, c, d, e = cfg.layers
    assert (a.heads, a.head_dim, a.value_dim, a.q_rank, a.kv_rank, a.score_scale) == (5, 40, 56, 72, 80, 0.16)
    assert (a.mlp, a.num_experts, a.experts_per_tok, a.intermediate) == (_lib.MLP_TABLE_MOE, 7, 3, 52)
    assert a.epilogue == _lib.EPILOGUE_RELU2 and c.epilogue == _lib.EPILOGUE_GEGLU
    assert b.mlp == _lib.MLP_NONE and c.mlp == _lib.MLP_DENSE and d.experts_per_tok == 1 and e.heads == 18
    assert read_config(tmp_path, "float32").torch_dtype == torch.float32


@pytest.mark.parametrize("change, text", [
    (lambda c: c.update(architecture="Nothing"), "unknown architecture"),
    (lambda c: c["layers"][1].update(type="window"), "layer 1: unknown mixer"),
    (lambda c: c["layers"][0].update(mlp={"kind": "other"}), "layer 0: unknown feed-forward"),
])
def test_registry_refuses_what_it_does_not_know(pkg, tmp_path, change, text):
    from sglang_cpp_b200.models import read_config

    cfg = copy.deepcopy(C.MIXED)
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(ValueError, match=text):
        read_config(tmp_path)


def test_registry_reads_the_uniform_models_too(pkg, tmp_path):
    from sglang_cpp_b200.models import ModelConfig, read_config

    raw = {"architectures": ["Qwen3MoeForCausalLM"], "num_hidden_layers": 2, "hidden_size": 256, "num_attention_heads": 4,
           "num_key_value_heads": 2, "head_dim": 128, "intermediate_size": 512, "vocab_size": 1024, "num_experts": 8,
           "num_experts_per_tok": 2, "moe_intermediate_size": 128, "rope_theta": 1e6}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg = read_config(tmp_path)
    assert isinstance(cfg, ModelConfig) and cfg.qk_norm and cfg.fused_residual and cfg.num_experts == 8
    raw["architectures"] = ["Qwen2ForCausalLM"]
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg = read_config(tmp_path)
    assert cfg.attention_bias and not cfg.qk_norm and cfg.num_experts == 0
    with pytest.raises(ValueError, match="float32"):
        read_config(tmp_path, "float32")


def test_packing_pads_with_zeros_and_keeps_every_number(pkg, tmp_path):
    from sglang_cpp_b200.models import read_config
    from sglang_cpp_b200.weights import load_checkpoint

    cfg, w = C.model("mixed")
    C.write_checkpoint(tmp_path, cfg, w)
    P = load_checkpoint(read_config(tmp_path, "float32"), tmp_path)
    D, hp = cfg["width"], 192
    assert P["embed"].shape == (256, hp) and P["lm_head"].shape == (256, hp)
    torch.testing.assert_close(P["embed"][:203, :D], w["embed"].float())
    assert float(P["embed"][203:].abs().sum()) == 0 and float(P["embed"][:, D:].abs().sum()) == 0
    L = P["layers"][0]                       # 5 heads of 40 / 56, latents 72 / 80
    assert L["down_qkv"].shape == (128 + 128, hp)
    torch.testing.assert_close(L["down_qkv"][:72, :D], w["l0.mix.dq"].float())
    torch.testing.assert_close(L["down_qkv"][128:208, :D], w["l0.mix.dkv"].float())
    assert L["uq"].shape == (5, 128, 128) and L["uk_absorb"].shape == (5, 128, 128) and L["o"].shape == (hp, 5, 128)
    uk = w["l0.mix.uk"].float().view(5, 40, 80)
    torch.testing.assert_close(L["uk_absorb"][:, :80, :40], uk.transpose(1, 2))
    torch.testing.assert_close(L["o"][:D, :, :56], w["l0.mix.o"].float().view(D, 5, 56))
    assert L["mlp_up"].shape == (7, 64, hp) and L["mlp_down"].shape == (7, hp, 64)
    torch.testing.assert_close(L["mlp_up"][6, :52, :D], w["l0.mlp.e6.up"].float())
    assert torch.equal(L["expert_table"], w["l0.mlp.table"]) and L["expert_table"].dtype == torch.int32
    assert "norm2" not in P["layers"][1] and "mlp_up" not in P["layers"][1]
    assert P["layers"][2]["mlp_up"].shape == (2 * 128, hp)
    torch.testing.assert_close(P["layers"][2]["mlp_up"][128:218, :D], w["l2.mlp.up"].float())


@pytest.mark.parametrize("change, err", [
    (lambda w: w.pop("l2.mix.uv"), KeyError),
    (lambda w: w.update({"l0.mix.dq": w["l0.mix.dq"][:-1]}), ValueError),
    (lambda w: w.update({"l0.mlp.table": w["l0.mlp.table"] + 5}), ValueError),
])
def test_packing_checks_names_shapes_and_tables(pkg, tmp_path, change, err):
    from sglang_cpp_b200.models import read_rapizen
    from sglang_cpp_b200.weights import pack_layer_stack

    cfg, w = C.model("mixed")
    w = dict(w)
    change(w)
    with pytest.raises(err):
        pack_layer_stack(read_rapizen(cfg), w)


def test_int32_tables_survive_safetensors(pkg, tmp_path):
    from sglang_cpp_b200.weights import read_safetensors, write_safetensors

    t = {"table": torch.arange(6, dtype=torch.int32).view(3, 2), "w": torch.randn(2, 3).bfloat16()}
    write_safetensors(tmp_path / "x.safetensors", t)
    back = read_safetensors(tmp_path / "x.safetensors")
    assert torch.equal(back["table"], t["table"]) and torch.equal(back["w"], t["w"])


# ---- requests fed in portions --------------------------------------------------------
class FakeEngine:
    dummy_table_idx = 2
    pt_cols = 256

    def __init__(self):
        self.steps = []

    def write_page_table(self, *a):
        pass

    def write_token_pool(self, *a):
        pass

    def forward_batch(self, phase, table_idx, cached, extend, write_pos=None, **kw):
        self.steps.append((phase, list(table_idx), list(cached), list(extend)))
        return self

    def synchronize(self):
        pass


def test_portions_pages_and_rows_are_handed_out_and_given_back(pkg):
    from sglang_cpp_b200.host_batch import HostBatcher

    eng = FakeEngine()
    hb = HostBatcher(eng, 4, 64, 2, enable_prefix_cache=False)
    a, b = hb.open_request(256), hb.open_request(256)
    hb.extend([a, b], [list(range(63)), [1, 2]])
    hb.extend([b, a], [[3], [9]])               # a reaches its page's last slot
    hb.extend([a], [[10]])                      # and crosses into the next
    assert [s[0] for s in eng.steps] == [0, 1, 1]
    assert eng.steps[1][2:] == ([2, 63], [1, 1])
    assert hb.pages_held(a) == 2 and hb.pages_held(b) == 1 and len(hb.cache_manager.free_pages) == 1
    rows = hb.tables.page_table
    assert rows[a.table_idx, 64] % 64 == 0 and rows[a.table_idx, 63] % 64 == 63
    hb.release(a)
    assert len(hb.cache_manager.free_pages) == 3 and hb.table_manager.available_size() == 1
    c = hb.open_request(256)
    hb.extend([c, b], [list(range(129)), [4]])  # the freed pages, a portion beside a single token
    assert eng.steps[-1][0] == 0 and hb.pages_held(c) == 3
    hb.release(b)
    hb.release(c)
    assert sorted(hb.cache_manager.free_pages) == [0, 64, 128, 192]
    with pytest.raises(ValueError, match="can take"):
        d = hb.open_request(3)
        hb.extend([d], [[1, 2, 3, 4]])


def test_replay_reports_every_step_and_writes_only_what_is_wanted(pkg, tmp_path):
    from sglang_cpp_b200.trace import replay

    class Run:
        def step(self, entries, end):
            want = sum(len(e["want"]) for e in entries)
            return np.full((want, 3), len(entries), np.float32)

    lines = [json.dumps({"step": 4, "entries": [{"id": "a", "tokens": [1, 2], "want": [0, 1]}], "end": []}), "",
             json.dumps({"step": 5, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": ["a"]})]
    done = []
    replay(lines, tmp_path / "out", Run(), done.append)
    assert done == [4, 5]
    assert np.fromfile(tmp_path / "out" / "4.f32", "<f4").tolist() == [1.0] * 6
    assert not (tmp_path / "out" / "5.f32").exists()
