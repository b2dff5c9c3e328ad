"""Pudizen's configuration and plan: what config.json says is what the parts are built with."""

import copy

import pytest
import torch

import plain_pudizen as PP
import pudizen_configs as PC
from ninfer_amd_mi50_b200.config.model_config import ConfigError
from ninfer_amd_mi50_b200.engine.loading import build_model
from ninfer_amd_mi50_b200.registry import architecture_names


def test_the_design_is_registered():
    assert "Pudizen" in architecture_names()


@pytest.mark.parametrize("name", sorted(PC.CONFIGS))
def test_what_each_layer_keeps_and_which_tensors_it_names(name):
    cfg, _ = PC.CONFIGS[name]
    typed, model = build_model(cfg)
    specs = model.tensor_specs()
    names = {s.name: s.shape for s in specs}
    assert len(names) == len(specs)
    caches, states = model.cache_specs(), model.state_specs()
    W = cfg["width"]
    expect = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram:
        expect["bigram"] = (bigram["buckets"] + 1, W)
        assert states[-1].shape == (1,) and len(states) == len(cfg["layers"]) + 1
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        assert states[i] is None
        expect[f"l{i}.norm1"] = (W,)
        expect[p + "q"], expect[p + "o"] = (H * D, W), (W, H * Dv)
        if L["type"] == "latent_attention":
            R = m["kv_rank"]
            expect.update({p + "dkv": (R, W), p + "dkv.norm": (R,), p + "uk": (H * D, R), p + "uv": (H * Dv, R), p + "g": (H, W)})
            assert (caches[i].kind, caches[i].row_width) == ("full", R)
        else:
            G = m["kv_heads"]
            expect.update({p + "k": (G * D, W), p + "v": (G * Dv, W)})
            if L["type"] == "attention":
                expect.update({p + "q.norm": (H * D,), p + "k.norm": (G * D,)})
                if D == Dv and D % 16 == 0:
                    assert (caches[i].kind, caches[i].num_kv_heads, caches[i].head_dim) == ("full", G, D)
                else:
                    assert (caches[i].kind, caches[i].row_width) == ("full", G * (D + Dv))
            else:
                expect[p + "pb"] = (H,)
                row = (max(D, Dv) + 15) // 16 * 16
                assert (caches[i].kind, caches[i].window, caches[i].num_kv_heads, caches[i].head_dim) == ("window", m["mask"]["size"], G, row)
        if L["mlp"]:
            expect.update({f"l{i}.mlp.up": (L["mlp"]["ff"], W), f"l{i}.mlp.down": (W, L["mlp"]["ff"])})
    assert names == expect


def test_sizes_and_constants_come_from_the_configuration():
    cfg = copy.deepcopy(PC.MIXED)
    typed, model = build_model(cfg)
    plan = model.plan
    assert plan.embedding_scale == 3.5 and not plan.tie_word_embeddings and plan.head_name == "head"
    e = model.embedding_extras[0]
    assert (e.buckets, e.mul_prev, e.mul_cur) == (53, 17, 5)
    att, lat, win = (model.blocks[i].mixer for i in (0, 1, 2))
    assert type(model.blocks[0]).__name__ == "ParallelBlock" and model.blocks[0].norm1.groups == 3
    assert (model.blocks[0].norm1.eps, model.final_norm.groups) == (1e-5, 3)
    assert (att.scale, att.heads, att.kv_heads, att.head_dim, att.value_dim) == (0.3, 6, 2, 16, 16)
    p = att.position
    assert (p.rotary_dim, p.theta, p.factor, p.low, p.high, p.original) == (8, 500.0, 4.0, 1.0, 3.0, 96.0)
    v = att.value_position
    assert (v.rotary_dim, v.theta) == (16, 500.0) and type(v).__name__ == "RotaryHalfSplit"
    assert not att.sigmoid and att.has_norm and not att.has_bias and not att.has_gate and att.window is None
    assert (lat.heads, lat.dim, lat.value_dim, lat.kv_rank, lat.q_rank, lat.rot_dim, lat.scale) == (3, 24, 40, 64, None, 0, 0.25)
    assert lat.gate_per_head and not lat.has_sink
    assert win.sigmoid and win.window == 20 and not win.has_norm and win.value_position is None
    assert type(win.position).__name__ == "RotaryInterleaved" and win.position.rotary_table(torch.device("cpu")) is None
    assert model.blocks[0].feed_forward.intermediate_size == 72 and not model.blocks[2].has_ff
    cfg["layers"][0]["mixer"].pop("rot")
    del cfg["embedding"], cfg["norm"]["groups"]
    typed, model = build_model(cfg)
    assert model.blocks[0].mixer.position is None and model.blocks[0].mixer.value_position is None
    assert model.plan.embedding_scale == 1.0 and not model.embedding_extras and model.final_norm.groups == 1
    # nothing of the keys is turned, the values are
    cfg["layers"][0]["mixer"]["rot"] = {"base": 77.0, "dims": 0}
    m = build_model(cfg)[1].blocks[0].mixer
    assert m.position is None and (m.value_position.theta, m.value_position.rotary_dim) == (77.0, 16)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "even and at most"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "even and at most"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=0.5), "low <= high"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=15), "in pairs"),
    (lambda c: c["layers"][2]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "at least 1"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0}), "scaling"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0].update(type="attention_3"), "known"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "known"),
    (lambda c: c["norm"].update(groups=5), "equal parts"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda c: c.pop("width"), "width"),
])
def test_a_configuration_that_cannot_run_is_refused(change, message):
    cfg = copy.deepcopy(PC.MIXED)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        build_model(cfg)


@pytest.mark.parametrize("rot", [
    {"base": 500.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 96}},
    {"base": 500000.0, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
    {"base": 10000.0, "dims": 6, "scaling": {"factor": 2.0, "low": 1.5, "high": 1.5, "original": 40}},       # no band between
    {"base": 50.0, "dims": 10, "scaling": {"factor": 16.0, "low": 2.0, "high": 8.0, "original": 1000000}},   # all waves short
    {"base": 300.0, "dims": 12, "scaling": {"factor": 3.0, "low": 1.0, "high": 9.0, "original": 3}},         # all waves long
    {"base": 300.0, "dims": 12, "scaling": {"factor": 1.0, "low": 1.0, "high": 4.0, "original": 64}},
    {"base": 70.0, "dims": 14},
])
def test_frequencies_are_the_plain_rules(rot):
    from ninfer_amd_mi50_b200.parts import position as P
    dev = torch.device("cpu")
    want = PP.frequencies(rot)
    if "scaling" in rot:
        part = P.RotaryHalfSplitBanded(head_dim=rot["dims"] + 4, theta=rot["base"], rotary_dim=rot["dims"], **rot["scaling"])
        parts = [part.pair_table(dev)]
    else:
        parts = [P.RotaryHalfSplit(rot["dims"] + 4, rot["base"], rot["dims"], double=True).pair_table(dev),
                 P.RotaryInterleaved(rot["dims"] + 4, rot["base"], rot["dims"]).pair_table(dev)]
        assert [p[2] for p in parts] == [False, True]
    for table, dims, _ in parts:
        assert dims == rot["dims"] and table.dtype == torch.float32
        assert torch.allclose(table.double(), want, rtol=1e-7, atol=0.0)


def test_the_pending_pair_is_summed_for_whoever_does_not_know_it():
    from ninfer_amd_mi50_b200.parts.base import PairSum, summed
    a, b = torch.randn(3, 5), torch.randn(3, 5)
    assert torch.equal(summed(PairSum(a, b)), a + b)


def test_a_windows_edge_in_the_plain_model():
    """Token i sees i - size + 1 and not i - size (the plain model the GPU tests lean on)."""
    see = PP.visible(9, 4)
    assert see[8].nonzero().flatten().tolist() == [5, 6, 7, 8] and see[2].nonzero().flatten().tolist() == [0, 1, 2]
