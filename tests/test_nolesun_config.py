"""Nolesun's configuration and plan: what config.json says is what the parts are built with; and the plain
implementation's own pieces against statements of their equations that share nothing with it."""

import copy
import math

import pytest
import torch

import nolesun_configs as NC
import plain_nolesun as PN
from ninfer_amd_mi50_b200.config.model_config import ConfigError
from ninfer_amd_mi50_b200.engine.loading import build_model
from ninfer_amd_mi50_b200.registry import architecture_names


def test_the_design_is_registered():
    assert "Nolesun" in architecture_names()


@pytest.mark.parametrize("name", sorted(NC.CONFIGS))
def test_which_tensors_each_layer_names_and_what_its_runs_keep(name):
    cfg, _ = NC.CONFIGS[name]
    typed, model = build_model(cfg)
    names = {s.name: s.shape for s in model.tensor_specs()}
    assert len(names) == len(model.tensor_specs())
    W = cfg["width"]
    expect = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop"):
        expect.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    for i, L in enumerate(cfg["layers"]):
        m, f, p = L["mixer"], L["mlp"], f"l{i}."
        for n in ("norm1", "norm1b", "ls1") + (("norm2", "norm2b", "ls2") if f else ()):
            expect[p + n] = (W,)
        a, r = m["left"], m["right"]
        H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        q = p + "mix.left."
        expect.update({q + "q": (H * D, W), q + "k": (G * D, W), q + "v": (G * Dv, W), q + "o": (W, H * Dv)})
        s = p + "mix.right."
        if L["type"] == "parallel_2":
            expect.update({q + "q.b": (H * D,), q + "k.b": (G * D,), q + "v.b": (G * Dv,), q + "o.b": (W,), q + "g": (H * Dv, W)})
            Hr, Gr, Dr, V, K = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
            for n, width in (("q", Gr * Dr), ("k", Gr * Dr), ("v", Hr * V)):
                expect.update({s + n: (width, W), s + n + ".conv": (width, K)})
            expect.update({s + "g": (Hr * V, W), s + "a": (Hr, W), s + "b": (Hr, W), s + "A_log": (Hr,), s + "dt_bias": (Hr,),
                           s + "norm": (V,), s + "o": (W, Hr * V)})
        else:
            inner, GN = r["heads"] * r["vdim"], r["groups"] * r["state"]
            expect.update({s + "in": (2 * inner + 2 * GN + r["heads"], W), s + "conv": (inner + 2 * GN, r["conv"]),
                           s + "conv.b": (inner + 2 * GN,), s + "dt_bias": (r["heads"],), s + "A_log": (r["heads"],),
                           s + "D": (r["heads"],), s + "norm": (inner,), s + "o": (W, inner)})
        if f and f["kind"] == "dense":
            expect.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
        elif f:
            E = f["router"]["experts"]
            expect.update({p + "mlp.router": (E, W), p + "mlp.router.b": (E,)})
            for e in range(E):
                expect.update({f"{p}mlp.e{e}.gate": (f["expert"]["ff"], W), f"{p}mlp.e{e}.up": (f["expert"]["ff"], W),
                               f"{p}mlp.e{e}.down": (W, f["expert"]["ff"])})
    assert names == expect
    # every run of a layer has pages and a state of its own
    runs = PN.layer_runs(cfg)
    caches, states = model.cache_specs(), model.state_specs()
    assert [c.layer for c in model.order] == [i for i, _ in runs] and len(caches) == len(states) == len(runs)
    assert [c.cache for c in model.order] == [c.state_slot() for c in model.order] == list(range(len(runs)))
    for (i, t), call, cache, state in zip(runs, model.order, caches, states):
        L = cfg["layers"][i]
        a, r = L["mixer"]["left"], L["mixer"]["right"]
        D, Dv = a["dim"], a["vdim"]
        if D == Dv and D % 16 == 0:
            assert (cache.num_kv_heads, cache.head_dim) == (a["kv_heads"], D)
        elif a.get("softcap"):
            assert (cache.num_kv_heads, cache.head_dim) == (a["kv_heads"], (max(D, Dv) + 15) // 16 * 16)
        else:
            assert cache.row_width == a["kv_heads"] * (D + Dv)
        if L["type"] == "parallel":
            C = r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            assert state.shape == ((r["conv"] - 1) * C + r["heads"] * r["vdim"] * r["state"],)
        else:
            conv = (r["conv"] - 1) * (2 * r["kv_heads"] * r["dim"] + r["heads"] * r["vdim"])
            assert state.shape == ((conv + 3) // 4 * 4 + r["heads"] * r["vdim"] * r["dim"],)
        enters = t is not None and i == cfg["loop"]["start"]
        assert call.project == ("loop.in" if enters else None) and call.add_vector == (("loop.step", t) if enters else None)


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "attention"), (("layers", 0, "mixer", "left", "kv_heads"), 3), (("layers", 0, "mixer", "left", "rot", "dims"), 34),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7), (("layers", 0, "mixer", "left", "softcap"), 5.0),
    (("layers", 1, "mixer", "left", "softcap"), -1.0), (("layers", 0, "mixer", "left", "scale"), 0.0),
    (("layers", 0, "mixer", "right", "groups"), 4), (("layers", 0, "mixer", "right", "norm_groups"), 7),
    (("layers", 1, "mixer", "right", "kv_heads"), 3), (("layers", 0, "mixer", "left_scale"), None), (("layers", 0, "mlp", "kind"), "gated"),
    (("layers", 0, "mlp", "router", "top"), 6), (("norm", "eps"), 0.0), (("loop", "stop"), 5), (("loop", "times"), 0),
    (("loop", "start"), 3), (("layers",), []), (("vocab",), "many"), (("layers", 0, "mixer", "right", "conv"), None),
])
def test_a_configuration_that_cannot_be_meant_is_refused(path, value):
    cfg = copy.deepcopy(NC.LOOPED)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        build_model(cfg)


def test_constants_reach_the_parts():
    typed, model = build_model(NC.LOOPED)
    b0, b1 = model.blocks[0], model.blocks[1]
    assert b0.mixer.scales == (0.7, 1.3) and b1.mixer.scales == (1.1, 0.6)
    left0, right0 = b0.mixer.mixers
    left1, right1 = b1.mixer.mixers
    assert left0.scale == 0.2 and not left0.softcap and not left0.has_gate and left1.softcap == 4.0 and left1.has_gate
    f, dims, neighbours = left0.position.pair_table(torch.device("cpu"))
    assert (dims, neighbours) == (16, False) and torch.allclose(f, torch.tensor([300.0 ** (-2 * i / 16) for i in range(8)]))
    assert left1.position.pair_table(torch.device("cpu"))[1:] == (8, True)
    assert right0.norm_groups == 2 and right1.taps == 4 and right1.query_scale == 24 ** -0.5
    assert model.plan.embedding_scale == 5.5 and b0.norm1.eps == b0.norm1b.eps == right0.eps == right1.eps == 1e-5
    assert b0.feed_forward.has_router_bias and b0.feed_forward.norm_topk_prob


# ---- the plain implementation's pieces ------------------------------------------------------------------

def test_the_plain_delta_rule_step_is_the_written_out_sum():
    g = torch.Generator().manual_seed(1)
    D, V = 5, 3
    S, q, k, v = (torch.randn(*s, generator=g, dtype=torch.float64) for s in ((D, V), (D,), (D,), (V,)))
    new, o = PN.delta_step(S, q, k, v, 0.7, 0.4)
    for j in range(V):
        known = sum(0.7 * float(S[i, j]) * float(k[i]) for i in range(D))
        u = 0.4 * (float(v[j]) - known)
        col = [0.7 * float(S[i, j]) + float(k[i]) * u for i in range(D)]
        assert max(abs(a - float(b)) for a, b in zip(col, new[:, j])) < 1e-12
        assert abs(sum(c * float(x) for c, x in zip(col, q)) - float(o[j])) < 1e-12


def test_the_plain_rotation_convolution_and_choice():
    x = torch.arange(12, dtype=torch.float64).view(3, 1, 4) / 7
    for neighbours, pairs in ((False, ((0, 2), (1, 3))), (True, ((0, 1), (2, 3)))):
        y = PN.turn(x, 10.0, 4, neighbours)
        for p in range(3):
            for i, (a, b) in enumerate(pairs):
                ang = p * 10.0 ** (-2 * i / 4)
                u, v = float(x[p, 0, a]), float(x[p, 0, b])
                assert abs(float(y[p, 0, a]) - (u * math.cos(ang) - v * math.sin(ang))) < 1e-12
                assert abs(float(y[p, 0, b]) - (v * math.cos(ang) + u * math.sin(ang))) < 1e-12
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    assert PN.short_conv(u, torch.tensor([[10.0, 1.0]], dtype=torch.float64)).flatten().tolist() == [1.0, 12.0, 24.0]
    idx, wts = PN.choose(torch.tensor([[0.0, 3.0, 1.0]], dtype=torch.float64), 2)
    assert idx.tolist() == [[1, 2]] and abs(float(wts[0, 0]) - 1 / (1 + math.exp(-2))) < 1e-12
