"""The Pudizen design in the engine against the plain whole-sequence implementation (`plain_pudizen`): each
mechanism alone, whole prompts, token-by-token decoding, portions down to two tokens, unequal requests in one
batch, pages and slots used again, long decoding, and greedy generation through the entry point.  Random
weights are scaled out of their nearly linear range, and where a fault would still hide (a far key among
hundreds, a window's edge) the weights are made so that it shows."""

import json
import os

import pytest
import torch

import plain_pudizen as PP
import pudizen_configs as PC
import schedules
from tiny_configs import random_tokens

pytestmark = pytest.mark.gpu

LENGTHS = [70, 5, 131, 33, 2, 97, 1]


def options(dtype, **kw):
    from ninfer_amd_mi50_b200.config import EngineOptions
    base = dict(dtype=dtype, page_size=16, num_sequences=4, max_context=256, cache_tokens=1024, use_graph=False)
    base.update(kw)
    return EngineOptions(**base)


def load(d, dtype, **kw):
    from ninfer_amd_mi50_b200.engine import load_runner
    return load_runner(d, options=options(dtype, **kw))


def run(runner, steps):
    """Drive the runner through a schedule -> float64 logits per request, in the order asked."""
    from ninfer_amd_mi50_b200 import kernels
    from ninfer_amd_mi50_b200.engine import StepEntry
    got = {}
    for st in steps:
        entries = []
        for e in st["entries"]:
            if not runner.cache.is_open(e["id"]):
                runner.open(e["id"])
            entries.append(StepEntry(e["id"], e["tokens"], e["want"]))
        out = runner.step(entries)
        r = 0
        for e in st["entries"]:
            n = len(e["want"])
            got.setdefault(e["id"], []).append(out[r:r + n].double().cpu())
            r += n
        for rid in st["end"]:
            runner.close(rid)
        runner.cache.check()
    kernels.check_status("schedule")
    return {k: torch.cat(v) for k, v in got.items()}


def plain(cfg, w, tokens):
    return PP.forward(cfg, w, list(tokens))[0]


def touchy_rows(cfg, w, tokens, want, tries=2):
    """Rows whose logits move by more than 2 % of the scale when every projection's output is disturbed by
    2^-9 of its size (a softmax that rests on two equal scores, a norm of a sum that nearly cancels)."""
    scale = want.abs().max().item()
    out = torch.zeros(want.shape[0], dtype=torch.bool)
    try:
        for i in range(tries):
            PP.NOISE = (torch.Generator().manual_seed(50 + i), 2.0 ** -9)
            out |= (plain(cfg, w, tokens) - want).abs().max(dim=1).values / scale > 2e-2
    finally:
        PP.NOISE = None
    return out


def compare(got, want, dtype, what, touchy=None):
    """float32 is the sharp comparison: 1e-4 of the largest logit for every row.  bfloat16 rounds every
    activation between kernels to 8 bits: every row within 4 %, the median row (of 16 rows or more) within
    1 %; rows found `touchy` only have to be finite."""
    scale = want.abs().max().item()
    err = (got - want).abs().max(dim=1).values / scale
    assert torch.isfinite(got).all(), what
    if dtype == "float32":
        assert err.max().item() <= 1e-4, f"{what}: row {int(err.argmax())} of {len(err)} differs by {err.max().item():.3e} of the scale"
        return
    if touchy is not None:
        assert len(touchy) < 16 or touchy.float().mean().item() <= 0.25, f"{what}: {int(touchy.sum())} of {len(touchy)} rows are touchy"
        err = err[~touchy]
    if len(err):
        assert err.max().item() <= 4e-2, f"{what}: row {int(err.argmax())} of {len(err)} steady rows differs by {err.max().item():.3e} of the scale"
    if len(err) >= 16:
        assert err.median().item() <= 1e-2, f"{what}: the median row differs by {err.median().item():.3e} of the scale"


@pytest.fixture(scope="module", params=sorted(PC.CONFIGS))
def folder(request, tmp_path_factory):
    cfg, seed = PC.CONFIGS[request.param]
    d = str(tmp_path_factory.mktemp("pudizen") / request.param)
    PC.write_folder(cfg, seed, d, scale=PC.SCALES.get(request.param))
    cfg, w = PC.read_folder(d)
    reqs = {f"r{i}": random_tokens(n, cfg["vocab"], 900 + i) for i, n in enumerate(LENGTHS)}
    want = {r: plain(cfg, w, t) for r, t in reqs.items()}
    touchy = {r: touchy_rows(cfg, w, t, want[r]) for r, t in reqs.items()}
    return request.param, d, cfg, w, reqs, want, touchy


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["whole", "tail", "portions", "pairs", "mixed"])
def test_every_way_of_cutting_matches_the_plain_model(folder, dtype, how):
    name, d, cfg, w, reqs, want, touchy = folder
    make = {"whole": schedules.whole, "tail": lambda r: schedules.tail_decoded(r, tail=40),
            "portions": schedules.portions, "pairs": lambda r: schedules.portions(r, cuts=[2, 3]),
            # a pool of 320 tokens for 339 in all, three slots for seven requests: pages and slots come back
            "mixed": lambda r: schedules.mixed(r, max_live=3, page=16, pool_tokens=320, tail=9)}[how]
    pool = 320 if how == "mixed" else 1024
    runner = load(d, dtype, cache_tokens=pool, num_sequences=3 if how == "mixed" else 4)
    got = run(runner, make(reqs))
    assert all(n == pool // 16 for n in runner.cache.pages_free())
    for r in reqs:
        compare(got[r], want[r], dtype, f"{name} {how} {r}", touchy[r])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_through_the_kernels_for_many_rows(folder, dtype):
    """More than 128 rows in one portion (the tcgen05 attention kernels, library products), then a second
    portion on top of the first one's cache, then decoded rows, beside a short request."""
    name, d, cfg, w, reqs, want, touchy = folder
    a, b = random_tokens(420, cfg["vocab"], 31), random_tokens(150, cfg["vocab"], 32)
    full = lambda i, t: {"id": i, "tokens": t, "want": list(range(len(t)))}
    steps = [{"entries": [full("a", a[:200])], "end": []},
             {"entries": [full("b", b[:100])], "end": []},
             # a portion of many rows beside a decoded token, then beside another portion
             {"entries": [full("b", b[100:101]), full("a", a[200:340])], "end": []},
             {"entries": [full("a", a[340:410]), full("b", b[101:140])], "end": []},
             {"entries": [full("c", a[:150]), full("d", b[:1])], "end": ["c", "d"]}]
    steps += [{"entries": [full("b", b[140 + i:141 + i]), full("a", a[410 + i:411 + i])], "end": ["a", "b"] if i == 9 else []}
              for i in range(10)]
    got = run(load(d, dtype, max_context=512, page_size=64), steps)
    for i, t in (("a", a), ("b", b), ("c", a[:150]), ("d", b[:1])):
        ref = plain(cfg, w, t)
        compare(got[i], ref, dtype, f"{name} {i}", touchy_rows(cfg, w, t, ref))


# ---- each mechanism alone ---------------------------------------------------------------------

def check_alone(tmp_path, cfg, dtype, n_tokens=90, cuts=(2, 3, 40, 1, 16), replace=None, scale=None, seed=7, **opt):
    d = PC.write_folder(cfg, seed, str(tmp_path / "m"), replace=replace, scale=scale)
    cfg, w = PC.read_folder(d)
    toks = random_tokens(n_tokens, cfg["vocab"], seed)
    want = plain(cfg, w, toks)
    touchy = touchy_rows(cfg, w, toks, want)
    got = run(load(d, dtype, **opt), schedules.whole({"a": toks}))["a"]
    compare(got, want, dtype, "whole", touchy)
    if cuts:
        compare(run(load(d, dtype, **opt), schedules.portions({"a": toks}, cuts=list(cuts)))["a"], want, dtype, "portions", touchy)
    return cfg, w, toks, want, got


def distance(a, b):
    return ((a - b).abs().max() / b.abs().max()).item()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", [
    PC.attention(2, 1, 8, 8, 0.3, rot=(100.0, 4)),                                            # one row a token, equal sizes
    PC.attention(4, 2, 16, 16, 0.25),                                                         # nothing turned
    PC.attention(4, 2, 16, 16, 0.25, rot=(60.0, 0)),                                          # the values turned, the keys not
    PC.attention(4, 4, 32, 32, 0.2, rot=(10000.0, 32), scaling=(4.0, 1.0, 4.0, 48)),          # the whole head
    PC.attention(6, 3, 16, 40, 0.3, rot=(50.0, 10), scaling=(16.0, 1.0, 2.0, 16)),            # values wider than keys
    PC.attention(3, 1, 24, 6, 0.2, rot=(700.0, 24)),                                          # keys wider than values
    PC.attention(8, 8, 64, 64, 0.15, rot=(1e6, 16), scaling=(1.0, 1.0, 4.0, 64)),             # factor 1: the plain frequencies
    PC.attention(2, 1, 48, 48, 0.15, rot=(300.0, 20)),                                        # a size without a split-key kernel
])
def test_softmax_attention_alone(tmp_path, dtype, mixer):
    check_alone(tmp_path, PC.model([PC.layer(mixer)], width=72), dtype, n_tokens=150)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norms_rotation_scaling_and_turned_values_each_change_the_answer(tmp_path, dtype):
    """The plain model without one of the mechanisms differs from the engine by far more than rounding."""
    mixer = PC.attention(4, 2, 16, 16, 0.3, rot=(100.0, 8), scaling=(8.0, 1.0, 2.0, 64))
    cfg, w, toks, want, got = check_alone(tmp_path, PC.model([PC.layer(mixer)]), dtype, cuts=None)
    for name in ("l0.mix.q.norm", "l0.mix.k.norm"):
        assert distance(got, plain(cfg, dict(w, **{name: torch.ones_like(w[name])}), toks)) > 0.05, name
    for change in ({"scaling": None}, {"dims": 0}, {"dims": 6}, {"base": 10.0}):
        cfg2 = json.loads(json.dumps(cfg))
        cfg2["layers"][0]["mixer"]["rot"].update(change)
        assert distance(got, plain(cfg2, w, toks)) > 0.05, change
    saved = PP.turn
    try:        # keys turned, values not: every call that turns all 16 dimensions is left out
        PP.turn = lambda x, a, dims, inter: x if dims == 16 else saved(x, a, dims, inter)
        assert distance(got, plain(cfg, w, toks)) > 0.05
    finally:
        PP.turn = saved


WINDOWED = [
    PC.windowed(4, 2, 16, 16, 0.25, 24, rot=(100.0, 8)),
    PC.windowed(2, 1, 8, 8, 0.3, 3, rot=(50.0, 8)),                     # widened to 16
    PC.windowed(6, 2, 16, 40, 0.3, 31),                                 # values wider than keys, nothing turned
    PC.windowed(3, 3, 24, 6, 0.2, 50, rot=(700.0, 24)),                 # keys wider than values
    PC.windowed(8, 1, 64, 64, 0.15, 64, rot=(1e4, 16)),
    PC.windowed(2, 2, 128, 128, 0.1, 129, rot=(1e4, 64)),
    PC.windowed(2, 1, 144, 100, 0.08, 70, rot=(1e3, 40)),               # beyond the flash kernel's sizes
    PC.windowed(4, 1, 32, 32, 0.2, 1, rot=(1e4, 32)),                   # itself alone
    PC.windowed(4, 1, 32, 32, 0.2, 4096, rot=(1e4, 32)),                # a window nothing reaches the end of
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", WINDOWED)
def test_sigmoid_attention_alone(tmp_path, dtype, mixer):
    check_alone(tmp_path, PC.model([PC.layer(mixer)], width=72), dtype, n_tokens=200)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_window_bias_pairs_and_missing_normalisation_each_change_the_answer(tmp_path, dtype):
    mixer = PC.windowed(4, 2, 16, 16, 0.3, 12, rot=(20.0, 8))
    cfg, w, toks, want, got = check_alone(tmp_path, PC.model([PC.layer(mixer)]), dtype, cuts=None)
    assert distance(got, plain(cfg, dict(w, **{"l0.mix.pb": torch.zeros_like(w["l0.mix.pb"])}), toks)) > 0.05
    for change in ({"mask": {"size": 11}}, {"mask": {"size": 13}}, {"rot": None}):
        cfg2 = json.loads(json.dumps(cfg))
        cfg2["layers"][0]["mixer"].update(change)
        assert distance(got, plain(cfg2, w, toks)) > 0.05, change
    saved = PP.turn
    try:
        PP.turn = lambda x, a, dims, inter: saved(x, a, dims, False)             # halves instead of neighbours
        assert distance(got, plain(cfg, w, toks)) > 0.05
    finally:
        PP.turn = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(3, 24, 40, 64, 0.2), (5, 10, 7, 33, 0.3), (8, 16, 16, 192, 0.15), (40, 8, 24, 128, 0.3), (1, 64, 64, 320, 0.1)])
def test_latent_attention_alone(tmp_path, dtype, sizes):
    cfg, w, toks, want, got = check_alone(tmp_path, PC.model([PC.layer(PC.latent(*sizes))], width=88), dtype, n_tokens=170)
    for name, value in (("l0.mix.g", 0.0), ("l0.mix.dkv.norm", 1.0)):
        assert distance(got, plain(cfg, dict(w, **{name: torch.full_like(w[name], value)}), toks)) > 0.05, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,rows", [(88, 3), (24, 40), (200, 300), (51, 12)])
def test_squared_relu_feed_forward_beside_its_mixer(tmp_path, dtype, ff, rows):
    """Both sublayers read one norm's output: the plain model with the feed-forward after the mixer, or with
    the relu not squared, is far off."""
    cfg, w, toks, want, got = check_alone(tmp_path, PC.model([PC.layer(PC.attention(2, 1, 8, 8, 0.3), ff)], groups=2), dtype,
                                          n_tokens=rows, cuts=None, max_context=512)
    saved = PP.relu2_mlp
    try:
        PP.relu2_mlp = lambda h, w_, p: PP.proj(torch.relu(PP.proj(h, w_[p + "up"])), w_[p + "down"])
        assert distance(got, plain(cfg, w, toks)) > 0.05
    finally:
        PP.relu2_mlp = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,groups", [(96, 1), (96, 6), (96, 96), (66, 3), (520, 2), (1200, 5)])
def test_norm_in_groups_and_the_scaled_hashed_embedding(tmp_path, dtype, width, groups):
    """Layers without feed-forward and with; the groups' sizes differ so much that one norm over the row, or
    another number of groups, is far off; the pair rows change the stream of every token but the first alike."""
    g = torch.Generator().manual_seed(3)
    cfg = PC.model([PC.layer(PC.attention(2, 1, 8, 8, 0.3), 40), PC.layer(PC.latent(2, 8, 8, 16, 0.3))], width=width, groups=groups,
                   scale=7.25, bigram=(29, 13, 1000003))
    ramp = torch.logspace(-1.0, 1.0, width)
    rep = {"embed": torch.randn(cfg["vocab"], width, generator=g) * 0.1 * ramp, "bigram": torch.randn(30, width, generator=g) * 0.5 * ramp}
    cfg, w, toks, want, got = check_alone(tmp_path, cfg, dtype, n_tokens=60, replace=rep)
    changes = [{"embedding": dict(cfg["embedding"], scale=1.0)}, {"embedding": {"scale": 7.25}},
               {"embedding": dict(cfg["embedding"], bigram=dict(cfg["embedding"]["bigram"], mul_prev=14))},
               {"embedding": dict(cfg["embedding"], bigram=dict(cfg["embedding"]["bigram"], mul_cur=1000004))}]
    if groups > 1:
        changes.append({"norm": dict(cfg["norm"], groups=1)})
    for change in changes:
        assert distance(got, plain(dict(cfg, **change), w, toks)) > 0.03, change
    # the first token's row is the last one of the table
    first = dict(w, bigram=torch.cat([w["bigram"][:-1], torch.zeros_like(w["bigram"][-1:])]))
    assert distance(got[:1], plain(cfg, first, toks[:1])) > 0.03


# ---- kernels against the plain kernel -----------------------------------------------------------------

def paged_case(lens, G, D, page, seed=5):
    """Random pages for requests of `lens` tokens each, all decoding their last one."""
    from ninfer_amd_mi50_b200.parts.base import StepContext
    g = torch.Generator(device="cuda").manual_seed(seed)
    S = len(lens)
    width = (max(lens) + page - 1) // page
    pages = (torch.randn(S * width + 1, 2, G, page, D, device="cuda", generator=g) * 0.7).bfloat16()
    table = torch.randperm(S * width, device="cuda", generator=g).to(torch.int32).view(S, width)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    ctx = StepContext(dtype=torch.bfloat16, device=torch.device("cuda"), T=S, S=S, token_ids=i32([0] * S),
                      positions=i32([n - 1 for n in lens]), row_seg=i32(list(range(S))), seg_row0=i32(list(range(S + 1))),
                      seg_pos0=i32([n - 1 for n in lens]), seg_slot=i32(list(range(S))), logit_rows=i32([0]),
                      seg_len_host=[1] * S, seg_pos0_host=[n - 1 for n in lens], max_rows_per_seg=1, max_context=max(lens))
    return pages, table, ctx, g


@pytest.mark.parametrize("rows", [3, 70])
@pytest.mark.parametrize("D", [16, 64, 128])
@pytest.mark.parametrize("window", [0, 1, 130])
def test_decode_kernels_with_sigmoid_weights_and_turned_values(rows, D, window):
    """The split-key kernels - one CTA a block (few blocks), the persistent form (many) - against the plain kernel of
    one warp a row and head on the same cache: sigmoid weights, and results turned back in the merge."""
    from ninfer_amd_mi50_b200 import kernels
    H, G, page = 16, 8, 16
    lens = [1 + (37 * i) % 330 for i in range(rows)]
    pages, table, ctx, g = paged_case(lens, G, D, page)
    q = (torch.randn(rows, H * D, device="cuda", generator=g) * 0.7).bfloat16()
    pb = torch.randn(H, device="cuda", generator=g)
    freq = torch.rand(D // 2, device="cuda", generator=g)
    sig = lambda: kernels.biased_window_attention(q, H, G, D, pages, table, page, ctx, window, 0, D ** -0.5, None, sigmoid_bias=pb)
    soft = lambda inter: kernels.paged_attention(q, H, G, D, pages, table, page, ctx, window, D ** -0.5, turn=(freq, D, inter))
    fast = [sig(), soft(False), soft(True)]
    saved = kernels.TUNING["bf16_attention"]
    try:
        kernels.TUNING["bf16_attention"] = "generic"
        plain_ = [sig(), soft(False), soft(True)]
    finally:
        kernels.TUNING["bf16_attention"] = saved
    kernels.check_status("decode kernels")
    for a, b in zip(fast, plain_):
        assert (a.float() - b.float()).abs().max() <= 2e-2 * b.float().abs().max()


@pytest.mark.parametrize("H,Dv,row,interleaved", [(3, 6, 16, False), (3, 6, 16, True), (4, 64, 64, False), (4, 64, 64, True), (5, 24, 24, True), (2, 40, 48, False)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_turning_back(H, Dv, row, interleaved, dtype):
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(1)
    T = 9
    o = torch.randn(T, H * row, device="cuda", generator=g).to(dtype)
    pos = torch.randint(0, 3000, (T,), device="cuda", generator=g, dtype=torch.int32)
    freq = torch.rand(Dv // 2, device="cuda", generator=g) * 0.1
    x = o.double().cpu().view(T, H, row)
    want = x.clone()
    angles = -(pos.cpu().double()[:, None] * freq.cpu().double()[None, :])
    want[..., :Dv] = PP.turn(x[..., :Dv], angles, Dv, interleaved)
    kernels.turn_back(o, pos, freq, H, Dv, row=row, interleaved=interleaved)
    tol = 2e-4 if dtype == torch.float32 else 2e-2
    assert (o.double().cpu().view(T, H, row) - want).abs().max() <= tol


@pytest.mark.parametrize("D,Dv,row,rot,interleaved,turned", [(16, 16, 16, 8, False, True), (16, 16, 16, 12, True, True), (24, 8, 32, 10, True, False),
                                                             (8, 24, 32, 8, False, True), (12, 20, 32, 12, False, False), (64, 64, 64, 0, True, True)])
@pytest.mark.parametrize("norm", [True, False])
@pytest.mark.parametrize("layout", ["heads", "rows"])
def test_append_in_every_form(D, Dv, row, rot, interleaved, turned, norm, layout):
    """Norms or none, both layouts of pairs, turned values, widened heads and rows, vector and scalar accesses."""
    from ninfer_amd_mi50_b200 import kernels
    H, G, T, page = 4, 2, 7, 8
    if layout == "rows":
        row = D
    g = torch.Generator(device="cuda").manual_seed(2)
    pages, table, ctx, _ = paged_case([1 + 5 * i for i in range(T)], G, 16, page)
    n = pages.shape[0]
    pages = torch.full((n, 2, G, page, row) if layout == "heads" else (n, page, G * (D + Dv)), 9.0, device="cuda")
    proj = torch.randn(T, H * D + G * (D + Dv), device="cuda", generator=g)
    wq, wk = (torch.rand(H * D, device="cuda", generator=g) + 0.5, torch.rand(G * D, device="cuda", generator=g) + 0.5) if norm else (None, None)
    freq = torch.rand(max(1, rot // 2), device="cuda", generator=g)
    vfreq = torch.rand(Dv // 2, device="cuda", generator=g) if turned else None
    q = kernels.whole_norm_rope_append(proj, 0, H * D, (H + G) * D, None, None, None, wq, wk, 1e-5, freq if rot else None, rot, 1.0,
                                       H, G, D, Dv, ctx, pages, table, page, torch.float32, interleaved=interleaved,
                                       value_freq=vfreq, row=row)
    p = proj.double().cpu()
    pos = ctx.positions.cpu()
    qw, kw, v = p[:, :H * D], p[:, H * D:(H + G) * D], p[:, (H + G) * D:].reshape(T, G, Dv)
    if norm:
        qw, kw = PP.rms(qw, 1e-5) * wq.double().cpu(), PP.rms(kw, 1e-5) * wk.double().cpu()
    angle = lambda f, k: pos.double()[:, None] * f.double().cpu()[None, :k]
    spin = lambda x: PP.turn(x, angle(freq, rot // 2), rot, interleaved) if rot else x
    qw, kw = spin(qw.reshape(T, H, D)), spin(kw.reshape(T, G, D))
    if turned:
        v = PP.turn(v, angle(vfreq, Dv // 2), Dv, interleaved)
    got_q = q.double().cpu().view(T, H, row)
    assert (got_q[..., :D] - qw).abs().max() <= 2e-4 and (got_q[..., D:] == 0).all()
    for t in range(T):
        pg, at = int(table[t, int(pos[t]) // page]), int(pos[t]) % page
        if layout == "heads":
            k_t, v_t = pages[pg, 0, :, at].double().cpu(), pages[pg, 1, :, at].double().cpu()
            assert (k_t[:, D:] == 0).all() and (v_t[:, Dv:] == 0).all()
        else:
            r = pages[pg, at].double().cpu()
            k_t, v_t = r[:G * D].view(G, D), r[G * D:].view(G, Dv)
        assert (k_t[:, :D] - kw[t]).abs().max() <= 2e-4 and (v_t[:, :Dv] - v[t]).abs().max() <= 2e-4


# ---- keys far away and at edges -----------------------------------------------------------------------

def twin_tokens(w0, width, seed=9):
    """Two tokens whose embeddings share the first half and have opposite second halves (an RMS norm treats
    both alike): `replace`-ready embedding with them as tokens 400 and 398."""
    g = torch.Generator().manual_seed(seed)
    a, b = torch.randn(width // 2, generator=g, dtype=torch.float64) * 0.08, torch.randn(width // 2, generator=g, dtype=torch.float64) * 0.08
    embed = w0["embed"].clone()
    embed[400], embed[398] = torch.cat([a, b]), torch.cat([a, -b])
    return embed


def steps_for(toks, how, cuts):
    n = len(toks)
    if how == "prompt":
        return [{"entries": [{"id": "a", "tokens": toks, "want": [n - 1]}], "end": ["a"]}]
    if how == "portions":
        cut = [c for c in cuts if c < n] + [n]
        return [{"entries": [{"id": "a", "tokens": toks[x:y], "want": [y - x - 1] if y == n else []}], "end": ["a"] if y == n else []}
                for x, y in zip(cut, cut[1:])]
    steps = [{"entries": [{"id": "a", "tokens": toks[:n - 3], "want": []}], "end": []}]
    return steps + [{"entries": [{"id": "a", "tokens": toks[i:i + 1], "want": [0] if i == n - 1 else []}],
                     "end": ["a"] if i == n - 1 else []} for i in range(n - 3, n)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", [PC.attention(4, 2, 32, 32, 0.5, rot=(500.0, 0)), PC.attention(4, 1, 32, 24, 0.5, rot=(500.0, 0)),
                                   PC.attention(2, 1, 128, 128, 0.125), PC.latent(4, 32, 16, 64, 6.0), PC.latent(3, 24, 10, 40, 6.0)])
def test_one_far_key_among_hundreds_is_found(tmp_path, dtype, mixer):
    """Queries and keys are made of the first half of the width by one matrix, so a query's best keys are those of
    tokens whose first half is its own.  A token and its twin (same first half, opposite second half, from which
    the values come) stand last and once before - at a page's first or last place, or hundreds back: a key that is
    lost, or read from the wrong place, changes the answer wholly.  In a prompt, in portions and decoded."""
    W = 64
    cfg = PC.model([PC.layer(mixer)], width=W, vocab=401)
    m = mixer["mixer"]
    d0 = PC.write_folder(cfg, 3, str(tmp_path / "m0"), scale={"embed": 4.0})
    _, w0 = PC.read_folder(d0)
    g = torch.Generator().manual_seed(4)
    rand = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64) * 0.2
    replace = {"embed": twin_tokens(w0, W), "l0.norm1": torch.ones(W)}
    H, D = m["heads"], m["dim"]
    if mixer["type"] == "attention":
        G = m["kv_heads"]
        wk = rand(G * D, W)
        wk[:, W // 2:] = 0.0
        kn = torch.ones(G * D, dtype=torch.float64)
        replace.update({"l0.mix.k": wk, "l0.mix.q": wk.view(G, D, W).repeat_interleave(H // G, dim=0).reshape(H * D, W),
                        "l0.mix.k.norm": kn, "l0.mix.q.norm": torch.ones(H * D), "l0.mix.v": rand(G * m["vdim"], W)})
    else:
        R, half = m["kv_rank"], m["kv_rank"] // 2
        dkv, uk, uv = rand(R, W), rand(H * D, R), rand(H * m["vdim"], R)
        dkv[:half, W // 2:], dkv[half:, :W // 2] = 0.0, 0.0     # the latent's first half from the first half of the width
        uk[:, half:], uv[:, :half] = 0.0, 0.0                   # keys from that, values from the rest
        replace.update({"l0.mix.dkv": dkv, "l0.mix.uk": uk, "l0.mix.uv": uv, "l0.mix.q": uk @ dkv, "l0.mix.dkv.norm": torch.ones(R)})
    d = PC.write_folder(cfg, 3, str(tmp_path / "m"), replace=replace, scale={"embed": 4.0})
    cfg, w = PC.read_folder(d)
    n = 500
    for place in (0, 15, 16, 17, 63, 64, 250, 463):
        toks = [1 + (i % 397) for i in range(n)]        # tokens 1..397
        toks[place], toks[-1] = 398, 400
        want = plain(cfg, w, toks)[-1:]
        without = list(toks)
        without[place] = 397
        assert distance(plain(cfg, w, without)[-1:], want) > 0.15, "the key does not matter"
        for how in ("prompt", "portions", "decoded"):
            got = run(load(d, dtype, max_context=512), steps_for(toks, how, [0, 14, 16, 19, 64, 67, 300]))
            compare(got["a"], want, dtype, f"place {place} {how}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", [PC.windowed(4, 2, 32, 32, 0.3, 74), PC.windowed(2, 1, 24, 40, 0.4, 33), PC.windowed(2, 2, 128, 128, 0.08, 130),
                                   PC.windowed(2, 1, 64, 64, 0.15, 16), PC.windowed(2, 1, 64, 64, 0.15, 200)])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, mixer):
    """As above for the sigmoid weights (a bias keeps every other key's weight small): the twin stands at the window's
    last visible place, one before it, or one or two beyond, for last positions whose window begins inside a page, at
    its first row and at its last."""
    W = 64
    m = mixer["mixer"]
    H, G, D, size = m["heads"], m["kv_heads"], m["dim"], m["mask"]["size"]
    cfg = PC.model([PC.layer(mixer)], width=W, vocab=401)
    d0 = PC.write_folder(cfg, 3, str(tmp_path / "m0"), scale={"embed": 4.0})
    _, w0 = PC.read_folder(d0)
    g = torch.Generator().manual_seed(4)
    wk = torch.randn(G * D, W, generator=g, dtype=torch.float64) * 0.2
    wk[:, W // 2:] = 0.0
    replace = {"embed": twin_tokens(w0, W), "l0.norm1": torch.ones(W), "l0.mix.k": wk,
               "l0.mix.q": wk.view(G, D, W).repeat_interleave(H // G, dim=0).reshape(H * D, W),
               "l0.mix.v": torch.randn(G * m["vdim"], W, generator=g, dtype=torch.float64) * 0.2,
               "l0.mix.pb": torch.full((H,), -9.0)}
    d = PC.write_folder(cfg, 3, str(tmp_path / "m"), replace=replace, scale={"embed": 4.0})
    cfg, w = PC.read_folder(d)
    for n in (size + 17, size + 32, size + 40, size + 64, size + 130):
        for back in (size - 1, size - 2, size, size + 1):
            place = n - 1 - back
            if place < 0 or back < 1:
                continue
            toks = [1 + (i % 397) for i in range(n)]
            toks[place], toks[-1] = 398, 400
            want = plain(cfg, w, toks)[-1:]
            other = json.loads(json.dumps(cfg))
            other["layers"][0]["mixer"]["mask"]["size"] = back if back < size else back + 1      # the key's side of the edge swapped
            assert distance(plain(other, w, toks)[-1:], want) > 0.1, "the key does not matter"
            for how in ("prompt", "portions", "decoded"):
                got = run(load(d, dtype, max_context=512), steps_for(toks, how, [0, 14, 16, 19, 64, 67, 150]))
                compare(got["a"], want, dtype, f"length {n} back {back} {how}")


# ---- the engine around the design ---------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folder, dtype):
    name, d, cfg, w, reqs, want, touchy = folder
    toks = random_tokens(236, cfg["vocab"], 77)
    ref = plain(cfg, w, toks)
    runner = load(d, dtype)
    got = run(runner, schedules.tail_decoded({"a": toks}, tail=229))
    compare(got["a"], ref, dtype, f"{name} long decoding", touchy_rows(cfg, w, toks, ref))
    assert all(n == 1024 // 16 for n in runner.cache.pages_free())


def test_pages_the_window_has_passed_go_back_while_a_request_runs(folder):
    name, d, cfg, w, reqs, want, touchy = folder
    runner = load(d, "float32")
    got = run(runner, [{"entries": [{"id": "a", "tokens": reqs["r2"][:100], "want": []}], "end": []}])
    for g, free in zip(runner.cache.groups, runner.cache.pages_free()):
        held = 1024 // 16 - free
        first = max(0, 100 - g.spec.window + 1) // 16 if g.spec.kind == "window" else 0
        assert held == 7 - first, (g.spec, held)
    runner.close("a")


def test_pages_and_slots_that_are_used_again_hold_nothing_of_their_last_user(folder):
    name, d, cfg, w, reqs, want, touchy = folder
    runner = load(d, "float32", num_sequences=1, cache_tokens=160)
    a, b = reqs["r0"], reqs["r3"]
    got = run(runner, schedules.whole({"a": a}) + schedules.portions({"b": b}) + schedules.whole({"c": a}))
    compare(got["b"], want["r3"], "float32", f"{name} second user of the pages and the slot")
    assert torch.equal(got["a"], got["c"])


def test_unequal_requests_in_one_batch_equal_each_alone(folder):
    name, d, cfg, w, reqs, want, touchy = folder
    runner = load(d, "float32")
    alone = run(runner, schedules.whole(reqs))
    pick = {r: reqs[r] for r in ("r0", "r1", "r3", "r6")}
    step = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in pick.items()], "end": list(pick)}]
    together = run(runner, step)
    for r in pick:
        assert (together[r] - alone[r]).abs().max() <= 1e-5 * alone[r].abs().max(), r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_rows_logits_do_not_depend_on_how_the_prompt_was_cut(folder, dtype):
    name, d, cfg, w, reqs, want, touchy = folder
    toks = reqs["r2"]
    runner = load(d, dtype)
    a = run(runner, schedules.whole({"a": toks}))["a"]
    b = run(runner, schedules.portions({"a": toks}, cuts=[2, 3, 50, 1, 16]))["a"]
    c = run(runner, schedules.tail_decoded({"a": toks}, tail=60))["a"]
    for other in (b, c):
        diff = (a - other).abs().max(dim=1).values / a.abs().max()
        if dtype == "float32":
            assert diff.max() <= 1e-5
        else:       # a row is served by another kernel when it arrives alone, which rounds elsewhere
            assert diff[~touchy["r2"]].max() <= 4e-2 and diff.median() <= 1e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decode_steps_replayed_from_graphs_equal_host_driven_ones(folder, dtype):
    """A captured step knows a bound of the context only, which sets how the latent attention cuts a row's keys
    into partial sums: equal up to rounding, and bit for bit from one replay to the next."""
    name, d, cfg, w, reqs, want, touchy = folder
    pick = {r: reqs[r][:40] for r in ("r0", "r2", "r5")}
    steps = [{"entries": [{"id": r, "tokens": t[:25], "want": [24]} for r, t in pick.items()], "end": []}]
    for i in range(25, 40):
        steps.append({"entries": [{"id": r, "tokens": t[i:i + 1], "want": [0]} for r, t in pick.items()],
                      "end": list(pick) if i == 39 else []})
    host = run(load(d, dtype), steps)
    runner = load(d, dtype, use_graph=True)
    assert runner.graphs is not None
    graphs, again = run(runner, steps), run(runner, steps)
    for r in pick:
        assert torch.equal(graphs[r], again[r]), r
        diff = (host[r] - graphs[r]).abs().max(dim=1).values / host[r].abs().max()
        steady = ~touchy[r][24:40]
        assert diff[steady].max() <= (1e-6 if dtype == "float32" else 2e-2), (r, diff.max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(folder, dtype):
    from ninfer_amd_mi50_b200.api import Ninfer
    name, d, cfg, w, reqs, want, touchy = folder
    prompts = [reqs["r1"], reqs["r3"], reqs["r4"], reqs["r0"][:40]]
    eng = Ninfer(d, max_context=128, prefill_chunk=16, num_sequences=3, dtype=dtype, page_size=16)
    got = eng.generate(prompts, max_new_tokens=10, temperature=0.0)
    for p, out in zip(prompts, got):
        assert len(out) == 10
        full = plain(cfg, w, list(p) + list(out))
        for k, t in enumerate(out):
            lg = full[len(p) - 1 + k]
            # the engine's token is the plain model's, or (bfloat16) one whose logit is as good as ties go
            slack = 1e-4 if dtype == "float32" else 4e-2
            assert float(lg[t]) >= float(lg.max()) - slack * float(lg.abs().max()), (name, len(p), k, t, int(lg.argmax()))


def test_trace_replay_program_runs_the_design(folder, tmp_path):
    """`bin/trace_run` picks the model class by config.json and gives the in-process logits."""
    import subprocess
    import sys
    import numpy as np
    name, d, cfg, w, reqs, want, touchy = folder
    small = {r: reqs[r] for r in ("r1", "r3", "r0")}
    steps = schedules.mixed(small, max_live=2, page=64, pool_tokens=192, tail=4)
    lines = "".join(json.dumps({"step": i, **st}) + "\n" for i, st in enumerate(steps))
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "192"], input=lines, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    got = run(load(d, "float32", page_size=64, cache_tokens=192, max_context=192), steps)
    rows = {r: 0 for r in small}
    for i, st in enumerate(steps):
        arr = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy()).double()
        at = 0
        for e in st["entries"]:
            n = len(e["want"])
            assert torch.equal(arr[at:at + n], got[e["id"]][rows[e["id"]]:rows[e["id"]] + n]), (i, e["id"])
            at += n
            rows[e["id"]] += n


@pytest.mark.parametrize("how", ["folder", "seed"])
def test_the_command_line_generates_from_the_design(tmp_path, how):
    """`bin/ninfer` on a Pudizen folder, and on a folder with only config.json and a seed."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg0, seed = PC.CONFIGS["mixed"]
    d = str(tmp_path / "m")
    if how == "folder":
        PC.write_folder(cfg0, seed, d)
    else:
        from ninfer_amd_mi50_b200.weights import write_random_model
        write_random_model(cfg0, seed, d)
    cfg, w = PC.read_folder(d)
    if how == "seed":
        os.remove(os.path.join(d, "model.safetensors"))
    prompt = random_tokens(30, cfg["vocab"], 12)
    cmd = [sys.executable, os.path.join(root, "bin", "ninfer"), d, "--prompt-ids", ",".join(map(str, prompt)),
           "--temperature", "0", "--max-new", "6", "--dtype", "fp32", "--prefill-chunk", "16", "--repeat-penalty", "1"]
    if how == "seed":
        cmd += ["--random-weights", str(seed)]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    got = [int(x) for x in p.stdout.split()]
    assert len(got) == 6
    full = plain(cfg, w, prompt + got)
    for k, t in enumerate(got):
        lg = full[len(prompt) - 1 + k]
        assert float(lg[t]) >= float(lg.max()) - 1e-4 * float(lg.abs().max())


def test_sampled_generation_and_a_request_preempted_and_recomputed(folder):
    """Sampling with a temperature through the scheduler, with a pool so small that a request is preempted and
    recomputed: its keys are written again from position 0, its previous token is forgotten, and the tokens are
    those of a roomy pool."""
    from ninfer_amd_mi50_b200.api import Ninfer
    name, d, cfg, w, reqs, want, touchy = folder
    prompts = [reqs["r0"][:50], reqs["r3"], reqs["r5"][:60]]
    roomy = Ninfer(d, max_context=128, prefill_chunk=32, num_sequences=3, dtype="float32", page_size=16)
    want_tokens = roomy.generate(prompts, max_new_tokens=24, temperature=0.8, top_k=20, seed=5)
    tight = Ninfer(d, max_context=128, prefill_chunk=32, num_sequences=3, dtype="float32", page_size=16, cache_tokens=160)
    got = tight.generate(prompts, max_new_tokens=24, temperature=0.8, top_k=20, seed=5)
    assert got == want_tokens
