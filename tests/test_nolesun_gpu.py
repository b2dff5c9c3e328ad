"""The Nolesun design in the engine against the plain whole-sequence implementation (`plain_nolesun`): each
mechanism alone, whole prompts, token-by-token decoding, portions down to two tokens, unequal requests in one
batch, pages and slots used again, long decoding, and greedy generation through the entry point; and the kernels
it brought, each against plain arithmetic.  Random weights are scaled out of their nearly linear range, and where a
fault would still hide (a far key among hundreds, a state that is lost) the weights are made so that it shows."""

import json
import os

import pytest
import torch

import nolesun_configs as NC
import plain_nolesun as PN
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


def run_chosen(runner, steps):
    """Drive the runner through a schedule -> (float64 logits per request, in the order asked; the experts the engine
    chose per request: a list over the routed layer runs of [tokens, top])."""
    from ninfer_amd_mi50_b200 import kernels
    from ninfer_amd_mi50_b200.engine import StepEntry
    from ninfer_amd_mi50_b200.parts.feedforward import SparseMoeSwiglu
    got, chosen = {}, {}
    record = runner.graphs is None
    for st in steps:
        entries = []
        for e in st["entries"]:
            if not runner.cache.is_open(e["id"]):
                runner.open(e["id"])
            entries.append(StepEntry(e["id"], e["tokens"], e["want"]))
        SparseMoeSwiglu.record_routing = [] if record else None
        try:
            out = runner.step(entries)
            routing = [i.long().cpu() for i in SparseMoeSwiglu.record_routing or []]
        finally:
            SparseMoeSwiglu.record_routing = None
        r = row = 0
        for e in st["entries"]:
            n, m = len(e["want"]), len(e["tokens"])
            got.setdefault(e["id"], []).append(out[r:r + n].double().cpu())
            chosen.setdefault(e["id"], []).append([i[row:row + m] for i in routing])
            r, row = r + n, row + m
        for rid in st["end"]:
            runner.close(rid)
        runner.cache.check()
    kernels.check_status("schedule")
    return {k: torch.cat(v) for k, v in got.items()}, {k: [torch.cat(run_) for run_ in zip(*v)] for k, v in chosen.items()}


def run(runner, steps):
    return run_chosen(runner, steps)[0]


def plain(cfg, w, tokens, forced=None):
    return PN.forward(cfg, w, list(tokens), forced)[0]


def touchy_rows(cfg, w, tokens, want, tries=2, forced=None):
    """Rows whose logits move by more than 2 % of the scale when every projection's output is disturbed by
    2^-9 of its size (a softmax that rests on two equal scores, a norm of a sum that nearly cancels), the choice of
    experts being `forced` or the undisturbed model's."""
    if forced is None:
        own = []
        PN.forward(cfg, w, list(tokens), None, own)
        forced = [idx for _, idx in own]
    scale = want.abs().max().item()
    out = torch.zeros(want.shape[0], dtype=torch.bool)
    try:
        for i in range(tries):
            PN.NOISE = (torch.Generator().manual_seed(50 + i), 2.0 ** -9)
            out |= (plain(cfg, w, tokens, forced) - want).abs().max(dim=1).values / scale > 2e-2
    finally:
        PN.NOISE = None
    return out


def reference(cfg, w, tokens, chosen, want, touchy):
    """(logits, touchy rows) to compare a bfloat16 run with: where rounding made the engine choose other experts than
    the plain model - only ever at a close call - the plain model is run with the engine's choice."""
    own = []
    PN.forward(cfg, w, list(tokens), None, own)
    if all(torch.equal(a.sort(-1).values, b.sort(-1).values) for a, (_, b) in zip(chosen, own)):
        return want, touchy
    seen = []
    want = PN.forward(cfg, w, list(tokens), chosen, seen)[0]
    for idx, (z, _) in zip(chosen, seen):
        worst, kth = torch.gather(z, 1, idx).min(dim=1).values, torch.topk(z, idx.shape[1], dim=1).values[:, -1]
        assert (kth - worst).max() <= 0.06 * z.abs().max(), "an expert was chosen that is not among the best"
    return want, touchy_rows(cfg, w, tokens, want, tries=1, forced=chosen)


def check(runner, steps, cfg, w, reqs, dtype, what, want=None, touchy=None):
    """Drive a schedule that asks for every position and compare each request with the plain model."""
    got, chosen = run_chosen(runner, steps)
    for r, t in reqs.items():
        ref = want[r] if want is not None else plain(cfg, w, t)
        if dtype == "float32":
            compare(got[r], ref, dtype, f"{what} {r}")
        else:
            rough = touchy[r] if touchy is not None else touchy_rows(cfg, w, t, ref)
            ref, rough = reference(cfg, w, t, chosen[r], ref, rough)
            compare(got[r], ref, dtype, f"{what} {r}", rough)
    return got


def compare(got, want, dtype, what, touchy=None):
    """float32 is the sharp comparison: 1e-4 of the largest logit for every row.  bfloat16 rounds every
    activation between kernels to 8 bits: every row within 6 %, the median row (of 16 rows or more) within
    1.5 %; rows found `touchy` only have to be finite."""
    scale = want.abs().max().item()
    err = (got - want).abs().max(dim=1).values / scale
    assert torch.isfinite(got).all(), what
    if dtype == "float32":
        assert err.max().item() <= 1e-4, f"{what}: row {int(err.argmax())} of {len(err)} differs by {err.max().item():.3e} of the scale"
        return
    if touchy is not None:
        assert len(touchy) < 16 or touchy.float().mean().item() <= 0.5, f"{what}: {int(touchy.sum())} of {len(touchy)} rows are touchy"
        err = err[~touchy]
    if len(err):
        assert err.max().item() <= 6e-2, f"{what}: row {int(err.argmax())} of {len(err)} steady rows differs by {err.max().item():.3e} of the scale"
    if len(err) >= 16:
        assert err.median().item() <= 1.5e-2, f"{what}: the median row differs by {err.median().item():.3e} of the scale"


@pytest.fixture(scope="module", params=sorted(NC.CONFIGS))
def folder(request, tmp_path_factory):
    cfg, seed = NC.CONFIGS[request.param]
    d = str(tmp_path_factory.mktemp("nolesun") / request.param)
    NC.write_folder(cfg, seed, d)
    cfg, w = NC.read_folder(d)
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
    check(runner, make(reqs), cfg, w, reqs, dtype, f"{name} {how}", want, touchy)
    assert all(n == pool // 16 for n in runner.cache.pages_free())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_through_the_kernels_for_many_rows(folder, dtype):
    """More than 128 rows in one portion (the tcgen05 attention kernels, library products, router logits on tensor
    cores), then a second portion on top of the first one's cache, then decoded rows, beside a short request."""
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
    check(load(d, dtype, max_context=512, page_size=64), steps, cfg, w, {"a": a, "b": b, "c": a[:150], "d": b[:1]}, dtype, name)


def test_the_stream_after_every_layer_run(folder):
    """What a layer run leaves in the stream, looked at between the runs."""
    name, d, cfg, w, reqs, want, touchy = folder
    runner = load(d, "float32")
    seen = []
    runner.model.probe = lambda i, h: seen.append(h.double().cpu().clone())
    run(runner, schedules.whole({"a": reqs["r3"]}))
    ref = PN.forward(cfg, w, reqs["r3"])[1]
    assert len(seen) == len(ref)
    for i, (a, b) in enumerate(zip(seen, ref)):
        assert (a - b).abs().max() <= 1e-4 * b.abs().max(), i


# ---- each mechanism alone ---------------------------------------------------------------------

def check_alone(tmp_path, cfg, dtype, n_tokens=90, cuts=(2, 3, 40, 1, 16), replace=None, scale=None, seed=7, **opt):
    d = NC.write_folder(cfg, seed, str(tmp_path / "m"), replace=replace, scale=scale)
    cfg, w = NC.read_folder(d)
    toks = random_tokens(n_tokens, cfg["vocab"], seed)
    want = plain(cfg, w, toks)
    touchy = touchy_rows(cfg, w, toks, want)
    got = check(load(d, dtype, **opt), schedules.whole({"a": toks}), cfg, w, {"a": toks}, dtype, "whole", {"a": want}, {"a": touchy})["a"]
    if cuts:
        check(load(d, dtype, **opt), schedules.portions({"a": toks}, cuts=list(cuts)), cfg, w, {"a": toks}, dtype, "portions", {"a": want}, {"a": touchy})
    return cfg, w, toks, want, got


def distance(a, b):
    return ((a - b).abs().max() / b.abs().max()).item()


SSM, DELTA = NC.state_space(2, 8, 8, 1, 2, 1), NC.delta(2, 1, 8, 8, 2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("left", [
    NC.attention(2, 1, 8, 8, 0.4, rot=(100.0, 4)),                     # one row a token, equal sizes
    NC.attention(4, 2, 16, 16, 0.3),                                   # nothing turned
    NC.attention(4, 4, 32, 32, 0.2, rot=(10000.0, 32)),                # the whole head, as many key heads as query heads
    NC.attention(6, 3, 16, 40, 0.3, rot=(50.0, 10)),                   # values wider than keys
    NC.attention(3, 1, 24, 6, 0.3, rot=(700.0, 24)),                   # keys wider than values
    NC.attention(8, 8, 64, 64, 0.15, rot=(1e6, 16)),
    NC.attention(2, 1, 48, 48, 0.2, rot=(300.0, 20)),                  # a size without a split-key kernel
])
@pytest.mark.parametrize("kind", ["first", "second"])
def test_attention_alone(tmp_path, dtype, left, kind):
    """Beside a recurrence that adds nothing; in the second kind capped, gated, biased and in interleaved pairs."""
    cfg = NC.model([NC.first(left, SSM)] if kind == "first" else [NC.second(dict(left, softcap=3.0), DELTA)], width=72)
    width = 2 * 8
    check_alone(tmp_path, cfg, dtype, n_tokens=150, replace={"l0.mix.right.o": torch.zeros(72, width)})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_piece_of_the_attentions_changes_the_answer(tmp_path, dtype):
    """The plain model without one of the pieces differs from the engine by far more than rounding."""
    left = NC.attention(4, 2, 16, 16, 0.5, rot=(20.0, 8), softcap=2.0)
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model([NC.second(left, DELTA)]), dtype, cuts=None,
                                          replace={"l0.mix.right.o": torch.zeros(80, 16)})
    for name in ("q.b", "k.b", "v.b", "o.b", "g"):
        name = "l0.mix.left." + name
        assert distance(got, plain(cfg, dict(w, **{name: torch.zeros_like(w[name])}), toks)) > 0.05, name
    for change in ({"softcap": 4.0}, {"rot": None}, {"rot": {"base": 20.0, "dims": 6}}, {"rot": {"base": 40.0, "dims": 8}}, {"scale": 0.4}):
        cfg2 = json.loads(json.dumps(cfg))
        cfg2["layers"][0]["mixer"]["left"].update(change)
        assert distance(got, plain(cfg2, w, toks)) > 0.05, change
    saved = PN.turn
    try:
        PN.turn = lambda x, base, dims, neighbours: saved(x, base, dims, not neighbours)
        assert distance(got, plain(cfg, w, toks)) > 0.05
    finally:
        PN.turn = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("right", [NC.state_space(4, 16, 24, 2, 4, 1), NC.state_space(3, 10, 12, 1, 1, 3), NC.state_space(6, 64, 128, 3, 2, 6),
                                   NC.state_space(1, 33, 40, 1, 8, 3), NC.state_space(2, 24, 200, 2, 3, 2)])
def test_state_space_beside_nothing(tmp_path, dtype, right):
    check_alone(tmp_path, NC.model([NC.first(NC.attention(1, 1, 8, 8, 0.3), right)], width=72), dtype, n_tokens=140,
                replace={"l0.mix.left.o": torch.zeros(72, 8)})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("right", [NC.delta(4, 2, 16, 24, 4), NC.delta(3, 3, 9, 7, 1), NC.delta(6, 1, 64, 64, 3), NC.delta(2, 2, 128, 32, 2),
                                   NC.delta(5, 5, 100, 21, 8), NC.delta(4, 1, 200, 16, 4), NC.delta(1, 1, 4, 6, 2)])
def test_delta_rule_beside_nothing(tmp_path, dtype, right):
    cfg = NC.model([NC.second(NC.attention(1, 1, 8, 8, 0.3, softcap=5.0), right)], width=72)
    check_alone(tmp_path, cfg, dtype, n_tokens=140, replace={"l0.mix.left.o": torch.zeros(72, 8), "l0.mix.left.o.b": torch.zeros(72)})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_piece_of_the_recurrences_changes_the_answer(tmp_path, dtype):
    layers = [NC.first(NC.attention(1, 1, 8, 8, 0.3), NC.state_space(4, 16, 24, 2, 3, 2)),
              NC.second(NC.attention(1, 1, 8, 8, 0.3, softcap=5.0), NC.delta(4, 2, 16, 24, 3))]
    zero = {f"l{i}.mix.left.{n}": torch.zeros(80, *s) for i, n, s in ((0, "o", (8,)), (1, "o", (8,)), (1, "o.b", ()))}
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model(layers), dtype, cuts=None, replace=zero)
    for n in ("l0.mix.right.conv.b", "l0.mix.right.D", "l0.mix.right.dt_bias", "l0.mix.right.A_log", "l1.mix.right.A_log",
              "l1.mix.right.dt_bias", "l1.mix.right.a", "l1.mix.right.b", "l1.mix.right.norm", "l0.mix.right.norm"):
        other = torch.ones_like(w[n]) if n.endswith("norm") else torch.zeros_like(w[n])
        assert distance(got, plain(cfg, dict(w, **{n: other}), toks)) > 0.02, n
    for n in ("l0.mix.right.conv", "l1.mix.right.q.conv", "l1.mix.right.k.conv", "l1.mix.right.v.conv"):
        flipped = torch.flip(w[n], [1])
        assert distance(got, plain(cfg, dict(w, **{n: flipped}), toks)) > 0.05, n
    cfg2 = json.loads(json.dumps(cfg))
    cfg2["layers"][0]["mixer"]["right"]["norm_groups"] = 1
    assert distance(got, plain(cfg2, w, toks)) > 0.02
    saved = PN.delta_step
    for wrong in (lambda S, q, k, v, g, b: (saved(S, q, k, v, g, b)[0], (g * S).T @ q),                      # read before the write
                  lambda S, q, k, v, g, b: (lambda N: (N, N.T @ q))(g * S + torch.outer(k, b * v)),          # nothing taken off
                  lambda S, q, k, v, g, b: (lambda N: (N, N.T @ q))(g * S + torch.outer(k, b * (v - S.T @ k)))):   # not decayed first
        try:
            PN.delta_step = wrong
            assert distance(got, plain(cfg, w, toks)) > 0.02
        finally:
            PN.delta_step = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [96, 66, 520, 1200])
def test_norms_around_the_sublayers_their_scales_and_the_mixers_factors(tmp_path, dtype, width):
    layers = [NC.first(NC.attention(2, 1, 8, 8, 0.3), SSM, (0.4, 1.7), NC.dense(40)), NC.second(NC.attention(2, 1, 8, 8, 0.3, softcap=5.0), DELTA, (1.9, 0.3))]
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model(layers, width=width, eps=2e-2, scale=4.5), dtype, n_tokens=60,
                                          scale={".right.o": 0.5, ".left.o": 0.5, ".down": 0.5})
    for i, names in ((0, ("norm1", "norm1b", "norm2", "norm2b", "ls1", "ls2")), (1, ("norm1", "norm1b", "ls1"))):
        for n in names:
            n = f"l{i}.{n}"
            assert distance(got, plain(cfg, dict(w, **{n: torch.zeros_like(w[n]) if "norm" in n else torch.ones_like(w[n])}), toks)) > 0.01, n
    changes = [{"norm": {"eps": 1e-6}}, {"embedding": {"scale": 1.0}}]
    for i in (0, 1):
        for k in ("left_scale", "right_scale"):
            L = json.loads(json.dumps(cfg["layers"]))
            L[i]["mixer"][k] *= 3.0
            changes.append({"layers": L})
    for change in changes:
        assert distance(got, plain(dict(cfg, **change), w, toks)) > 0.01, change


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,rows", [(88, 3), (200, 300), (51, 12)])
def test_squared_relu_feed_forward(tmp_path, dtype, ff, rows):
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model([NC.first(NC.attention(2, 1, 8, 8, 0.3), SSM, mlp=NC.dense(ff))]), dtype,
                                          n_tokens=rows, cuts=None, max_context=512)
    saved = PN.relu2_mlp
    try:
        PN.relu2_mlp = lambda h, w_, p: PN.proj(torch.relu(PN.proj(h, w_[p + "up"])), w_[p + "down"])
        assert distance(got, plain(cfg, w, toks)) > 0.05
    finally:
        PN.relu2_mlp = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,ff,width", [(12, 3, 40, 80), (5, 1, 24, 72), (4, 4, 33, 66), (40, 6, 64, 128)])
@pytest.mark.parametrize("rows", [1, 7, 14, 30, 60, 200])
def test_experts_with_a_bias_on_the_routers_logits(tmp_path, dtype, experts, top, ff, width, rows):
    """Every arrangement of the routing (one cluster, one launch, inside the experts' launch, tensor-core logits).
    Where rounding turns a close call the plain model follows the engine's choice."""
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model([NC.first(NC.attention(2, 1, 8, 8, 0.3), SSM, mlp=NC.moe(ff, experts, top))],
                                                             width=width), dtype, n_tokens=rows, cuts=None)
    if top < experts and rows >= 7:
        assert distance(got, plain(cfg, dict(w, **{"l0.mlp.router.b": torch.zeros(experts)}), toks)) > 0.05
    if top > 1 and rows >= 7:
        saved = PN.choose
        try:
            def over_all(z, k):
                best, idx = torch.topk(z, k, dim=-1)
                return idx, torch.full_like(best, 1.0 / k)
            PN.choose = over_all
            assert distance(got, plain(cfg, w, toks)) > 0.02
        finally:
            PN.choose = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("loop", [(0, 1, 4), (1, 2, 2), (0, 2, 2), (1, 2, 1)])
def test_a_repeated_run_enters_through_its_matrix_with_state_of_its_own(tmp_path, dtype, loop):
    layers = [NC.first(NC.attention(2, 1, 16, 16, 0.3, rot=(50.0, 8)), SSM), NC.second(NC.attention(2, 1, 16, 16, 0.3, softcap=4.0), DELTA)]
    cfg, w, toks, want, got = check_alone(tmp_path, NC.model(layers, loop=loop, scale=2.5), dtype, n_tokens=80)
    W = cfg["width"]
    m = w["loop.in"]
    for other in (torch.cat([m[:, W:], m[:, :W]], 1), torch.cat([m[:, :W], torch.zeros(W, W)], 1), torch.cat([torch.zeros(W, W), m[:, W:]], 1)):
        assert distance(got, plain(cfg, dict(w, **{"loop.in": other}), toks)) > 0.05
    assert distance(got, plain(cfg, dict(w, **{"loop.step": torch.zeros_like(w["loop.step"])}), toks)) > 0.05
    if loop[2] > 1:
        assert distance(got, plain(cfg, dict(w, **{"loop.step": torch.flip(w["loop.step"], [0])}), toks)) > 0.03
        assert distance(got, plain(dict(cfg, loop=dict(cfg["loop"], times=loop[2] - 1)), w, toks)) > 0.05


# ---- kernels against plain arithmetic -----------------------------------------------------------------

def step_context(lens, pos0, dtype, slots=None):
    from ninfer_amd_mi50_b200.parts.base import StepContext
    S, T = len(lens), sum(lens)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    row0 = [sum(lens[:i]) for i in range(S + 1)]
    return StepContext(dtype=dtype, device=torch.device("cuda"), T=T, S=S, token_ids=i32([0] * T),
                       positions=i32([p + j for n, p in zip(lens, pos0) for j in range(n)]), row_seg=i32([s for s, n in enumerate(lens) for _ in range(n)]),
                       seg_row0=i32(row0), seg_pos0=i32(pos0), seg_slot=i32(slots or list(range(S))), logit_rows=i32([0]),
                       seg_len_host=list(lens), seg_pos0_host=list(pos0), max_rows_per_seg=max(lens), max_context=max(n + p for n, p in zip(lens, pos0)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 16, 24), (3, 3, 9, 7), (6, 1, 64, 64), (2, 2, 128, 40), (4, 1, 100, 16), (2, 1, 160, 33), (1, 1, 256, 8), (2, 2, 1, 1)])
@pytest.mark.parametrize("strong", [False, True])
def test_delta_rule_kernels_in_every_length(H, G, D, V, dtype, strong):
    """Chunks of every length, from and into slots in another order, then single rows on top; with decays near one
    and with decays that wipe the state out."""
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(3)
    lens, off = [1, 8, 23, 2, 9, 64], 4
    slots, n_slots = [5, 0, 3, 1, 7, 2], 8
    width = 2 * G * D + H * V
    rand = lambda *s: torch.randn(*s, device="cuda", generator=g)
    state = rand(n_slots, off + H * V * D) * 0.3
    dt_bias, A_log = rand(H), rand(H) + (2.0 if strong else -3.0)
    ref = {s: state[s, off:].double().cpu().view(H, V, D).transpose(1, 2).clone() for s in range(n_slots)}
    for lens in (lens, [1] * 6):
        ctx = step_context(lens, [0] * 6, dtype, slots)
        T = sum(lens)
        qkv = rand(T, width).to(dtype)
        ab = (rand(T, 2 * H + 3) * 2).to(dtype)
        out = kernels.delta_rule(qkv, 0, G * D, 2 * G * D, ab, 1, H + 2, dt_bias, A_log, D ** -0.5, state, off, ctx, H, G, D, V)
        x, y = qkv.double().cpu(), ab.double().cpu()
        q, k = PN.unit(x[:, :G * D].view(T, G, D)) * D ** -0.5, PN.unit(x[:, G * D:2 * G * D].view(T, G, D))
        v = x[:, 2 * G * D:].view(T, H, V)
        dec = torch.exp(-torch.exp(A_log.double().cpu()) * PN.softplus(y[:, 1:1 + H] + dt_bias.double().cpu()))
        beta = torch.sigmoid(y[:, H + 2:2 * H + 2])
        want = torch.zeros(T, H, V, dtype=torch.float64)
        r = 0
        for s, n in zip(slots, lens):
            for t in range(r, r + n):
                for h in range(H):
                    ref[s][h], want[t, h] = PN.delta_step(ref[s][h], q[t, h // (H // G)], k[t, h // (H // G)], v[t, h], dec[t, h], beta[t, h])
            r += n
        assert (out.double().cpu().view(T, H, V) - want).abs().max() <= 3e-5 * max(1.0, want.abs().max().item()), lens
        for s in slots:
            assert (state[s, off:].double().cpu().view(H, V, D).transpose(1, 2) - ref[s]).abs().max() <= 3e-5 * max(1.0, ref[s].abs().max().item())


def test_delta_rule_state_does_not_depend_on_the_cut():
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(4)
    H, G, D, V, T = 2, 1, 64, 32, 100
    qkv = torch.randn(T, 2 * G * D + H * V, device="cuda", generator=g)
    ab = torch.randn(T, 2 * H, device="cuda", generator=g)
    one = torch.zeros(H, device="cuda")
    outs = []
    for cuts in ([100], [2, 3, 8, 16, 1, 1, 40, 29], [1] * 100):
        state = torch.zeros(1, H * V * D, device="cuda")
        r, o = 0, []
        for n in cuts:
            ctx = step_context([n], [r], torch.float32)
            o.append(kernels.delta_rule(qkv[r:r + n].contiguous(), 0, G * D, 2 * G * D, ab[r:r + n].contiguous(), 0, H, one, one, 1.0, state, 0,
                                        ctx, H, G, D, V))
            r += n
        outs.append((torch.cat(o), state))
    for o, s in outs[1:]:
        assert (o - outs[0][0]).abs().max() <= 1e-5 and (s - outs[0][1]).abs().max() <= 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [8, 66, 100, 512, 2048, 4100, 9000])
@pytest.mark.parametrize("form", ["pair", "single", "routed", "none", "plain_sum"])
def test_residual_norm_in_every_form(W, dtype, form):
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(5)
    T, k = 11, 3
    rand = lambda *s: torch.randn(*s, device="cuda", generator=g)
    h, a, b = rand(T, W), (rand(T, W) * 3).to(dtype), rand(T, W).to(dtype)
    y, inv = rand(T * k, W).to(dtype), torch.randperm(T * k, device="cuda", generator=g).to(torch.int32)
    wts, bias, w1, w2 = torch.rand(T, k, device="cuda", generator=g), rand(W), rand(W), rand(W)
    args = {"pair": dict(a=a, scale_a=0.7, b=b, scale_b=-1.3, bias=bias), "single": dict(a=a), "none": {}, "plain_sum": dict(a=a, bias=bias),
            "routed": dict(routed=(y, inv, wts, k))}[form]
    D = lambda t: t.double().cpu()
    d = torch.zeros(T, W, dtype=torch.float64)
    if "a" in args:
        d = args.get("scale_a", 1.0) * D(a) + (args["scale_b"] * D(b) if "b" in args else 0) + (D(bias) if "bias" in args else 0)
    elif form == "routed":
        d = (D(wts)[:, :, None] * D(y)[inv.long().cpu()].view(T, k, W)).sum(1)
    inner = form in ("pair", "single", "routed")
    if inner:
        args.update(inner_weight=w1, inner_eps=1e-2)
        d = d / torch.sqrt((d * d).mean(1, keepdim=True) + 1e-2) * D(w1)
    x = D(h) + d
    normed = x / torch.sqrt((x * x).mean(1, keepdim=True) + 1e-3) * D(w2)
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    # some rows only, the stream left as it is
    rows = torch.tensor([7, 0, 3], dtype=torch.int32, device="cuda")
    before, out = h.clone(), torch.empty(3, W, dtype=dtype, device="cuda")
    kernels.residual_norm(h, w2, 1e-3, out, rows=rows, **args)
    assert torch.equal(h, before) and (D(out) - normed[[7, 0, 3]]).abs().max() <= tol * normed.abs().max()
    # all rows into a range of columns of wider ones
    wide = torch.full((T, 2 * W + 8), 5.0, dtype=dtype, device="cuda")
    kernels.residual_norm(h.clone(), w2, 1e-3, wide[:, W + 4:2 * W + 4], **args)
    assert (D(wide[:, W + 4:2 * W + 4]) - normed).abs().max() <= tol * normed.abs().max()
    assert (wide[:, :W + 4] == 5).all() and (wide[:, 2 * W + 4:] == 5).all()
    # the stream itself, and its rounding
    out = torch.empty(T, W, dtype=dtype, device="cuda")
    kernels.residual_norm(h, None, 0.0, out, **args)
    assert (D(h) - x).abs().max() <= (2e-5 if form != "routed" or dtype == torch.float32 else 3e-2) * x.abs().max()
    assert torch.equal(out, h.to(dtype))
    kernels.residual_norm(before, None, 0.0, None, **args)
    assert torch.equal(before, h)


def paged(lens, G, D, page, seed=5):
    g = torch.Generator(device="cuda").manual_seed(seed)
    S, width = len(lens), (max(lens) + page - 1) // page
    pages = (torch.randn(S * width + 1, 2, G, page, D, device="cuda", generator=g) * 0.7).bfloat16()
    table = torch.randperm(S * width, device="cuda", generator=g).to(torch.int32).view(S, width)
    return pages, table, g


@pytest.mark.parametrize("D", [16, 48, 64, 96, 128])
@pytest.mark.parametrize("G,H", [(8, 16), (2, 16)])
@pytest.mark.parametrize("what", ["few", "many", "prompt", "mixed"])
@pytest.mark.parametrize("cap", [0.8, 30.0])
def test_capped_scores_in_every_attention_kernel(D, G, H, what, cap):
    """One CTA a block of keys, the persistent form, the two flash kernels, and a mixed step, against the plain
    kernel of one warp a row and head on the same cache - and that one against plain arithmetic."""
    from ninfer_amd_mi50_b200 import kernels
    page = 16
    held = {"few": [1 + (53 * i) % 200 for i in range(3)], "many": [1 + (37 * i) % 330 for i in range(70)],
            "prompt": [150, 40], "mixed": [140, 61, 1, 333]}[what]
    rows = {"few": [1] * 3, "many": [1] * 70, "prompt": [150, 33], "mixed": [130, 1, 1, 2]}[what]
    pages, table, g = paged(held, G, D, page)
    ctx = step_context(rows, [n - r for n, r in zip(held, rows)], torch.bfloat16)
    q = (torch.randn(sum(rows), H * D, device="cuda", generator=g) * 1.5).bfloat16()
    scale = 1.5 * D ** -0.5
    attend = lambda: kernels.paged_attention(q, H, G, D, pages, table, page, ctx, 0, scale, softcap=cap)
    fast = attend()
    saved = kernels.TUNING["bf16_attention"]
    try:
        kernels.TUNING["bf16_attention"] = "generic"
        slow = attend()
        uncapped = kernels.paged_attention(q, H, G, D, pages, table, page, ctx, 0, scale)
    finally:
        kernels.TUNING["bf16_attention"] = saved
    kernels.check_status("capped attention")
    assert (fast.float() - slow.float()).abs().max() <= 2e-2 * slow.float().abs().max()
    if cap < 1:
        assert (uncapped.float() - slow.float()).abs().max() > 0.1 * slow.float().abs().max()
    r = 0
    for s, (n, m) in enumerate(zip(held, rows)):
        k, v = ([pages[table[s].long(), i].transpose(0, 1).reshape(G, -1, D)[:, :n].double().cpu() for i in (0, 1)])
        t = r + m - 1                                                      # the segment's last row sees everything
        for h in (0, H - 1):
            z = cap * torch.tanh((k[h // (H // G)] @ q[t, h * D:(h + 1) * D].double().cpu()) * scale / cap)
            want = torch.softmax(z, 0) @ v[h // (H // G)]
            assert (slow[t, h * D:(h + 1) * D].double().cpu() - want).abs().max() <= 1e-2
        r += m


@pytest.mark.parametrize("rows", [1, 5, 8, 12, 20, 32, 50, 200])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_router_bias_in_every_form_of_the_routing(rows, dtype):
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(6)
    E, k, H = 24, 3, 96
    x = torch.randn(rows, H, device="cuda", generator=g).to(dtype)
    w = torch.randn(E, H, device="cuda", generator=g).bfloat16().float()
    bias = torch.randn(E, device="cuda", generator=g) * 6
    idx, wts, _, plan = kernels.route(x, w, E, k, True, split=kernels.split_router(w), bias=bias)
    z = x.double().cpu() @ w.double().cpu().T + bias.double().cpu()
    best, want = torch.topk(z, k, dim=-1)
    assert torch.equal(idx.long().cpu(), want)
    assert (wts.double().cpu() - torch.softmax(best, -1)).abs().max() <= 1e-4
    assert int(plan.offsets[-1]) == rows * k


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Dv,P,ld,g0", [(3, 6, 16, 40, 5), (4, 24, 32, 200, 100), (2, 64, 64, 128, 0), (5, 8, 16, 48, 8)])
def test_the_gate_takes_the_values_out_of_wider_heads(H, Dv, P, ld, g0, dtype):
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(7)
    o = torch.randn(9, H * P, device="cuda", generator=g).to(dtype)
    src = torch.randn(9, ld, device="cuda", generator=g)
    out = kernels.sigmoid_gate_rows(o, src, g0, heads=H, Dv=Dv)
    want = o.double().cpu().view(9, H, P)[..., :Dv].reshape(9, H * Dv) * torch.sigmoid(src.double().cpu()[:, g0:g0 + H * Dv])
    assert out.shape == (9, H * Dv) and (out.double().cpu() - want).abs().max() <= (1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,K,col0,ld", [(24, 4, 8, 40), (7, 3, 1, 12), (64, 1, 0, 64), (16, 8, 16, 48)])
def test_single_rows_shift_the_convolutions_inputs_themselves(C, K, col0, ld, dtype):
    from ninfer_amd_mi50_b200 import kernels
    g = torch.Generator(device="cuda").manual_seed(8)
    taps = torch.randn(K, C, device="cuda", generator=g)
    src = torch.randn(12, ld, device="cuda", generator=g).to(dtype)
    outs = []
    for cuts in ([12], [1] * 12, [5, 1, 1, 2, 1, 2]):
        state = torch.zeros(1, max(1, (K - 1) * C), device="cuda")
        r, o = 0, []
        for n in cuts:
            o.append(kernels.causal_conv_silu(src[r:r + n].contiguous(), col0, C, taps, None, state, step_context([n], [r], dtype)))
            r += n
        outs.append((torch.cat(o), state))
    for o, s in outs[1:]:
        assert torch.equal(o, outs[0][0]) and torch.equal(s, outs[0][1])
    want = PN.silu(PN.short_conv(src.double().cpu()[:, col0:col0 + C], taps.double().cpu().T))
    assert (outs[0][0].double().cpu() - want).abs().max() <= (1e-4 if dtype == torch.float32 else 2e-2) * want.abs().max()


# ---- keys far away, states that must not be lost ---------------------------------------------------------

def twin_tokens(w0, width, seed=9):
    """Two tokens whose embeddings share the first half and have opposite second halves (an RMS norm treats
    both alike): `replace`-ready embedding with them as tokens 400 and 398."""
    g = torch.Generator().manual_seed(seed)
    a, b = torch.randn(width // 2, generator=g, dtype=torch.float64) * 0.3, torch.randn(width // 2, generator=g, dtype=torch.float64) * 0.3
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
@pytest.mark.parametrize("left,kind", [(NC.attention(4, 2, 32, 32, 0.6), "first"), (NC.attention(4, 1, 32, 24, 0.6), "first"),
                                       (NC.attention(2, 1, 128, 128, 0.15, softcap=25.0), "second"),
                                       (NC.attention(2, 2, 24, 40, 0.6, softcap=30.0), "second"), (NC.attention(4, 1, 64, 64, 0.3, softcap=25.0), "second")])
def test_one_far_key_among_hundreds_is_found(tmp_path, dtype, left, kind):
    """Queries and keys are made of the first half of the width by one matrix, so a query's best keys are those of
    tokens whose first half is its own.  A token and its twin (same first half, opposite second half, from which
    the values come) stand last and once before - at a page's first or last place, or hundreds back: a key that is
    lost, or read from the wrong place, changes the answer wholly.  In a prompt, in portions and decoded."""
    W = 64
    cfg = NC.model([NC.first(left, SSM)] if kind == "first" else [NC.second(left, DELTA)], width=W, vocab=401)
    d0 = NC.write_folder(cfg, 3, str(tmp_path / "m0"))
    _, w0 = NC.read_folder(d0)
    g = torch.Generator().manual_seed(4)
    rand = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64) * 0.2
    H, G, D, Dv = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
    wk, wv = rand(G * D, W), rand(G * Dv, W)
    wk[:, W // 2:] = 0.0
    wv[:, :W // 2] = 0.0
    replace = {"embed": twin_tokens(w0, W), "l0.norm1": torch.zeros(W), "l0.mix.left.k": wk, "l0.mix.left.v": wv,
               "l0.mix.left.q": wk.view(G, D, W).repeat_interleave(H // G, dim=0).reshape(H * D, W), "l0.mix.right.o": torch.zeros(W, 16),
               "l0.ls1": torch.full((W,), 2.0)}
    if kind == "second":
        replace.update({f"l0.mix.left.{n}.b": torch.zeros(k) for n, k in (("q", H * D), ("k", G * D), ("v", G * Dv), ("o", W))})
    d = NC.write_folder(cfg, 3, str(tmp_path / "m"), replace=replace)
    cfg, w = NC.read_folder(d)
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


@pytest.mark.parametrize("kind", ["first", "second"])
def test_a_token_far_back_reaches_the_answer_through_the_state(tmp_path, kind):
    """Slow decays: what one token left in the state - and, just before the end, in the convolution's inputs - still
    shows hundreds of tokens later, in 32-bit beyond doubt.  At the first tokens, at chunk and page borders, in a
    prompt, in portions and decoded."""
    W = 64
    if kind == "first":
        right = NC.state_space(2, 16, 64, 1, 4, 1)
        cfg = NC.model([NC.first(NC.attention(1, 1, 8, 8, 0.3), right)], width=W, vocab=401)
        replace = {"l0.mix.left.o": torch.zeros(W, 8), "l0.mix.right.dt_bias": torch.full((2,), -2.0)}
    else:
        right = NC.delta(2, 1, 128, 16, 4)
        cfg = NC.model([NC.second(NC.attention(1, 1, 8, 8, 0.3, softcap=5.0), right)], width=W, vocab=401)
        replace = {"l0.mix.left.o": torch.zeros(W, 8), "l0.mix.left.o.b": torch.zeros(W)}
    replace["l0.mix.right.A_log"] = torch.full((2,), -8.0)
    d = NC.write_folder(cfg, 3, str(tmp_path / "m"), replace=replace)
    cfg, w = NC.read_folder(d)
    n = 200
    base = [1 + (i * 7) % 397 for i in range(n)]
    for place in (0, 1, 7, 8, 15, 16, 63, 64, 120, 193, 196, 198):
        toks = list(base)
        toks[place] = 400
        want = plain(cfg, w, toks)[-1:]
        assert distance(plain(cfg, w, base)[-1:], want) > 2e-3, "the token does not matter"
        for how in ("prompt", "portions", "decoded"):
            got = run(load(d, "float32"), steps_for(toks, how, [0, 2, 9, 14, 16, 19, 64, 67, 150]))
            compare(got["a"], want, "float32", f"place {place} {how}")


def test_the_first_tokens_start_from_nothing(folder):
    """Slots and pages that others have used: a request's first tokens see zeros before their start."""
    name, d, cfg, w, reqs, want, touchy = folder
    runner = load(d, "float32", num_sequences=2)
    run(runner, schedules.whole({"x": reqs["r2"], "y": reqs["r5"]}))
    for cuts in ([1, 1, 1, 1, 1], [2, 3], [4, 1]):
        got = run(runner, schedules.portions({"a": reqs["r1"]}, cuts=cuts))
        compare(got["a"], want["r1"], "float32", f"{name} {cuts}")


# ---- the engine around the design ---------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folder, dtype):
    name, d, cfg, w, reqs, want, touchy = folder
    toks = random_tokens(236, cfg["vocab"], 77)
    runner = load(d, dtype)
    check(runner, schedules.tail_decoded({"a": toks}, tail=229), cfg, w, {"a": toks}, dtype, f"{name} long decoding")
    assert all(n == 1024 // 16 for n in runner.cache.pages_free())


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
        assert (together[r] - alone[r]).abs().max() <= 2e-5 * alone[r].abs().max(), r


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
            assert diff.max() <= 4e-5
        else:       # a row is served by another kernel when it arrives alone, which rounds elsewhere
            assert diff[~touchy["r2"]].max() <= 6e-2 and diff.median() <= 1.5e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decode_steps_replayed_from_graphs_equal_host_driven_ones(folder, dtype):
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
        assert not steady.any() or diff[steady].max() <= (1e-5 if dtype == "float32" else 4e-2), (r, diff.max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(folder, dtype):
    from ninfer_amd_mi50_b200.api import Ninfer
    name, d, cfg, w, reqs, want, touchy = folder
    prompts = [reqs["r1"], reqs["r3"], reqs["r4"], reqs["r0"][:40]]
    eng = Ninfer(d, max_context=128, prefill_chunk=16, num_sequences=3, dtype=dtype, page_size=16)
    got = eng.generate(prompts, max_new_tokens=10, temperature=0.0)
    for p, out in zip(prompts, got):
        assert len(out) == 10
        full = list(p) + list(out)
        ref = plain(cfg, w, full)
        shaky = torch.zeros(len(full), dtype=torch.bool)
        if dtype == "bfloat16":         # the same tokens once more, for the experts chosen
            chosen = run_chosen(load(d, dtype), schedules.whole({"a": full}))[1]["a"]
            ref, shaky = reference(cfg, w, full, chosen, ref, touchy_rows(cfg, w, full, ref))
        for k, t in enumerate(out):
            lg = ref[len(p) - 1 + k]
            # the engine's token is the plain model's, or (bfloat16) one whose logit is as good as ties go
            slack = 1e-4 if dtype == "float32" else 6e-2
            if not shaky[len(p) - 1 + k]:
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
    """`bin/ninfer` on a Nolesun folder, and on a folder with only config.json and a seed."""
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg0, seed = NC.CONFIGS["looped"]
    d = str(tmp_path / "m")
    if how == "folder":
        NC.write_folder(cfg0, seed, d)
    else:
        from ninfer_amd_mi50_b200.weights import write_random_model
        write_random_model(cfg0, seed, d)
    cfg, w = NC.read_folder(d)
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
    recomputed: its keys are written again from position 0, its states start from zero again, and the tokens are
    those of a roomy pool."""
    from ninfer_amd_mi50_b200.api import Ninfer
    name, d, cfg, w, reqs, want, touchy = folder
    prompts = [reqs["r0"][:50], reqs["r3"], reqs["r5"][:60]]
    roomy = Ninfer(d, max_context=128, prefill_chunk=32, num_sequences=3, dtype="float32", page_size=16)
    want_tokens = roomy.generate(prompts, max_new_tokens=24, temperature=0.8, top_k=20, seed=5)
    tight = Ninfer(d, max_context=128, prefill_chunk=32, num_sequences=3, dtype="float32", page_size=16, cache_tokens=160)
    got = tight.generate(prompts, max_new_tokens=24, temperature=0.8, top_k=20, seed=5)
    assert got == want_tokens
