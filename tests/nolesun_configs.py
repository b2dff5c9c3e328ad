"""Small Nolesun configurations for the tests, and a writer of model folders with lively weights.  The sizes are
awkward on purpose: head sizes that are equal and unequal, multiples of 16 and not, one key head and as many as
query heads, part of a head turned, all of it and nothing, one and several groups in the state-space mixer and its
norm, heads of the recurrences that share keys and that do not, one tap and several, a repeated run in the middle, at
either end and over everything, one pass and several, every expert chosen and one, layers without a feed-forward."""

import torch

import vekasun_configs as VC

read_folder = VC.read_folder


def attention(heads, kv_heads, dim, vdim, scale, rot=None, softcap=None):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        a["rot"] = {"base": rot[0], "dims": rot[1]}
    if softcap is not None:
        a["softcap"] = softcap
    return a


def state_space(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def first(left, right, scales=(0.7, 1.3), mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def second(left, right, scales=(1.1, 0.6), mlp=None):
    return dict(first(left, right, scales, mlp), type="parallel_2")


def model(layers, width=80, vocab=173, eps=1e-5, scale=None, loop=None):
    cfg = {"architecture": "Nolesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        cfg["embedding"] = {"scale": scale}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# a run of two in the middle, three passes; both mixers inside and outside of it
LOOPED = model([
    first(attention(4, 2, 32, 32, 0.2, rot=(300.0, 16)), state_space(6, 20, 24, 3, 3, 2), mlp=moe(40, 5, 2)),
    second(attention(6, 3, 16, 40, 0.3, rot=(100.0, 8), softcap=4.0), delta(4, 2, 24, 16, 4), mlp=dense(72)),
    first(attention(3, 1, 24, 48, 0.25, rot=(50.0, 24)), state_space(4, 32, 16, 1, 5, 1), mlp=moe(24, 3, 3)),
    second(attention(4, 4, 64, 64, 0.15, rot=(2000.0, 40), softcap=6.0), delta(3, 3, 40, 12, 2), mlp=None),
], width=96, scale=5.5, loop=(1, 3, 3))

# nothing a multiple of 8 where it can be helped, no factor on the embedding, the whole model repeated, a large eps
AWKWARD = model([
    second(attention(3, 1, 10, 14, 0.4, rot=(30.0, 6), softcap=2.5), delta(6, 2, 9, 7, 3), (0.9, 1.0), mlp=moe(20, 4, 1)),
    first(attention(2, 2, 12, 12, 0.35), state_space(3, 10, 12, 3, 4, 3), (1.0, 1.0), mlp=dense(36)),
    second(attention(2, 1, 20, 6, 0.3, softcap=50.0), delta(5, 1, 33, 21, 1), mlp=None),
], width=100, vocab=97, eps=3e-3, loop=(0, 3, 2))

# heads of 64 and 128 (the split-key, persistent and tcgen05 kernels, capped and not), wide recurrences, no loop
WIDE = model([
    first(attention(8, 2, 64, 64, 0.1, rot=(1000.0, 64)), state_space(4, 64, 64, 2, 4, 4), mlp=dense(96)),
    second(attention(8, 1, 128, 128, 0.08, rot=(250.0, 128), softcap=5.0), delta(4, 2, 128, 64, 4), mlp=moe(48, 8, 2)),
    second(attention(8, 8, 64, 64, 0.15, rot=(1000.0, 32), softcap=3.0), delta(2, 1, 160, 32, 4), mlp=moe(64, 12, 4)),
    first(attention(4, 1, 128, 128, 0.07, rot=(20000.0, 32)), state_space(2, 128, 128, 1, 2, 1), mlp=None),
], width=128, vocab=131, scale=3.0)

# one layer, run once through the entry of the repeated run
ONE_PASS = model([second(attention(2, 1, 48, 16, 0.25, rot=(77.0, 48), softcap=1.5), delta(2, 2, 16, 48, 8), mlp=dense(24))],
                 width=64, vocab=61, scale=2.0, loop=(0, 1, 1))

CONFIGS = {"looped": (LOOPED, 81), "awkward": (AWKWARD, 82), "wide": (WIDE, 83), "one_pass": (ONE_PASS, 84)}

# factors that take the random weights (standard deviation 0.02) out of their nearly linear range; a name ends with
# exactly one of these
LIVELY = {"embed": 10.0, "loop.in": 4.0, "loop.step": 25.0, ".left.q": 4.0, ".left.k": 4.0, ".left.v": 6.0, ".left.g": 10.0,
          ".left.q.b": 20.0, ".left.k.b": 20.0, ".left.v.b": 20.0, ".left.o.b": 10.0, ".left.o": 4.0,
          ".right.in": 4.0, ".right.conv": 15.0, ".right.conv.b": 15.0, ".right.q.conv": 25.0, ".right.k.conv": 25.0,
          ".right.v.conv": 25.0, ".right.dt_bias": 40.0, ".right.A_log": 40.0, ".right.D": 80.0, ".right.q": 4.0, ".right.k": 4.0,
          ".right.v": 7.0, ".right.a": 7.0, ".right.b": 8.0, ".right.g": 8.0, ".right.o": 4.0, ".up": 4.0, ".gate": 5.0,
          ".down": 4.0, ".router": 4.0, ".router.b": 50.0}


def lively_tensors(cfg, seed):
    """Norm weights around zero and channel scales that vary over the row."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    spread = lambda n=W: torch.rand(n, generator=g) * 1.2 - 0.6
    out = {"final.norm": spread()}
    for i, L in enumerate(cfg["layers"]):
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L["mlp"] else ()):
            out[f"l{i}.{n}"] = spread()
        for n in ("ls1",) + (("ls2",) if L["mlp"] else ()):
            out[f"l{i}.{n}"] = spread() + 1.0
        r = L["mixer"]["right"]
        out[f"l{i}.mix.right.norm"] = spread(r["vdim"] if L["type"] == "parallel_2" else r["heads"] * r["vdim"]) + 1.0
    return out


def write_folder(config, seed, out_dir, replace=None, scale=None):
    """A model folder with the engine's seeded random tensors scaled out of their linear range, the lively
    replacements above and whatever `replace` names on top; `scale` changes single factors."""
    new = lively_tensors(config, seed)
    new.update(replace or {})
    return VC.write_folder(config, seed, out_dir, replace=new, scale=dict(LIVELY, **(scale or {})))
