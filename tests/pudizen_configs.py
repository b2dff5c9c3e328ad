"""Small Pudizen configurations for the tests.  The sizes are awkward on purpose: widths that are no power of
two, key and value sizes that are equal (the head-major pages) and that differ (one row a token, or heads
widened with zeros), sizes that are no multiple of 8, one key head and as many as query heads, rotated
dimensions fewer than the head, all of it and none, plain and band-scaled frequencies, values that are turned
and that are not, windows from one token to more than a page, latents of 64 times something and not, one norm
group and several, with and without the hashed pair rows, layers without a feed-forward, every order of mixers."""

import torch

import vekasun_configs as VC

read_folder = VC.read_folder


def attention(heads, kv_heads, dim, vdim, scale, rot=None, scaling=None):
    """`rot` (base, dims); `scaling` (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def windowed(heads, kv_heads, dim, vdim, scale, size, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention_2", "mixer": m}


def latent(heads, dim, vdim, kv_rank, scale):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}}


def layer(mixer, ff=None):
    return dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def model(layers, width=96, vocab=113, eps=1e-5, groups=1, scale=None, bigram=None):
    c = {"architecture": "Pudizen", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "layers": layers}
    e = {}
    if scale is not None:
        e["scale"] = scale
    if bigram is not None:
        e["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if e:
        c["embedding"] = e
    return c


# every mixer twice, in another form each time; head-major pages, one row a token, widened heads
MIXED = model([
    layer(attention(6, 2, 16, 16, 0.3, rot=(500.0, 8), scaling=(4.0, 1.0, 3.0, 96)), 72),
    layer(latent(3, 24, 40, 64, 0.25), 56),
    layer(windowed(4, 4, 16, 16, 0.2, 20, rot=(300.0, 16)), None),
    layer(attention(4, 4, 8, 24, 0.35, rot=(10000.0, 8)), 40),
    layer(windowed(6, 3, 24, 8, 0.25, 37, rot=(100.0, 10)), 88),
    layer(latent(5, 16, 8, 48, 0.3), None),
], width=96, vocab=211, groups=3, scale=3.5, bigram=(53, 17, 5))

# nothing a multiple of 8 where it can be helped; one norm group; no factor on the embedding, no pair rows; a window of one token
AWKWARD = model([
    layer(windowed(3, 1, 12, 20, 0.3, 5, rot=(50.0, 4)), 36),
    layer(latent(5, 10, 7, 33, 0.3), 52),
    layer(attention(3, 3, 12, 20, 0.4, rot=(300.0, 6), scaling=(2.0, 0.5, 0.5, 32)), 20),
    layer(windowed(2, 2, 20, 20, 0.3, 1), 44),
    layer(attention(2, 1, 20, 20, 0.22), None),
], width=100, vocab=97, eps=2e-5)

# heads of 64 and 128 (the split-key decode kernel, the flash and the tcgen05 kernels), one key head for eight query
# heads, windows around a page and two key blocks, a latent of two times 64, latents that are expanded for prompts of
# many rows, the whole head turned
WIDE = model([
    layer(windowed(8, 2, 64, 64, 0.1, 65, rot=(1000.0, 64)), 64),
    layer(attention(8, 1, 128, 128, 0.05, rot=(250.0, 128), scaling=(8.0, 2.0, 16.0, 128)), 40),
    layer(latent(12, 32, 48, 128, 0.15), 64),
    layer(windowed(4, 1, 128, 128, 0.07, 130, rot=(20000.0, 32)), 48),
    layer(attention(8, 2, 64, 64, 0.06, rot=(1000.0, 32)), 64),
    layer(latent(3, 128, 128, 64, 0.1), 40),
    layer(latent(2, 64, 64, 96, 0.15), None),
], width=128, vocab=131, groups=8, scale=0.5, bigram=(1009, 3, 1))

CONFIGS = {"mixed": (MIXED, 71), "awkward": (AWKWARD, 72), "wide": (WIDE, 73)}

# factors that take the random weights (standard deviation 0.02) out of their nearly linear range
LIVELY = {".mix.q": 6.0, ".mix.k": 6.0, ".mix.v": 5.0, ".mix.dkv": 4.0, ".mix.uk": 6.0, ".mix.uv": 4.0, ".mix.g": 10.0,
          ".mix.pb": 60.0, ".up": 6.0, ".down": 2.0, "embed": 4.0, "bigram": 4.0}
MILD = dict(LIVELY, **{".mix.q": 3.0, ".mix.k": 3.0, ".mix.v": 3.0, ".up": 4.0})
SCALES = {"wide": MILD}


def lively_tensors(cfg, seed):
    """Norms on q and k that vary over the projection, latent and stream norms that vary over the row."""
    g = torch.Generator().manual_seed(seed)
    out = {"final.norm": torch.rand(cfg["width"], generator=g) * 1.2 + 0.4}
    for i, L in enumerate(cfg["layers"]):
        m = L["mixer"]
        out[f"l{i}.norm1"] = torch.rand(cfg["width"], generator=g) * 1.2 + 0.4
        if L["type"] == "attention":
            out[f"l{i}.mix.q.norm"] = torch.rand(m["heads"] * m["dim"], generator=g) * 1.4 + 0.3
            out[f"l{i}.mix.k.norm"] = torch.rand(m["kv_heads"] * m["dim"], generator=g) * 1.4 + 0.3
        elif L["type"] == "latent_attention":
            out[f"l{i}.mix.dkv.norm"] = torch.rand(m["kv_rank"], generator=g) * 1.4 + 0.3
    return out


def write_folder(config, seed, out_dir, replace=None, scale=None):
    """A model folder with the engine's seeded random tensors scaled out of their linear range, the lively
    replacements above and whatever `replace` names on top."""
    new = lively_tensors(config, seed)
    new.update(replace or {})
    return VC.write_folder(config, seed, out_dir, replace=new, scale=LIVELY if scale is None else scale)
