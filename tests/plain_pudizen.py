"""A plain, slow, whole-sequence implementation of the Pudizen design, one function per mechanism.

Written from the design's equations in double precision on the CPU with torch's elementary
operations only; it shares no code with the engine.  `forward(cfg, w, tokens)` runs one request's
tokens at once and returns the logits of every position and the stream after every layer.

The design: a scaled token embedding plus a row looked up by a hash of (previous token, token); layers
whose mixer and feed-forward read one norm's output side by side (`x += mixer(h) + ff(h)`, an RMS norm
in groups); three mixers - softmax attention with one norm over the whole q and the whole k projection
and values that are turned by their position and turned back in the output; sigmoid attention without
normalisation in a sliding window, rotation in interleaved pairs; attention over a latent without
positions and a gate number a head - and a squared-ReLU feed-forward; an output table of its own.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64

# (generator, size) or None: every projection's output is disturbed by that fraction of itself, which shows the
# rows whose logits hang on a near-cancellation
NOISE = None


def proj(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    y = h @ w.T
    if NOISE is not None:
        y = y * (1.0 + NOISE[1] * torch.randn(y.shape, generator=NOISE[0], dtype=F64))
    return y


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_rms(x: torch.Tensor, groups: int, w: torch.Tensor, eps: float) -> torch.Tensor:
    """Each of `groups` equal consecutive parts over its own root mean square, the whole times w."""
    parts = x.view(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * w


def embed(cfg: Dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    e = cfg.get("embedding") or {}
    x = w["embed"][torch.tensor(tokens)] * float(e.get("scale", 1.0))
    b = e.get("bigram")
    if b:
        rows = [int(b["buckets"])]
        for prev, cur in zip(tokens, tokens[1:]):
            rows.append((prev * int(b["mul_prev"]) + cur * int(b["mul_cur"])) % int(b["buckets"]))
        x = x + w["bigram"][torch.tensor(rows)]
    return x


def frequencies(rot: Dict) -> torch.Tensor:
    """Frequency of pair i for i < dims / 2, with long waves stretched if `scaling` says so."""
    dims, base = int(rot["dims"]), float(rot["base"])
    sc = rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wave = 2.0 * math.pi / f
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            if wave < original / high:
                pass
            elif wave > original / low:
                f = f / factor
            else:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def turn(x: torch.Tensor, angles: torch.Tensor, dims: int, interleaved: bool) -> torch.Tensor:
    """x [T, heads, n], angles [T, dims / 2]: the first `dims` of each head turned pair by pair."""
    y = x.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        c, s = torch.cos(angles[:, i])[:, None], torch.sin(angles[:, i])[:, None]
        y[..., a] = x[..., a] * c - x[..., b] * s
        y[..., b] = x[..., b] * c + x[..., a] * s
    return y


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: Optional[Dict], interleaved: bool) -> torch.Tensor:
    if not rot or not int(rot["dims"]):
        return x
    return turn(x, positions.to(F64)[:, None] * frequencies(rot)[None, :], int(rot["dims"]), interleaved)


def visible(T: int, window: int = 0) -> torch.Tensor:
    """[i, j]: position i sees j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < window) if window else j <= i


def attention_mixer(h, w, p: str, m: Dict, eps: float, positions: torch.Tensor) -> torch.Tensor:
    """Softmax attention, whole-projection norms, half-split rotation, values turned and turned back."""
    T = h.shape[0]
    H, G, D, Dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    rot = m.get("rot")
    q = rms(proj(h, w[p + "q"]), eps) * w[p + "q.norm"]
    k = rms(proj(h, w[p + "k"]), eps) * w[p + "k.norm"]
    q = rotate(q.view(T, H, D), positions, rot, False)
    k = rotate(k.view(T, G, D), positions, rot, False)
    v = proj(h, w[p + "v"]).view(T, G, Dv)
    if rot:
        f = torch.tensor([float(rot["base"]) ** (-2.0 * i / Dv) for i in range(Dv // 2)], dtype=F64)
        angles = positions.to(F64)[:, None] * f[None, :]
        v = turn(v, angles, Dv, False)
    out = torch.zeros((T, H, Dv), dtype=F64)
    see = visible(T)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(m["scale"])
        out[:, hd] = torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, g]
    if rot:
        out = turn(out, -angles, Dv, False)
    return proj(out.reshape(T, H * Dv), w[p + "o"])


def sigmoid_mixer(h, w, p: str, m: Dict, positions: torch.Tensor) -> torch.Tensor:
    """Sliding window, interleaved rotation, weights sigmoid(score + a number a head), not normalised."""
    T = h.shape[0]
    H, G, D, Dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q = rotate(proj(h, w[p + "q"]).view(T, H, D), positions, m.get("rot"), True)
    k = rotate(proj(h, w[p + "k"]).view(T, G, D), positions, m.get("rot"), True)
    v = proj(h, w[p + "v"]).view(T, G, Dv)
    see = visible(T, int(m["mask"]["size"])).to(F64)
    out = torch.zeros((T, H, Dv), dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(m["scale"]) + w[p + "pb"][hd]
        out[:, hd] = (torch.sigmoid(s) * see) @ v[:, g]
    return proj(out.reshape(T, H * Dv), w[p + "o"])


def latent_mixer(h, w, p: str, m: Dict, eps: float) -> torch.Tensor:
    """Keys and values of every head projected from one normed latent a token; no positions; a gate a head."""
    T = h.shape[0]
    H, D, Dv = (int(m[k]) for k in ("heads", "dim", "vdim"))
    q = proj(h, w[p + "q"]).view(T, H, D)
    c = rms(proj(h, w[p + "dkv"]), eps) * w[p + "dkv.norm"]
    k = proj(c, w[p + "uk"]).view(T, H, D)
    v = proj(c, w[p + "uv"]).view(T, H, Dv)
    gate = torch.sigmoid(proj(h, w[p + "g"]))
    see = visible(T)
    out = torch.zeros((T, H, Dv), dtype=F64)
    for hd in range(H):
        s = (q[:, hd] @ k[:, hd].T) * float(m["scale"])
        out[:, hd] = (torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, hd]) * gate[:, hd:hd + 1]
    return proj(out.reshape(T, H * Dv), w[p + "o"])


def relu2_mlp(h, w, p: str) -> torch.Tensor:
    return proj(torch.relu(proj(h, w[p + "up"])) ** 2, w[p + "down"])


def forward(cfg: Dict, weights: Dict[str, torch.Tensor], tokens: List[int]):
    """-> (logits [T, vocab], streams [layers, T, width]) in double precision."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups", 1))
    positions = torch.arange(len(tokens))
    x = embed(cfg, w, tokens)
    streams = []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = group_rms(x, groups, w[p + "norm1"], eps)
        if L["type"] == "attention":
            y = attention_mixer(h, w, p + "mix.", m, eps, positions)
        elif L["type"] == "attention_2":
            y = sigmoid_mixer(h, w, p + "mix.", m, positions)
        elif L["type"] == "latent_attention":
            y = latent_mixer(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + relu2_mlp(h, w, p + "mlp.")
        x = x + y
        streams.append(x.clone())
    return group_rms(x, groups, w["final.norm"], eps) @ w["head"].T, torch.stack(streams)
