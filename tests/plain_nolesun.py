"""A plain, slow, whole-sequence implementation of the Nolesun design, one function per mechanism.

Written from the design's equations in double precision on the CPU with torch's elementary
operations only; it shares no code with the engine.  `forward(cfg, w, tokens)` runs one request's
tokens at once and returns the logits of every position and the stream after every layer run.

The design: a scaled token embedding x0; layers with a norm before and after each sublayer and a
scale per channel behind the second one; a run of layers that may be repeated, where each pass
starts from a projection of [x; x0] plus a vector of its own; two mixers, each of which is an
attention and a recurrence side by side on one input, their outputs added with fixed factors; a
squared-ReLU feed-forward or routed silu-gated experts; an output table of its own.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64

# (generator, size) or None: what a 16-bit engine would round - projections and what enters them, convolutions - is
# disturbed by that fraction of itself, which shows the rows whose logits hang on a near-cancellation or on a close
# choice of experts
NOISE = None


def rounded(x: torch.Tensor) -> torch.Tensor:
    return x if NOISE is None else x * (1.0 + NOISE[1] * torch.randn(x.shape, generator=NOISE[0], dtype=F64))


def proj(h: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = h @ w.T
    if b is not None:
        y = y + b
    return rounded(y)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight lies around zero."""
    return rounded(rms(x, eps) * (1.0 + w))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


# ---- attention ----------------------------------------------------------------------------------

def turn(x: torch.Tensor, base: float, dims: int, neighbours: bool) -> torch.Tensor:
    """x [T, heads, D]: the first `dims` numbers of every head turned by position * base^(-2 i / dims); pair i is
    (i, i + dims / 2), or (2 i, 2 i + 1) with `neighbours`."""
    half = dims // 2
    if half == 0:
        return x
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    a = (torch.arange(x.shape[0], dtype=F64)[:, None] * f)[:, None, :]
    c, s = torch.cos(a), torch.sin(a)
    out = x.clone()
    u, v = (x[..., 0:dims:2], x[..., 1:dims:2]) if neighbours else (x[..., :half], x[..., half:dims])
    if neighbours:
        out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        out[..., :half], out[..., half:dims] = u * c - v * s, v * c + u * s
    return out


def cap_scores(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if not cap else cap * torch.tanh(s / cap)


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, neighbours: bool, biased: bool,
              gated: bool) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    bias = lambda n: w[p + n + ".b"] if biased else None
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    spin = lambda x: turn(x, float(rot["base"]), int(rot["dims"]), neighbours)
    q = spin(proj(h, w[p + "q"], bias("q")).view(T, H, D))
    k = spin(proj(h, w[p + "k"], bias("k")).view(T, G, D))
    v = proj(h, w[p + "v"], bias("v")).view(T, G, Dv)
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = torch.zeros((T, H, Dv), dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = cap_scores((q[:, hd] @ k[:, g].T) * float(m["scale"]), m.get("softcap"))
        out[:, hd] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g]
    o = out.reshape(T, H * Dv)
    if gated:
        o = o * torch.sigmoid(proj(h, w[p + "g"]))
    return proj(rounded(o), w[p + "o"], bias("o"))


# ---- recurrences --------------------------------------------------------------------------------

def short_conv(u: torch.Tensor, taps: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """u [T, C], taps [C, K] (the last column is the current token's), zeros before the start."""
    T, C = u.shape
    K = taps.shape[1]
    pad = torch.cat([torch.zeros(K - 1, C, dtype=F64), u], dim=0)
    out = torch.zeros(T, C, dtype=F64) if bias is None else bias[None, :].repeat(T, 1)
    for j in range(K):
        out = out + pad[j:j + T] * taps[:, j]
    return out


def state_space(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    """S_t = exp(-exp(A) dt) S_{t-1} + dt B x^T, y_t = S_t^T C + D x_t; gate before the norm in parts."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, u, dt = torch.split(proj(h, w[p + "in"]), [inner, inner + 2 * G * N, H], dim=1)
    u = rounded(silu(short_conv(u, w[p + "conv"], w[p + "conv.b"])))
    x, B, C = u[:, :inner].view(T, H, P), u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    rate = torch.exp(w[p + "A_log"])
    y = torch.zeros((T, H, P), dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        S = torch.zeros((N, P), dtype=F64)
        for t in range(T):
            S = torch.exp(-rate[hd] * dt[t, hd]) * S + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            y[t, hd] = S.T @ C[t, g] + w[p + "D"][hd] * x[t, hd]
    y = y.reshape(T, inner) * silu(z)
    parts = int(m["norm_groups"])
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return proj(rounded(y), w[p + "o"])


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_step(S: torch.Tensor, q, k, v, g, beta) -> Tuple[torch.Tensor, torch.Tensor]:
    """One token of the gated delta rule for one head: decay, write what the state does not know yet, read."""
    S = g * S
    S = S + torch.outer(k, beta * (v - S.T @ k))
    return S, S.T @ q


def delta_rule(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (rounded(silu(short_conv(proj(h, w[p + n]), w[p + n + ".conv"]))) for n in ("q", "k", "v"))
    q, k, v = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D)), v.view(T, H, V)
    beta = torch.sigmoid(proj(h, w[p + "b"]))
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(proj(h, w[p + "a"]) + w[p + "dt_bias"]))
    out = torch.zeros((T, H, V), dtype=F64)
    for hd in range(H):
        S = torch.zeros((D, V), dtype=F64)
        kh = hd // (H // G)
        for t in range(T):
            S, out[t, hd] = delta_step(S, q[t, kh], k[t, kh], v[t, hd], g[t, hd], beta[t, hd])
    o = (rms(out, eps) * w[p + "norm"]).reshape(T, H * V)
    return proj(rounded(o * silu(proj(h, w[p + "g"]))), w[p + "o"])


def mixer(h, w, p: str, L: Dict, eps: float) -> torch.Tensor:
    m = L["mixer"]
    if L["type"] == "parallel":
        left = attention(h, w, p + "left.", m["left"], neighbours=False, biased=False, gated=False)
        right = state_space(h, w, p + "right.", m["right"], eps)
    elif L["type"] == "parallel_2":
        left = attention(h, w, p + "left.", m["left"], neighbours=True, biased=True, gated=True)
        right = delta_rule(h, w, p + "right.", m["right"], eps)
    else:
        raise ValueError(L["type"])
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# ---- feed-forward -------------------------------------------------------------------------------

def relu2_mlp(h, w, p: str) -> torch.Tensor:
    return proj(torch.relu(proj(h, w[p + "up"])) ** 2, w[p + "down"])


def choose(z: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """The `top` largest logits, and the softmax over those alone."""
    best, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(best, dim=-1)


def moe(h, w, p: str, f: Dict, forced: Optional[torch.Tensor] = None, record: Optional[list] = None) -> torch.Tensor:
    """`forced` [T, top]: the experts to use instead of the largest logits' (weighted by the softmax over theirs);
    `record` receives (logits, experts)."""
    z = proj(h, w[p + "router"], w[p + "router.b"])
    idx, wts = choose(z, int(f["router"]["top"]))
    if forced is not None:
        idx, wts = forced, torch.softmax(torch.gather(z, 1, forced), dim=-1)
    if record is not None:
        record.append((z, idx))
    out = torch.zeros_like(h)
    for e in range(int(f["router"]["experts"])):
        rows, j = torch.nonzero(idx == e, as_tuple=True)
        if len(rows) == 0:
            continue
        u = h[rows]
        y = proj(silu(proj(u, w[f"{p}e{e}.gate"])) * proj(u, w[f"{p}e{e}.up"]), w[f"{p}e{e}.down"])
        out.index_add_(0, rows, y * wts[rows, j][:, None])
    return out


# ---- the model ----------------------------------------------------------------------------------

def layer_runs(cfg: Dict) -> List[Tuple[int, Optional[int]]]:
    """(layer, pass) in the order they run; pass is None outside the repeated run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(int(loop["times"])) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def enter_pass(x, x0, w, t: int) -> torch.Tensor:
    return proj(torch.cat([x, x0], dim=1), w["loop.in"]) + w["loop.step"][t]


def forward(cfg: Dict, weights: Dict[str, torch.Tensor], tokens: List[int], forced: Optional[list] = None,
            record: Optional[list] = None):
    """-> (logits [T, vocab], streams [layer runs, T, width]) in double precision.  `forced`: the experts [T, top] of
    every routed run, in order; `record` receives each routed run's (logits, experts)."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = x0 = w["embed"][torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    streams, routed = [], 0
    for i, t in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if t is not None and i == int(cfg["loop"]["start"]):
            x = enter_pass(x, x0, w, t)
        y = mixer(norm(x, w[p + "norm1"], eps), w, p + "mix.", L, eps)
        x = x + norm(y, w[p + "norm1b"], eps) * w[p + "ls1"]
        f = L.get("mlp")
        if f:
            h = norm(x, w[p + "norm2"], eps)
            if f["kind"] == "dense":
                y = relu2_mlp(h, w, p + "mlp.")
            else:
                y = moe(h, w, p + "mlp.", f, None if forced is None else forced[routed], record)
                routed += 1
            x = x + norm(y, w[p + "norm2b"], eps) * w[p + "ls2"]
        streams.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T, torch.stack(streams)
