"""Pudizen: its config.json keys, and configuration -> plan of parts.

A decoder-only model whose layers are listed one by one in config.json.  The stream starts as the token's
embedding times a factor, plus a row of a second table looked up by a hash of (previous token, token).  Every
layer has one norm (an RMS norm in groups) whose output the mixer and the feed-forward both read:
``x += mixer(norm1(x)) + ff(norm1(x))``.  Three mixers:

* ``attention``: grouped-query softmax attention with one RMS norm over the whole q and the whole k
  projection, a half-split rotation whose frequencies may be scaled by bands of their wavelength
  (``rot.scaling``), and values that are turned by their position over all their dimensions; each head's
  output is turned back by the query's position.
* ``attention_2``: a sliding window, a rotation in interleaved pairs, and no softmax: a key weighs
  ``sigmoid(score + pb_head)``, not normalised over keys.
* ``latent_attention``: keys and values of every head projected from one normed latent a token, which alone
  is cached; no positions; each head's output times a sigmoid gate.

The feed-forward is dense, ``W_down relu(W_up h)^2``, or absent.  The head is a table of its own.

config.json (every size and constant comes from here or from a tensor's shape)::

    architecture   "Pudizen"
    vocab, width
    norm           {eps, groups?}
    embedding?     {scale?, bigram?: {buckets, mul_prev, mul_cur}}
    layers[i]      {type, mixer, mlp}
      attention mixer         {heads, kv_heads, dim, vdim, scale,
                               rot?: {base, dims, scaling?: {factor, low, high, original}}}
      attention_2 mixer       {heads, kv_heads, dim, vdim, scale, mask: {size}, rot?: {base, dims}}
      latent_attention mixer  {heads, dim, vdim, kv_rank, scale}
      mlp    null, or {kind: "dense", ff}

Tensors: ``embed``, ``bigram`` [buckets + 1, width], ``head``, ``final.norm`` and per layer ``l<i>.norm1``,
``l<i>.mix.*``, ``l<i>.mlp.{up,down}``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import (ConfigError, LayerCall, LayerSpec, ModelPlan, PartSpec, opt_float, req_int)
from ..registry import register_architecture

LAYER_TYPES = ("attention", "attention_2", "latent_attention")
_NAMES = (("norm1", "norm1"), ("mixer", "mix"), ("norm2", "norm2"), ("feed_forward", "mlp"))


def _obj(d: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key!r} must be an object")
    return v


def _float(d: Dict[str, Any], key: str, where: str) -> float:
    if key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key {where}{key!r} is missing")
    try:
        return opt_float(d, key, 0.0)
    except ConfigError as e:
        raise ConfigError(str(e).replace("config.json: ", f"config.json: {where}")) from None


def _int(d: Dict[str, Any], key: str, where: str, least: int = 1) -> int:
    try:
        v = req_int(d, key)
    except ConfigError as e:
        raise ConfigError(str(e).replace("config.json: ", f"config.json: {where}")) from None
    if v < least:
        raise ConfigError(f"config.json: {where}{key!r} must be at least {least}, got {v}")
    return v


@dataclass(frozen=True)
class RotationSizes:
    base: float
    dims: int
    # (factor, low, high, original) of the frequencies' bands, or None for the plain ones
    scaling: Optional[Tuple[float, float, float, float]]


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationSizes]
    window: Optional[int]           # attention_2 only


@dataclass(frozen=True)
class LatentAttentionSizes:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float


@dataclass(frozen=True)
class PudizenLayer:
    type: str
    mixer: Any                      # AttentionSizes | LatentAttentionSizes
    ff: Optional[int]               # width of the dense feed-forward, None without one


def _rotation(m: Dict[str, Any], where: str, dim: int, scaled: bool) -> Optional[RotationSizes]:
    if m.get("rot") is None:
        return None
    rot = _obj(m, "rot", where)
    where += "rot."
    dims, base = _int(rot, "dims", where, least=0), _float(rot, "base", where)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}dims={dims} must be even and at most dim={dim}")
    if base <= 0:
        raise ConfigError(f"config.json: {where}base must be positive")
    scaling = None
    if rot.get("scaling") is not None:
        if not scaled:
            raise ConfigError(f"config.json: {where}scaling is not known for this kind of attention")
        sc = _obj(rot, "scaling", where)
        scaling = tuple(_float(sc, k, where + "scaling.") for k in ("factor", "low", "high", "original"))
        if min(scaling) <= 0 or scaling[2] < scaling[1]:
            raise ConfigError(f"config.json: {where}scaling needs positive numbers and low <= high")
    return RotationSizes(base, dims, scaling)


def _attention(m: Dict[str, Any], where: str, windowed: bool) -> AttentionSizes:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads={heads} is not a multiple of kv_heads={kv}")
    dim, vdim = _int(m, "dim", where), _int(m, "vdim", where)
    window = _int(_obj(m, "mask", where), "size", where + "mask.") if windowed else None
    rot = _rotation(m, where, dim, scaled=not windowed)
    if rot is not None and not windowed and vdim % 2:
        raise ConfigError(f"config.json: {where}vdim={vdim} must be even: values are turned in pairs")
    return AttentionSizes(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=_float(m, "scale", where), rot=rot, window=window)


def _latent(m: Dict[str, Any], where: str) -> LatentAttentionSizes:
    return LatentAttentionSizes(heads=_int(m, "heads", where), dim=_int(m, "dim", where), vdim=_int(m, "vdim", where),
                                kv_rank=_int(m, "kv_rank", where), scale=_float(m, "scale", where))


def _mlp(f: Optional[Dict[str, Any]], where: str) -> Optional[int]:
    if f is None:
        return None
    if not isinstance(f, dict):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    if f.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}kind = {f.get('kind')!r}; known: ['dense']")
    return _int(f, "ff", where)


@dataclass(frozen=True)
class PudizenConfig:
    vocab: int
    width: int
    eps: float
    groups: int
    embedding_scale: float
    bigram: Optional[Tuple[int, int, int]]          # (buckets, mul_prev, mul_cur)
    layers: Tuple[PudizenLayer, ...]

    ARCHITECTURE = "Pudizen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PudizenConfig":
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[PudizenLayer] = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = L.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type = {kind!r}; known: {list(LAYER_TYPES)}")
            m, mw = _obj(L, "mixer", where), where + "mixer."
            mixer = _latent(m, mw) if kind == "latent_attention" else _attention(m, mw, windowed=kind == "attention_2")
            layers.append(PudizenLayer(kind, mixer, _mlp(L.get("mlp"), where + "mlp.")))
        norm = _obj(d, "norm", "")
        eps = _float(norm, "eps", "norm.")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        groups = _int(norm, "groups", "norm.") if norm.get("groups") is not None else 1
        width = _int(d, "width", "")
        if width % groups:
            raise ConfigError(f"config.json: width={width} does not split into norm.groups={groups} equal parts")
        emb = _obj(d, "embedding", "") if d.get("embedding") is not None else {}
        scale = _float(emb, "scale", "embedding.") if emb.get("scale") is not None else 1.0
        bigram = None
        if emb.get("bigram") is not None:
            b, bw = _obj(emb, "bigram", "embedding."), "embedding.bigram."
            bigram = (_int(b, "buckets", bw), _int(b, "mul_prev", bw, least=0), _int(b, "mul_cur", bw, least=0))
        return cls(vocab=_int(d, "vocab", ""), width=width, eps=eps, groups=groups, embedding_scale=scale, bigram=bigram,
                   layers=tuple(layers))


def _position_spec(L: PudizenLayer) -> Optional[PartSpec]:
    m = L.mixer
    if m.rot is None or m.rot.dims == 0:
        return None
    if L.type == "attention_2":
        return PartSpec.make("rotary_interleaved", head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims)
    if m.rot.scaling is None:
        return PartSpec.make("rotary_half_split", head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims, double=True)
    factor, low, high, original = m.rot.scaling
    return PartSpec.make("rotary_half_split_banded", head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims,
                         factor=factor, low=low, high=high, original=original)


def _mixer_spec(cfg: PudizenConfig, L: PudizenLayer) -> PartSpec:
    m = L.mixer
    if L.type == "latent_attention":
        return PartSpec.make("latent_attention", hidden_size=cfg.width, heads=m.heads, dim=m.dim, rot_dim=0,
                             value_dim=m.vdim, kv_rank=m.kv_rank, q_rank=None, scale=m.scale, eps=cfg.eps,
                             position=PartSpec.make("none"), sink=False, output_gate=True, gate_per_head=True)
    common = dict(hidden_size=cfg.width, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                  scale=m.scale, eps=cfg.eps, position=_position_spec(L), bias=False, gate=False)
    if L.type == "attention_2":
        return PartSpec.make("whole_norm_gated_attention", norm=False, window=m.window, weights="sigmoid", **common)
    value_position = None
    if m.rot is not None:
        # values turn with the plain frequencies, whatever the keys' are scaled by
        value_position = PartSpec.make("rotary_half_split", head_dim=m.vdim, theta=m.rot.base, double=True)
    return PartSpec.make("whole_norm_gated_attention", value_position=value_position, **common)


def build_plan(cfg: PudizenConfig) -> ModelPlan:
    norm = PartSpec.make("group_rms_norm", size=cfg.width, eps=cfg.eps, groups=cfg.groups, weight_name="")
    layers = []
    for i, L in enumerate(cfg.layers):
        ff = (PartSpec.make("none") if L.ff is None else
              PartSpec.make("dense_relu2", hidden_size=cfg.width, intermediate_size=L.ff))
        layers.append(LayerSpec("parallel", norm, _mixer_spec(cfg, L), ff, prefix=f"l{i}.", names=_NAMES))
    extras = ()
    if cfg.bigram is not None:
        extras = (PartSpec.make("hashed_pair", hidden_size=cfg.width, buckets=cfg.bigram[0], mul_prev=cfg.bigram[1],
                                mul_cur=cfg.bigram[2], name="bigram"),)
    order = tuple(LayerCall(i, i, True) for i in range(len(layers)))
    return ModelPlan(vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers), order=order, final_norm=norm,
                     tie_word_embeddings=False, embedding_name="embed", final_norm_name="final.norm.", head_name="head",
                     embedding_scale=cfg.embedding_scale, embedding_extras=extras)


register_architecture(PudizenConfig.ARCHITECTURE, PudizenConfig.from_dict, build_plan)
