"""Nolesun: its config.json keys, and configuration -> plan of parts.

A decoder-only model whose layers are listed one by one in config.json.  The stream starts as the token's
embedding times a factor.  Every layer has a norm (RMS, stored weight around zero) before and after each
sublayer and scales the second one's result per channel: ``x += ls1 * norm1b(mixer(norm1(x)))``, then
``x += ls2 * norm2b(ff(norm2(x)))``.  A run of layers may be repeated with the same weights (``loop``): each
pass has cache and state of its own and begins by replacing the stream, ``x <- W_in [x; x0] + step[pass]``,
x0 being what the stream started as.  Two mixers, each of which is two mixers side by side on one input whose
outputs are added with fixed factors:

* ``parallel``: grouped-query softmax attention with a half-split rotation, beside a state-space mixer in the
  dual (Mamba-2) form;
* ``parallel_2``: grouped-query softmax attention with biases, a rotation in interleaved pairs, capped scores
  and an elementwise output gate, beside a gated delta rule.

The feed-forward is dense, ``W_down relu(W_up h)^2``, or a mixture of silu-gated experts: the router's logits
have a bias, the largest are chosen, and the weights are the softmax over the chosen ones.  Either may be
absent.  The head is a table of its own.

config.json (every size and constant comes from here or from a tensor's shape)::

    architecture   "Nolesun"
    vocab, width
    norm           {eps}
    embedding?     {scale?}
    loop?          {start, stop, times}: layers start .. stop-1 run `times` times in a row
    layers[i]      {type, mixer: {left, right, left_scale, right_scale}, mlp}
      left                    {heads, kv_heads, dim, vdim, scale, rot?: {base, dims}}, parallel_2: softcap? too
      right of parallel       {heads, vdim, state, groups, conv, norm_groups}
      right of parallel_2     {heads, kv_heads, dim, vdim, conv}
      mlp    null, {kind: "dense", ff}, or {kind: "moe", expert: {ff}, router: {experts, top}}

Tensors: ``embed``, ``head``, ``final.norm``, ``loop.in`` [width, 2 width], ``loop.step`` [times, width], and per
layer ``l<i>.norm1``, ``.norm1b``, ``.norm2``, ``.norm2b``, ``.ls1``, ``.ls2``, ``l<i>.mix.left.*``,
``l<i>.mix.right.*``, ``l<i>.mlp.*``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import (ConfigError, LayerCall, LayerSpec, ModelPlan, PartSpec, opt_float, req_int)
from ..registry import register_architecture

LAYER_TYPES = ("parallel", "parallel_2")
_NAMES = (("norm1", "norm1"), ("norm1b", "norm1b"), ("mixer", "mix"), ("norm2", "norm2"), ("norm2b", "norm2b"),
          ("feed_forward", "mlp"), ("scale1", "ls1"), ("scale2", "ls2"))
LOOP_VECTORS, LOOP_MATRIX = "loop.step", "loop.in"


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
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Tuple[float, int]]        # (base, dims); None: nothing is turned
    softcap: Optional[float]


@dataclass(frozen=True)
class StateSpaceSizes:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class DeltaRuleSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MlpSizes:
    kind: str                               # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class NolesunLayer:
    type: str
    left: AttentionSizes
    right: Any                              # StateSpaceSizes | DeltaRuleSizes
    left_scale: float
    right_scale: float
    mlp: Optional[MlpSizes]


def _heads(m: Dict[str, Any], where: str) -> Tuple[int, int]:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads={heads} is not a multiple of kv_heads={kv}")
    return heads, kv


def _attention(m: Dict[str, Any], where: str, capped: bool) -> AttentionSizes:
    heads, kv = _heads(m, where)
    dim = _int(m, "dim", where)
    rot = None
    if m.get("rot") is not None:
        r, rw = _obj(m, "rot", where), where + "rot."
        dims, base = _int(r, "dims", rw, least=0), _float(r, "base", rw)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {rw}dims={dims} must be even and at most dim={dim}")
        if base <= 0:
            raise ConfigError(f"config.json: {rw}base must be positive")
        rot = (base, dims) if dims else None
    softcap = None
    if m.get("softcap") is not None:
        if not capped:
            raise ConfigError(f"config.json: {where}softcap is not known for this kind of attention")
        softcap = _float(m, "softcap", where)
        if softcap <= 0:
            raise ConfigError(f"config.json: {where}softcap must be positive")
    scale = _float(m, "scale", where)
    if scale <= 0:
        raise ConfigError(f"config.json: {where}scale must be positive")
    return AttentionSizes(heads, kv, dim, _int(m, "vdim", where), scale, rot, softcap)


def _state_space(m: Dict[str, Any], where: str) -> StateSpaceSizes:
    s = StateSpaceSizes(heads=_int(m, "heads", where), vdim=_int(m, "vdim", where), state=_int(m, "state", where),
                        groups=_int(m, "groups", where), conv=_int(m, "conv", where), norm_groups=_int(m, "norm_groups", where))
    if s.heads % s.groups:
        raise ConfigError(f"config.json: {where}heads={s.heads} is not a multiple of groups={s.groups}")
    if (s.heads * s.vdim) % s.norm_groups:
        raise ConfigError(f"config.json: {where}heads * vdim does not split into norm_groups={s.norm_groups}")
    return s


def _delta_rule(m: Dict[str, Any], where: str) -> DeltaRuleSizes:
    heads, kv = _heads(m, where)
    return DeltaRuleSizes(heads, kv, _int(m, "dim", where), _int(m, "vdim", where), _int(m, "conv", where))


def _mlp(f: Optional[Dict[str, Any]], where: str) -> Optional[MlpSizes]:
    if f is None:
        return None
    if not isinstance(f, dict):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    kind = f.get("kind")
    if kind == "dense":
        return MlpSizes("dense", _int(f, "ff", where))
    if kind == "moe":
        ro = _obj(f, "router", where)
        m = MlpSizes("moe", _int(_obj(f, "expert", where), "ff", where + "expert."), _int(ro, "experts", where + "router."),
                     _int(ro, "top", where + "router."))
        if m.top > m.experts:
            raise ConfigError(f"config.json: {where}router.top={m.top} exceeds experts={m.experts}")
        return m
    raise ConfigError(f"config.json: {where}kind = {kind!r}; known: ['dense', 'moe']")


@dataclass(frozen=True)
class NolesunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[NolesunLayer, ...]
    loop: Optional[Tuple[int, int, int]]    # (start, stop, times); None: every layer runs once

    ARCHITECTURE = "Nolesun"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NolesunConfig":
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[NolesunLayer] = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = L.get("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type = {kind!r}; known: {list(LAYER_TYPES)}")
            m, mw = _obj(L, "mixer", where), where + "mixer."
            right = _state_space if kind == "parallel" else _delta_rule
            layers.append(NolesunLayer(
                kind, _attention(_obj(m, "left", mw), mw + "left.", capped=kind == "parallel_2"),
                right(_obj(m, "right", mw), mw + "right."), _float(m, "left_scale", mw), _float(m, "right_scale", mw),
                _mlp(L.get("mlp"), where + "mlp.")))
        loop = None
        if d.get("loop") is not None:
            lp = _obj(d, "loop", "")
            loop = (_int(lp, "start", "loop.", least=0), _int(lp, "stop", "loop.", least=0), _int(lp, "times", "loop."))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop {loop[0]}..{loop[1]} is no run of the {len(layers)} layers")
        eps = _float(_obj(d, "norm", ""), "eps", "norm.")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        emb = _obj(d, "embedding", "") if d.get("embedding") is not None else {}
        scale = _float(emb, "scale", "embedding.") if emb.get("scale") is not None else 1.0
        return cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), eps=eps, embedding_scale=scale, layers=tuple(layers),
                   loop=loop)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) in the order they run; pass is None outside the loop."""
        n = len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (n, n, 0)
        return ([(i, None) for i in range(start)] + [(i, t) for t in range(times) for i in range(start, stop)]
                + [(i, None) for i in range(stop, n)])


def _mixer_spec(cfg: NolesunConfig, L: NolesunLayer) -> PartSpec:
    a, second = L.left, L.type == "parallel_2"
    position = None
    if a.rot is not None:
        base, dims = a.rot
        position = (PartSpec.make("rotary_interleaved", head_dim=a.dim, theta=base, rotary_dim=dims) if second else
                    PartSpec.make("rotary_half_split", head_dim=a.dim, theta=base, rotary_dim=dims, double=True))
    left = PartSpec.make("whole_norm_gated_attention", hidden_size=cfg.width, heads=a.heads, kv_heads=a.kv_heads,
                         head_dim=a.dim, value_dim=a.vdim, scale=a.scale, eps=cfg.eps, position=position, norm=False,
                         bias=second, gate=second, out_bias=second, softcap=a.softcap)
    r = L.right
    if second:
        right = PartSpec.make("gated_delta_rule", hidden_size=cfg.width, heads=r.heads, kv_heads=r.kv_heads, dim=r.dim,
                              value_dim=r.vdim, conv_taps=r.conv, eps=cfg.eps)
    else:
        right = PartSpec.make("state_space_dual", hidden_size=cfg.width, heads=r.heads, head_dim=r.vdim, state_size=r.state,
                              groups=r.groups, conv_taps=r.conv, norm_groups=r.norm_groups, eps=cfg.eps)
    return PartSpec.make("parallel_scaled", branches=(("left", left), ("right", right)), scales=(L.left_scale, L.right_scale))


_MOE_NAMES = (("router", "router"), ("router_bias", "router.b"), ("gate", "e{e}.gate"), ("up", "e{e}.up"), ("down", "e{e}.down"))


def _ff_spec(cfg: NolesunConfig, f: Optional[MlpSizes]) -> PartSpec:
    if f is None:
        return PartSpec.make("none")
    if f.kind == "dense":
        return PartSpec.make("dense_relu2", hidden_size=cfg.width, intermediate_size=f.ff)
    # the softmax over the chosen logits is the softmax over all of them, divided by the chosen ones' sum
    return PartSpec.make("sparse_moe_swiglu", hidden_size=cfg.width, num_experts=f.experts, top_k=f.top, norm_topk_prob=True,
                         moe_intermediate_size=f.ff, shared_intermediate_size=0, tensor_names=_MOE_NAMES, router_bias=True)


def build_plan(cfg: NolesunConfig) -> ModelPlan:
    norm = PartSpec.make("rms_norm", size=cfg.width, eps=cfg.eps, weight_name="", one_plus=True)
    layers = tuple(LayerSpec("norms_around_scaled", norm, _mixer_spec(cfg, L), _ff_spec(cfg, L.mlp), prefix=f"l{i}.", names=_NAMES)
                   for i, L in enumerate(cfg.layers))
    # every run of a layer has cache and state of its own: slot = the run's number
    order = []
    for slot, (i, t) in enumerate(cfg.runs()):
        enters = t is not None and i == cfg.loop[0]
        order.append(LayerCall(i, slot, True, state=slot, add_vector=(LOOP_VECTORS, t) if enters else None,
                               project=LOOP_MATRIX if enters else None))
    return ModelPlan(vocab_size=cfg.vocab, hidden_size=cfg.width, layers=layers, order=tuple(order), final_norm=norm,
                     tie_word_embeddings=False, embedding_name="embed", final_norm_name="final.norm.", head_name="head",
                     embedding_scale=cfg.embedding_scale,
                     stream_vectors=((LOOP_VECTORS, cfg.loop[2]),) if cfg.loop else (),
                     stream_projections=(LOOP_MATRIX,) if cfg.loop else ())


register_architecture(NolesunConfig.ARCHITECTURE, NolesunConfig.from_dict, build_plan)
