"""Typed configuration of a Nefelorn decoder, read from its ``config.json``.

The file gives every size and every constant that differs between models of the design, layer by layer::

    {"architecture": "Nefelorn", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": s}, "logit_softcap": c,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "kv_from": j,
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": ...},
                {"type": "attention_2",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"}, "rot": {"base", "dims"}},
                 "mlp": ...}, ...]}

with ``mlp`` null, ``{"kind": "dense", "ff": F}`` or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale"}}``.
``mask.size`` is the length of a run of tokens in an ``attention`` layer and of a sliding window in an ``attention_2`` layer.
``kv_from`` names an earlier layer whose cached keys and values the layer uses.  ``kv_from``, ``mask``, ``keep_first``, ``rot``,
``rot.scaling``, ``router.scale``, ``embedding`` and ``logit_softcap`` may be absent and then mean "none of it" or 1.  Required keys
fail with the key's path, in the manner of the reference's config readers (src/model/LlmConfig.cpp:64-93).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .bigerax_config import _At
from .model_config import ConfigError
from .segorax_config import YarnScaling
from .tupunex_config import _optional_number

ARCHITECTURE = "Nefelorn"
TYPES = ("attention", "attention_2")


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                         # the last tokens a query sees (0: no limit)
    chunk: int = 0                          # the runs of tokens a query cannot look out of (0: none)
    keep: int = 0                           # first tokens that are always seen
    rot_dims: int = 0
    rot_base: float = 1.0
    rot_scaling: Optional[YarnScaling] = None
    kv_from: Optional[int] = None           # the layer whose keys and values this one uses


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int


@dataclass(frozen=True)
class ExpertsFeedForward:
    ff: int
    experts: int
    top: int
    scale: float


@dataclass(frozen=True)
class NefelornLayer:
    type: str
    mixer: AttentionMixer
    mlp: Optional[Union[DenseFeedForward, ExpertsFeedForward]]


@dataclass(frozen=True)
class NefelornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: float                    # 0: logits as they are
    layers: Tuple[NefelornLayer, ...]
    max_positions: int
    eos_token_ids: Tuple[int, ...] = ()


def _mixer(m: _At, kind: str, where: str) -> AttentionMixer:
    heads, kv = m.integer("heads"), m.integer("kv_heads")
    if heads % kv:
        raise ConfigError(f"{where}: '{m._name('heads')}' = {heads} is not a multiple of kv_heads = {kv}")
    dim = m.integer("dim")
    rot = m.maybe("rot")
    dims = rot.integer("dims", 0) if rot is not None else 0
    if dims % 2 or dims > dim:
        raise ConfigError(f"{where}: '{m._name('rot.dims')}' = {dims} must be even and at most dim = {dim}")
    scaling = None
    s = rot.maybe("scaling") if rot is not None and dims else None
    if s is not None:
        scaling = YarnScaling(*(s.number(k) for k in ("factor", "original", "fast", "slow")))
        if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0:
            raise ConfigError(f"{where}: the numbers of '{m._name('rot.scaling')}' must be positive")
    base = rot.number("base") if dims else 1.0
    if dims and (base <= 0 or (scaling is not None and base == 1.0)):
        raise ConfigError(f"{where}: '{m._name('rot.base')}' = {base!r} cannot be a rotation's base")
    mask = m.maybe("mask")
    size = mask.integer("size") if mask is not None else 0
    keep = mask.integer("keep_first", 0) if mask is not None and kind == "attention_2" and mask.obj.get("keep_first") is not None else 0
    return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, vdim=m.integer("vdim"), scale=m.number("scale"),
                          window=size if kind == "attention_2" else 0, chunk=size if kind == "attention" else 0, keep=keep, rot_dims=dims,
                          rot_base=base, rot_scaling=scaling, kv_from=m.integer("kv_from", 0) if m.obj.get("kv_from") is not None else None)


def _feed_forward(f: _At, where: str):
    kind = f.need("kind")
    if kind == "dense":
        return DenseFeedForward(ff=f.integer("ff"))
    if kind != "moe":
        raise ConfigError(f"{where}: '{f._name('kind')}' = {kind!r} is not one of 'dense', 'moe'")
    router = f.child("router")
    experts, top = router.integer("experts"), router.integer("top")
    if top > experts:
        raise ConfigError(f"{where}: '{router._name('top')}' = {top} of {experts} experts")
    return ExpertsFeedForward(ff=f.child("expert").integer("ff"), experts=experts, top=top, scale=_optional_number(router, "scale", 1.0))


def _layer(raw: Any, i: int, where: str) -> NefelornLayer:
    at = _At(raw, f"layers[{i}]", where)
    kind = at.need("type")
    if kind not in TYPES:
        raise ConfigError(f"{where}: layers[{i}].type = {kind!r} is not one of {', '.join(repr(t) for t in TYPES)}")
    mlp = at.maybe("mlp")
    return NefelornLayer(type=kind, mixer=_mixer(at.child("mixer"), kind, where), mlp=_feed_forward(mlp, where) if mlp is not None else None)


def _check_sharing(layers: Tuple[NefelornLayer, ...], where: str) -> None:
    for i, layer in enumerate(layers):
        j = layer.mixer.kv_from
        if j is None:
            continue
        name = f"layers[{i}].mixer.kv_from"
        if j >= i:
            raise ConfigError(f"{where}: '{name}' = {j} does not name an earlier layer")
        other = layers[j].mixer
        if other.kv_from is not None:
            raise ConfigError(f"{where}: '{name}' = {j}, a layer without keys and values of its own")
        mine, theirs = layer.mixer, other
        if (mine.kv_heads, mine.dim, mine.vdim) != (theirs.kv_heads, theirs.dim, theirs.vdim):
            raise ConfigError(f"{where}: '{name}' = {j}, whose keys and values have other sizes")


def parse_nefelorn_config(obj: Dict[str, Any], where: str = "config.json") -> NefelornConfig:
    top = _At(obj, "", where)
    raw_layers = top.need("layers")
    if not isinstance(raw_layers, list) or not raw_layers:
        raise ConfigError(f"{where}: 'layers' must be a non-empty list")
    layers = tuple(_layer(raw, i, where) for i, raw in enumerate(raw_layers))
    _check_sharing(layers, where)
    emb = top.maybe("embedding")
    cap = _optional_number(top, "logit_softcap", 0.0)
    if cap < 0:
        raise ConfigError(f"{where}: 'logit_softcap' must not be negative")
    eos = obj.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, list) else ((eos,) if isinstance(eos, int) else ())
    max_pos = obj.get("max_positions")
    return NefelornConfig(architecture=str(obj.get("architecture", ARCHITECTURE)), vocab=top.integer("vocab"), width=top.integer("width"),
                          norm_eps=top.child("norm").number("eps"),
                          embedding_scale=_optional_number(emb, "scale", 1.0) if emb is not None else 1.0, logit_softcap=cap, layers=layers,
                          max_positions=int(max_pos) if isinstance(max_pos, int) and max_pos > 0 else 1 << 20, eos_token_ids=eos_ids)
