"""Typed configuration of a Segorax decoder, read from its ``config.json``.

The file gives every size and every constant that differs between models of the design, layer by layer::

    {"architecture": "Segorax", "vocab": V, "width": D, "norm": {"eps": e}, "residual_mult": m, "logit_scale": s,
     "embedding": {"scale": s},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}}, "mlp": ...},
                {"type": "latent_attention_2",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "scale",
                           "rot": {"base", "dims", "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": ...}, ...]}

with ``mlp`` null, ``{"kind": "dense", "ff": F}`` or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups":
{"count", "keep"}}, "shared": {"ff"}}``.  ``groups``, ``shared``, ``rot``, ``rot.scaling``, ``embedding``, ``residual_mult`` and
``logit_scale`` may be absent and then mean "none of it" or 1.  Required keys fail with the key's path, in the manner of the
reference's config readers (src/model/LlmConfig.cpp:64-93).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .bigerax_config import _At
from .model_config import ConfigError
from .tupunex_config import _optional_number

ARCHITECTURE = "Segorax"


@dataclass(frozen=True)
class YarnScaling:
    """Frequencies of a rotation stretched from ``original`` positions by ``factor``."""
    factor: float
    original: float
    fast: float
    slow: float

    def as_dict(self) -> Dict[str, float]:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class LatentMixer:
    """Keys and values of every head made from one cached latent vector per token, plus one rotated key part."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    q_rank: int = 0                         # 0: queries straight from the layer's input
    sink: bool = False
    rot_dims: int = 0
    rot_base: float = 1.0
    rot_scaling: Optional[YarnScaling] = None


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int


@dataclass(frozen=True)
class ExpertsFeedForward:
    ff: int
    experts: int
    top: int
    groups: int
    keep: int
    shared_ff: Optional[int]


@dataclass(frozen=True)
class SegoraxLayer:
    type: str                               # "latent_attention" or "latent_attention_2"
    mixer: LatentMixer
    mlp: Optional[Union[DenseFeedForward, ExpertsFeedForward]]


@dataclass(frozen=True)
class SegoraxConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[SegoraxLayer, ...]
    max_positions: int
    eos_token_ids: Tuple[int, ...] = ()


def _mixer(m: _At, low_rank_q: bool, where: str) -> LatentMixer:
    rot_dim = m.integer("rot_dim", 0)
    rot = m.maybe("rot")
    dims = rot.integer("dims", 0) if rot is not None else 0
    if dims % 2 or dims > rot_dim:
        raise ConfigError(f"{where}: '{m._name('rot.dims')}' = {dims} must be even and at most rot_dim = {rot_dim}")
    scaling = None
    s = rot.maybe("scaling") if rot is not None and dims else None
    if s is not None:
        scaling = YarnScaling(*(s.number(k) for k in ("factor", "original", "fast", "slow")))
        if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0:
            raise ConfigError(f"{where}: the numbers of '{m._name('rot.scaling')}' must be positive")
    base = rot.number("base") if dims else 1.0
    if dims and (base <= 0 or (scaling is not None and base == 1.0)):
        raise ConfigError(f"{where}: '{m._name('rot.base')}' = {base!r} cannot be a rotation's base")
    scale = m.number("scale")
    return LatentMixer(heads=m.integer("heads"), dim=m.integer("dim"), rot_dim=rot_dim, vdim=m.integer("vdim"), kv_rank=m.integer("kv_rank"),
                       scale=scale, q_rank=m.integer("q_rank") if low_rank_q else 0, sink=low_rank_q, rot_dims=dims, rot_base=base,
                       rot_scaling=scaling)


def _feed_forward(f: _At, where: str):
    kind = f.need("kind")
    if kind == "dense":
        return DenseFeedForward(ff=f.integer("ff"))
    if kind != "moe":
        raise ConfigError(f"{where}: '{f._name('kind')}' = {kind!r} is not one of 'dense', 'moe'")
    router = f.child("router")
    experts, top = router.integer("experts"), router.integer("top")
    groups = router.maybe("groups")
    count, keep = (groups.integer("count"), groups.integer("keep")) if groups is not None else (1, 1)
    if experts % count or keep > count:
        raise ConfigError(f"{where}: '{router._name('groups')}': {experts} experts do not form {count} equal groups of which {keep} can be kept")
    if top > keep * (experts // count):
        raise ConfigError(f"{where}: '{router._name('top')}' = {top} experts cannot be chosen from {keep} groups of {experts // count}")
    shared = f.maybe("shared")
    return ExpertsFeedForward(ff=f.child("expert").integer("ff"), experts=experts, top=top, groups=count, keep=keep,
                              shared_ff=shared.integer("ff") if shared is not None else None)


def _layer(raw: Any, i: int, where: str) -> SegoraxLayer:
    at = _At(raw, f"layers[{i}]", where)
    kind = at.need("type")
    if kind not in ("latent_attention", "latent_attention_2"):
        raise ConfigError(f"{where}: layers[{i}].type = {kind!r} is not one of 'latent_attention', 'latent_attention_2'")
    mlp = at.maybe("mlp")
    return SegoraxLayer(type=kind, mixer=_mixer(at.child("mixer"), kind == "latent_attention", where),
                        mlp=_feed_forward(mlp, where) if mlp is not None else None)


def parse_segorax_config(obj: Dict[str, Any], where: str = "config.json") -> SegoraxConfig:
    top = _At(obj, "", where)
    raw_layers = top.need("layers")
    if not isinstance(raw_layers, list) or not raw_layers:
        raise ConfigError(f"{where}: 'layers' must be a non-empty list")
    emb = top.maybe("embedding")
    eos = obj.get("eos_token_id")
    eos_ids = tuple(eos) if isinstance(eos, list) else ((eos,) if isinstance(eos, int) else ())
    max_pos = obj.get("max_positions")
    return SegoraxConfig(architecture=str(obj.get("architecture", ARCHITECTURE)), vocab=top.integer("vocab"), width=top.integer("width"),
                         norm_eps=top.child("norm").number("eps"), residual_mult=_optional_number(top, "residual_mult", 1.0),
                         embedding_scale=_optional_number(emb, "scale", 1.0) if emb is not None else 1.0,
                         logit_scale=_optional_number(top, "logit_scale", 1.0),
                         layers=tuple(_layer(raw, i, where) for i, raw in enumerate(raw_layers)),
                         max_positions=int(max_pos) if isinstance(max_pos, int) and max_pos > 0 else 1 << 20, eos_token_ids=eos_ids)
