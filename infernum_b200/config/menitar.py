"""Typed configuration of the Menitar decoder (``"architecture": "Menitar"``).

config.json of this design is nested:

    architecture, vocab, width, logit_scale, norm.eps, embedding.scale
    loop                                null or {start, stop, times}
    layers[i].type                      "attention"
    layers[i].mixer                     {heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {dims, base}}
    layers[i].mlp                       null or {kind: "dense", ff, limit}

Every size and constant is read here and nowhere else.  Keys that a model leaves
out mean what their absence says: no ``loop`` - every layer runs once; no
``mask`` - queries see all earlier keys; no ``rot`` (or ``dims`` 0) - no rotation;
no ``limit`` - nothing is clamped; ``kv_heads`` and ``vdim`` default to ``heads`` and
``dim``, ``scale`` to the inverse root of ``dim``, ``embedding.scale`` and
``logit_scale`` to 1.  One key is not the design's and optional: ``max_position``
bounds the scheduler's default sequence length.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError
from .base import take_float, take_int


def _section(d: Mapping[str, Any], key: str, where: str, optional: bool = False) -> Optional[Mapping[str, Any]]:
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


@dataclass(frozen=True)
class MenitarAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int  # positions in a run that see one another; 0: no such bound
    rot_dims: int  # 0: no rotation
    rot_base: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "MenitarAttentionConfig":
        heads, dim = take_int(d, "heads"), take_int(d, "dim")
        mask = _section(d, "mask", where, optional=True)
        rot = _section(d, "rot", where, optional=True)
        cfg = cls(heads=heads, kv_heads=take_int(d, "kv_heads", default=heads), dim=dim,
                  vdim=take_int(d, "vdim", default=dim), scale=take_float(d, "scale", default=dim ** -0.5),
                  chunk=take_int(mask, "size", default=0) if mask is not None else 0,
                  rot_dims=take_int(rot, "dims", default=dim, minimum=0) if rot is not None else 0,
                  rot_base=take_float(rot, "base", default=10000.0) if rot is not None else 10000.0)
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"config.json: {where}{cfg.heads} heads are not a multiple of {cfg.kv_heads} kv_heads")
        if cfg.rot_dims % 2 or cfg.rot_dims > dim:
            raise ConfigError(f"config.json: {where}rot.dims {cfg.rot_dims} must be even and at most {dim}")
        if cfg.rot_dims and cfg.rot_base <= 0:
            raise ConfigError(f"config.json: {where}rot.base must be positive")
        return cfg


@dataclass(frozen=True)
class MenitarMlpConfig:
    ff: int
    limit: Optional[float]  # None: nothing is clamped

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "MenitarMlpConfig":
        kind = d.get("kind", "dense")
        if kind != "dense":
            raise ConfigError(f"config.json: {where}kind {kind!r} is not supported (dense)")
        return cls(ff=take_int(d, "ff"), limit=take_float(d, "limit", default=None))


@dataclass(frozen=True)
class MenitarLayerConfig:
    type: str
    mixer: MenitarAttentionConfig
    mlp: Optional[MenitarMlpConfig]


@dataclass(frozen=True)
class MenitarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    loop: Optional[Tuple[int, int, int]]  # (start, stop, times)
    layers: Tuple[MenitarLayerConfig, ...]
    max_position: int = 32768
    architecture: str = "Menitar"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MenitarConfig":
        if d.get("architecture") != "Menitar":
            raise ConfigError(f"MenitarConfig cannot read architecture {d.get('architecture')!r}")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, ld in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(ld, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = ld.get("type")
            if kind != "attention":
                raise ConfigError(f"config.json: {where}type {kind!r} is not supported (attention)")
            mixer = MenitarAttentionConfig.from_dict(_section(ld, "mixer", where), where + "mixer.")
            mlp_d = _section(ld, "mlp", where, optional=True)
            layers.append(MenitarLayerConfig(kind, mixer,
                                             MenitarMlpConfig.from_dict(mlp_d, where + "mlp.") if mlp_d is not None else None))
        loop_d = _section(d, "loop", "", optional=True)
        loop = None
        if loop_d is not None:
            loop = (take_int(loop_d, "start", minimum=0), take_int(loop_d, "stop", minimum=0),
                    take_int(loop_d, "times", default=1))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"config.json: loop {loop[0]}..{loop[1]} does not name a run of the {len(layers)} layers")
        emb = _section(d, "embedding", "", optional=True)
        return cls(vocab=take_int(d, "vocab"), width=take_int(d, "width"), norm_eps=take_float(_section(d, "norm", ""), "eps"),
                   embedding_scale=take_float(emb, "scale", default=1.0) if emb is not None else 1.0,
                   logit_scale=take_float(d, "logit_scale", default=1.0), loop=loop, layers=tuple(layers),
                   max_position=take_int(d, "max_position", default=32768))
