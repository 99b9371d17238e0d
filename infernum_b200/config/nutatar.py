"""Typed configuration of the Nutatar decoder (``"architecture": "Nutatar"``).

config.json of this design is nested:

    architecture, vocab, width, norm.eps, embedding.scale
    layers[i].type                      "attention", "gla" or "latent_attention"
    layers[i].mixer                     attention:        {heads, kv_heads, dim, vdim, scale, mask: {size},
                                                           rot: {dims, base}}
                                        gla:              {heads, dim, vdim, tau}
                                        latent_attention: {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, kv_from,
                                                           rot: {dims, base, scaling: {factor, original, fast, slow}}}
    layers[i].mlp                       null, {kind: "dense", ff} or
                                        {kind: "moe", expert: {ff, limit}, shared: {ff, limit},
                                         router: {experts, top, groups: {count, keep}}}

Every size and constant is read here and nowhere else.  Keys that a model leaves
out mean what their absence says: no ``mask`` - every earlier token is visible; no
``rot`` (or ``dims`` 0) - no rotation; no ``scaling`` - plain frequencies; no ``kv_from``
- the layer keeps a cache of its own; no ``groups`` - every expert can be chosen; no
``limit`` - nothing is clamped; no ``shared`` - no expert that all tokens use;
``kv_heads`` and ``vdim`` default to ``heads`` and ``dim``, ``scale`` to the inverse root
of the query's size, ``tau`` and ``embedding.scale`` to 1.  One key is not the design's
and optional: ``max_position`` bounds the scheduler's default sequence length.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError
from .base import take_float, take_int
from .vodatar import PairRotation


def _section(d: Mapping[str, Any], key: str, where: str, optional: bool = False) -> Optional[Mapping[str, Any]]:
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


@dataclass(frozen=True)
class KeyValueAttentionConfig:
    """Attention whose values are its keys."""

    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int  # 0: every earlier token is visible
    rot_dims: int  # 0: no rotation
    rot_base: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "KeyValueAttentionConfig":
        heads, dim = take_int(d, "heads"), take_int(d, "dim")
        mask = _section(d, "mask", where, optional=True)
        rot = _section(d, "rot", where, optional=True)
        cfg = cls(heads=heads, kv_heads=take_int(d, "kv_heads", default=heads), dim=dim,
                  scale=take_float(d, "scale", default=dim ** -0.5),
                  window=take_int(mask, "size", default=0) if mask is not None else 0,
                  rot_dims=take_int(rot, "dims", default=dim, minimum=0) if rot is not None else 0,
                  rot_base=take_float(rot, "base", default=10000.0) if rot is not None else 10000.0)
        if take_int(d, "vdim", default=dim) != dim:
            raise ConfigError(f"config.json: {where}values are keys: vdim must be dim")
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"config.json: {where}{cfg.heads} heads are not a multiple of {cfg.kv_heads} kv_heads")
        if cfg.rot_dims % 2 or cfg.rot_dims > dim:
            raise ConfigError(f"config.json: {where}rot.dims {cfg.rot_dims} must be even and at most {dim}")
        if cfg.rot_dims and cfg.rot_base <= 0:
            raise ConfigError(f"config.json: {where}rot.base must be positive")
        return cfg


@dataclass(frozen=True)
class GlaConfig:
    heads: int
    dim: int
    vdim: int
    tau: float

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "GlaConfig":
        dim = take_int(d, "dim")
        cfg = cls(heads=take_int(d, "heads"), dim=dim, vdim=take_int(d, "vdim", default=dim),
                  tau=take_float(d, "tau", default=1.0))
        if not cfg.tau > 0:
            raise ConfigError(f"config.json: {where}tau must be positive")
        return cfg


@dataclass(frozen=True)
class SharedLatentConfig:
    heads: int
    dim: int  # unrotated query/key dimensions per head
    rot_dim: int  # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: PairRotation
    kv_from: Optional[int]  # the layer whose latents are read; None: its own

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "SharedLatentConfig":
        dim, rot_dim = take_int(d, "dim", minimum=0), take_int(d, "rot_dim", default=0, minimum=0)
        if dim + rot_dim <= 0:
            raise ConfigError(f"config.json: {where}a head needs query dimensions")
        rot_d = _section(d, "rot", where, optional=True)
        rot = PairRotation.from_dict(rot_d, where + "rot.", rot_dim) if rot_dim else PairRotation(0, 10000.0, None)
        return cls(heads=take_int(d, "heads"), dim=dim, rot_dim=rot_dim, vdim=take_int(d, "vdim", default=max(dim, 1)),
                   q_rank=take_int(d, "q_rank"), kv_rank=take_int(d, "kv_rank"),
                   scale=take_float(d, "scale", default=(dim + rot_dim) ** -0.5), rot=rot,
                   kv_from=take_int(d, "kv_from", default=None, minimum=0))


@dataclass(frozen=True)
class NutatarMlpConfig:
    kind: str  # "dense" | "moe"
    ff: int  # the dense width, or one expert's
    limit: Optional[float] = None  # of the experts; None: nothing is clamped
    experts: int = 0
    top: int = 0
    group_count: int = 1
    group_keep: int = 1
    shared_ff: int = 0  # 0: no expert that every token uses
    shared_limit: Optional[float] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "NutatarMlpConfig":
        kind = d.get("kind", "dense")
        if kind == "dense":
            return cls(kind="dense", ff=take_int(d, "ff"))
        if kind != "moe":
            raise ConfigError(f"config.json: {where}kind {kind!r} is not supported (dense, moe)")
        expert, router = _section(d, "expert", where), _section(d, "router", where)
        shared = _section(d, "shared", where, optional=True)
        experts, top = take_int(router, "experts"), take_int(router, "top")
        groups = _section(router, "groups", where + "router.", optional=True)
        count = keep = 1
        if groups is not None:
            count = take_int(groups, "count")
            keep = take_int(groups, "keep", default=count)
        if top > experts:
            raise ConfigError(f"config.json: {where}router.top {top} exceeds the {experts} experts")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"config.json: {where}{experts} experts in {count} groups of which {keep} stay open "
                              f"cannot give {top} choices")
        cfg = cls(kind="moe", ff=take_int(expert, "ff"), limit=take_float(expert, "limit", default=None), experts=experts,
                  top=top, group_count=count, group_keep=keep,
                  shared_ff=take_int(shared, "ff") if shared is not None else 0,
                  shared_limit=take_float(shared, "limit", default=None) if shared is not None else None)
        for limit in (cfg.limit, cfg.shared_limit):
            if limit is not None and limit < 0:
                raise ConfigError(f"config.json: {where}a limit must not be negative")
        return cfg


@dataclass(frozen=True)
class NutatarLayerConfig:
    type: str  # "attention" | "gla" | "latent_attention"
    mixer: Any  # KeyValueAttentionConfig | GlaConfig | SharedLatentConfig
    mlp: Optional[NutatarMlpConfig]


_MIXERS = {"attention": KeyValueAttentionConfig, "gla": GlaConfig, "latent_attention": SharedLatentConfig}


@dataclass(frozen=True)
class NutatarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[NutatarLayerConfig, ...]
    max_position: int = 32768
    architecture: str = "Nutatar"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "NutatarConfig":
        if d.get("architecture") != "Nutatar":
            raise ConfigError(f"NutatarConfig cannot read architecture {d.get('architecture')!r}")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, ld in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(ld, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = ld.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is not supported ({', '.join(sorted(_MIXERS))})")
            mixer = _MIXERS[kind].from_dict(_section(ld, "mixer", where), where + "mixer.")
            mlp_d = _section(ld, "mlp", where, optional=True)
            layers.append(NutatarLayerConfig(kind, mixer, NutatarMlpConfig.from_dict(mlp_d, where + "mlp.")
                                             if mlp_d is not None else None))
        for i, layer in enumerate(layers):
            j = layer.mixer.kv_from if layer.type == "latent_attention" else None
            if j is None:
                continue
            if j >= i or layers[j].type != "latent_attention":
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from must name an earlier layer of latent attention")
            src = layers[j].mixer
            if src.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from names layer {j}, which keeps no cache")
            if (src.kv_rank, src.rot_dim, src.rot) != (layer.mixer.kv_rank, layer.mixer.rot_dim, layer.mixer.rot):
                raise ConfigError(f"config.json: layers[{i}] reads layer {j}'s cache but differs from it in kv_rank, "
                                  f"rot_dim or rotation")
        emb = _section(d, "embedding", "", optional=True)
        return cls(vocab=take_int(d, "vocab"), width=take_int(d, "width"), norm_eps=take_float(_section(d, "norm", ""), "eps"),
                   embedding_scale=take_float(emb, "scale", default=1.0) if emb is not None else 1.0,
                   layers=tuple(layers), max_position=take_int(d, "max_position", default=32768))
