"""The Nutatar decoder as a model description.

A decoder-only model whose layers norm a sub-layer's result, not its input:
``x <- x + norm1(mixer(x))``, then ``x <- x + norm2(ff(x))``, RMS norms.  A layer's mixer
is one of three: ``attention`` - grouped-query attention within a sliding window
whose values are its projected keys, with one RMS norm over all of a token's
queries and one over all of its keys, rotation of halves in a part of each head,
and a one more in the softmax's denominator; ``gla`` - gated linear attention: a
matrix state per head whose key channels fade by decays made from the token;
``latent_attention`` - attention through a low-rank latent of keys and values (which
an earlier layer may have cached), neighbours rotated with frequencies rescaled
along a ramp, a learned sink and a sigmoid gate per head.  Feed-forwards are a
squared-relu layer or a mixture of clamped-swish experts routed by a softmax over
all of them within the best groups, beside an expert that every token uses.  The
embedding is scaled.

Checkpoint names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (attention: ``q, k, o, q.norm,
k.norm``; gla: ``q, k, v, g, a1, a2, a2.b, norm, o``; latent_attention: ``dq, dq.norm, uq,
dkv, dkv.norm, uk, uv, sink, g, o``), ``l<i>.mlp.{up, down}`` or ``l<i>.mlp.{router,
e<j>.{gate, up, down}, shared.{gate, up, down}}``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.nutatar import NutatarConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleItem
from ..registry import register_architecture

SWISH_ALPHA = 1.702


def _mixer(kind: str, m, cfg: NutatarConfig, prefix: str) -> PartSpec:
    common = {"hidden_size": cfg.width, "num_heads": m.heads, "prefix": prefix}
    if kind == "attention":
        return PartSpec("attention", {
            **common, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "window": m.window, "scale": m.scale,
            "position": {"kind": "rotary", "params": {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base}}
            if m.rot_dims else None,
            "names": {"q": "q", "k": "k", "o": "o"}, "value_from_key": True, "sink_logit": 0.0,
            "qk_norm": {"q": "q.norm", "k": "k.norm", "eps": cfg.norm_eps, "over": "projection"}})
    if kind == "gla":
        return PartSpec("gla", {**common, "head_dim": m.dim, "vdim": m.vdim, "tau": m.tau, "eps": cfg.norm_eps})
    s = m.rot.scaling
    return PartSpec("latent_attention", {
        **common, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
        "scale": m.scale, "window": 0, "eps": cfg.norm_eps, "rotary_dim": m.rot.dims, "theta": m.rot.base,
        "rotary_scaling": {"rope_type": "ramp", "factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
        if s is not None else None,
        "rotary_pairing": "adjacent", "kv_shared": m.kv_from is not None, "sink": "sink", "gate": "g"})


def _feed_forward(f, cfg: NutatarConfig, prefix: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("mlp", {"hidden_size": cfg.width, "intermediate_size": f.ff, "prefix": prefix,
                                "activation": "relu2"})
    return PartSpec("moe", {
        "hidden_size": cfg.width, "expert_size": f.ff, "experts": f.experts, "top": f.top, "activation": "clamped_swish",
        "limit": f.limit, "alpha": SWISH_ALPHA, "prefix": prefix, "router_bias": None, "scoring": "softmax_all",
        "renormalize": False, "groups": {"count": f.group_count, "keep": f.group_keep, "top": 1},
        "shared": {"size": f.shared_ff, "prefix": "shared.", "gate": None, "limit": f.shared_limit} if f.shared_ff else None})


def build_nutatar_spec(cfg: NutatarConfig) -> ModelSpec:
    def norm(name: str, optional: bool = False) -> PartSpec:
        return PartSpec("part_rmsnorm", {"hidden_size": cfg.width, "eps": cfg.norm_eps, "weight": name,
                                         "optional": optional})

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        # (a layer without a feed-forward may come with its second norm; nothing reads it)
        parts = {"norm1": norm(p + "norm1"), "norm2": norm(p + "norm2", optional=layer.mlp is None),
                 "mixer": _mixer(layer.type, layer.mixer, cfg, p + "mix.")}
        if layer.mlp is not None:
            parts["ffn"] = _feed_forward(layer.mlp, cfg, p + "mlp.")
        layers.append(LayerSpec(block="subnorm", name=p, parts=parts))
        schedule.append(ScheduleItem(i, cache_of=getattr(layer.mixer, "kv_from", None)))
    return ModelSpec(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed",
                                               "act": True, "scale": cfg.embedding_scale}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "head"}),
        max_position=cfg.max_position,
    )


register_architecture("Nutatar", NutatarConfig.from_dict, build_nutatar_spec)
