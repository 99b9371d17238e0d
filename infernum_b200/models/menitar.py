"""The Menitar decoder as a model description.

A decoder-only model of parallel layers: mixer and feed-forward read two RMS
norms of the same stream and their sum is added to it.  The mixer is grouped-
query attention within runs of positions (a query sees the keys of its own run),
with one RMS norm over all of a token's queries and one over all of its keys,
rotation of halves in a part of each head, scores scaled per head and then
exchanged among all heads by a learned matrix, and one sigmoid gate per head on
the result.  Feed-forwards are gated with a clamped swish, ``g sigmoid(1.702 g)
(u + 1)``.  A run of layers may be walked several times with the same weights;
every pass begins with the sum of the stream, a learned vector and - but for the
first - the embedding's output.  The embedding is scaled; the head is the
embedding table, its logits scaled.

Checkpoint names: ``embed``, ``loop.step``, ``l<i>.norm1|norm2``, ``l<i>.mix.{q, k, v, o,
q.norm, k.norm, talk, temp, g}``, ``l<i>.mlp.{gate, up, down}``, ``final.norm``.
"""

from __future__ import annotations

from ..config.menitar import MenitarConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleItem
from ..registry import register_architecture

SWISH_ALPHA = 1.702


def build_menitar_spec(cfg: MenitarConfig) -> ModelSpec:
    def norm(name: str, optional: bool = False) -> PartSpec:
        return PartSpec("rmsnorm", {"hidden_size": cfg.width, "eps": cfg.norm_eps, "weight": name, "optional": optional})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        parts = {
            "norm1": norm(p + "norm1"),
            # (a layer without a feed-forward may come with its second norm; nothing reads it)
            "norm2": norm(p + "norm2", optional=layer.mlp is None),
            "mixer": PartSpec("talking_attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                "scale": m.scale, "chunk": m.chunk,
                "rotary": {"dims": m.rot_dims, "theta": m.rot_base} if m.rot_dims else None,
                "qk_norm": {"q": "q.norm", "k": "k.norm", "eps": cfg.norm_eps},
                "talk": "talk", "temp": "temp", "gate": "g", "prefix": p + "mix."})}
        if layer.mlp is not None:
            parts["ffn"] = PartSpec("swiglu", {
                "hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "prefix": p + "mlp.",
                "names": {"gate": "gate", "up": "up", "down": "down"}, "activation": "clamped_swish",
                "limit": layer.mlp.limit, "alpha": SWISH_ALPHA})
        layers.append(LayerSpec(block="parallel_prenorm", name=p, parts=parts))

    L = len(layers)
    schedule, entry = [ScheduleItem(i) for i in range(L)], None
    if cfg.loop is not None:
        start, stop, times = cfg.loop
        schedule = [ScheduleItem(i) for i in range(start)]
        for t in range(times):
            schedule += [ScheduleItem(i, enter=t if i == start else None) for i in range(start, stop)]
        schedule += [ScheduleItem(i) for i in range(stop, L)]
        entry = PartSpec("add_reentry", {"hidden_size": cfg.width, "passes": times, "step": "loop.step"})
    return ModelSpec(
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {
            "vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed", "keep_origin": entry is not None,
            "scale": cfg.embedding_scale}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "weight": "embed",
                                         "tied_to": "embed", "scale": cfg.logit_scale}),
        max_position=cfg.max_position,
        pass_entry=entry,
    )


register_architecture("Menitar", MenitarConfig.from_dict, build_menitar_spec)
