"""The Menitar decoder restated plainly: whole sequences, no cache, no batching,
one function per mechanism, float64 unless told otherwise.  It shares no code
with the package; the tests hold the package against it.

Notation: ``x`` [T, width] is one sequence's residual stream, ``W`` tensors are
stored [out, in] and applied as ``x @ W.T``; ``w`` is the dictionary of the
checkpoint's tensors by name, ``cfg`` the dictionary of config.json.
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """Every row divided by the root of (the mean of its squares + eps), times ``weight``."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def rotate_half(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x`` [T, heads, d]: elements i and i + dims/2 (i < dims/2) of each head turned by
    ``position * base^(-2i/dims)``; elements from ``dims`` on as they are."""
    if not dims:
        return x
    half = dims // 2
    freqs = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None] * freqs[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def visible(T: int, chunk: Optional[int]) -> torch.Tensor:
    """[T, T] booleans: query i sees key j <= i, and with ``chunk`` only in its own run of ``chunk``
    positions, runs counted from position 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if chunk:
        see = see & (i // chunk == j // chunk)
    return see


def mixed_scores(q: torch.Tensor, k: torch.Tensor, scale: float, temp: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """``q`` [T, H, d], ``k`` [T, G, d] -> [H, T, T]: the heads' scaled scores times the head's
    temperature, then every head's row replaced by the combination of all heads' that its row of
    ``talk`` names."""
    H, G = q.shape[1], k.shape[1]
    raw = torch.stack([q[:, a] @ k[:, a // (H // G)].T for a in range(H)]) * scale
    return torch.einsum("hg,gij->hij", talk, raw * temp[:, None, None])


def softmax_over(scores: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    s = scores.masked_fill(~see, float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def attention(h: torch.Tensor, m: Dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, e = m.get("kv_heads") or H, m.get("vdim") or d
    scale = m["scale"] if m.get("scale") is not None else d ** -0.5
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    pos = torch.arange(T)
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, e)
    q = rotate_half(q, pos, rot["dims"], rot["base"])
    k = rotate_half(k, pos, rot["dims"], rot["base"])
    prob = softmax_over(mixed_scores(q, k, scale, w[p + "temp"], w[p + "talk"]),
                        visible(T, (m.get("mask") or {}).get("size")))
    gate = torch.sigmoid(h @ w[p + "g"].T)  # [T, H]
    o = torch.stack([(prob[a] @ v[:, a // (H // G)]) * gate[:, a, None] for a in range(H)], dim=1)
    return o.reshape(T, H * e) @ w[p + "o"].T


def clamped_gated(h: torch.Tensor, mlp: Dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    limit = mlp.get("limit")
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    if limit is not None:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def layer(x: torch.Tensor, spec: Dict, cfg: Dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    eps = cfg["norm"]["eps"]
    y = attention(rms_norm(x, w[p + "norm1"], eps), spec["mixer"], w, p + "mix.", eps)
    if spec.get("mlp") is not None:
        y = y + clamped_gated(rms_norm(x, w[p + "norm2"], eps), spec["mlp"], w, p + "mlp.")
    return x + y


def run_order(cfg: Dict):
    """(layer, pass or None) of every run; the pass's number stands at its first layer only."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(tokens: List[int], cfg: Dict, weights: Dict[str, torch.Tensor], dtype=F, keep_layers: bool = False):
    """Logits [T, vocab]; with ``keep_layers`` also the stream after every run of a layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    x0 = w["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    x, kept = x0, []
    for i, enter in run_order(cfg):
        if enter is not None:
            if enter > 0:
                x = x + x0
            x = x + w["loop.step"][enter]
        x = layer(x, cfg["layers"][i], cfg, w, f"l{i}.")
        kept.append(x)
    x = rms_norm(x, w["final.norm"], cfg["norm"]["eps"])
    logits = x @ w["embed"].T * cfg.get("logit_scale", 1.0)
    return (logits, torch.stack(kept)) if keep_layers else logits


def argmax(logits: torch.Tensor) -> int:
    """The lowest index among the largest values."""
    return int((logits == logits.max()).nonzero()[0])


def read_config(folder_or_dict) -> dict:
    import json
    import os

    if isinstance(folder_or_dict, dict):
        return folder_or_dict
    with open(os.path.join(folder_or_dict, "config.json")) as fh:
        return json.load(fh)


def read_weights(folder: str) -> Dict[str, torch.Tensor]:
    import os

    from safetensors.torch import load_file

    return {k: (v.to(F) if v.is_floating_point() else v) for k, v in
            load_file(os.path.join(folder, "model.safetensors")).items()}


class Plain:
    """The plain implementation over a model folder, logits cached by sequence."""

    def __init__(self, folder: Optional[str], config: Optional[dict] = None, weights=None):
        self.cfg = read_config(folder if folder is not None else config)
        self.weights = read_weights(folder) if folder is not None else weights
        self._cache: Dict[tuple, torch.Tensor] = {}

    def logits(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._cache:
            with torch.no_grad():
                self._cache[key] = forward(list(tokens), self.cfg, self.weights).to(torch.float32)
        return self._cache[key]
