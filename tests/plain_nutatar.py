"""The Nutatar decoder restated plainly: whole sequences, no cache, no batching,
one function per mechanism, float64 unless told otherwise.  It shares no code
with the package; the tests hold the package against it.

Notation: ``x`` [T, width] is one sequence's residual stream, ``W`` tensors are
stored [out, in] and applied as ``x @ W.T``; ``w`` is the dictionary of the
checkpoint's tensors by name, ``cfg`` the dictionary of config.json.
"""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """Every row divided by the root of (the mean of its squares + eps), times ``weight``."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


# ---- positions ---------------------------------------------------------------------------
def frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def ramp_frequencies(dims: int, base: float, s: Optional[Dict]):
    """(frequencies, magnitude): with ``s`` = {factor, original, fast, slow} every frequency is a blend of
    itself and itself over ``factor``; the share of the latter climbs with the pair's index."""
    f = frequencies(dims, base)
    if s is None:
        return f, 1.0

    def index_with(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_with(s["fast"])), 0), min(math.ceil(index_with(s["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        share = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(share * v / s["factor"] + (1.0 - share) * v)
    return out, 0.1 * math.log(s["factor"]) + 1.0


def cos_sin(T: int, freqs: List[float], dtype):
    angle = torch.arange(T, dtype=dtype)[:, None] * torch.tensor(freqs, dtype=dtype)[None, :]
    return torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]


def rotate_half(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x`` [T, heads, d]: elements i and i + dims/2 (i < dims/2) of each head turned by position times
    frequency i; elements from ``dims`` on as they are."""
    if not dims:
        return x
    c, s = cos_sin(x.shape[0], frequencies(dims, base), x.dtype)
    a, b = x[..., : dims // 2], x[..., dims // 2: dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def rotate_neighbours(x: torch.Tensor, dims: int, base: float, scaling: Optional[Dict]) -> torch.Tensor:
    """``x`` [T, heads, d]: elements 2i and 2i + 1 (i < dims/2) of each head turned, cosine and sine times
    the magnitude that comes with ``scaling``; elements from ``dims`` on as they are."""
    if not dims:
        return x
    freqs, mag = ramp_frequencies(dims, base, scaling)
    c, s = cos_sin(x.shape[0], freqs, x.dtype)
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = (a * c - b * s) * mag
    out[..., 1:dims:2] = (b * c + a * s) * mag
    return out


# ---- softmaxes ----------------------------------------------------------------------------
def visible(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] booleans: query i sees key j when 0 <= i - j, and with ``window`` i - j < window."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax_beside(scores: torch.Tensor, see: torch.Tensor, sink) -> torch.Tensor:
    """Softmax over the visible keys with exp(sink) more in the denominator (``sink`` a number)."""
    s = scores.masked_fill(~see, float("-inf"))
    top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(float(sink) - top))


# ---- mixers -------------------------------------------------------------------------------
def attention(h: torch.Tensor, m: Dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G = m.get("kv_heads") or H
    scale = m["scale"] if m.get("scale") is not None else d ** -0.5
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    raw_k = h @ w[p + "k"].T
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(raw_k, w[p + "k.norm"], eps).reshape(T, G, d)
    v = raw_k.reshape(T, G, d)
    q, k = rotate_half(q, rot["dims"], rot["base"]), rotate_half(k, rot["dims"], rot["base"])
    see = visible(T, (m.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        g = a // (H // G)
        heads.append(softmax_beside(q[:, a] @ k[:, g].T * scale, see, 0.0) @ v[:, g])
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def latents(h: torch.Tensor, m: Dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    """(latent c [T, kv_rank], rotated key part [T, rot_dim]) of every token."""
    R, rd = m["kv_rank"], m.get("rot_dim") or 0
    both = h @ w[p + "dkv"].T
    c = rms_norm(both[:, :R], w[p + "dkv.norm"], eps)
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    r = rotate_neighbours(both[:, None, R: R + rd], rot.get("dims", rd), rot["base"], rot.get("scaling"))[:, 0]
    return c, r


def latent_attention(h: torch.Tensor, cr, m: Dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """``cr``: what ``latents`` gave, of this layer or of the one it reads."""
    T = h.shape[0]
    H, d, rd = m["heads"], m["dim"], m.get("rot_dim") or 0
    e = m.get("vdim") or d
    scale = m["scale"] if m.get("scale") is not None else (d + rd) ** -0.5
    rot = m.get("rot") or {"dims": 0, "base": 10000.0}
    c, r = cr
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, d + rd)
    qr = rotate_neighbours(q[..., d:], rot.get("dims", rd), rot["base"], rot.get("scaling"))
    k, v = (c @ w[p + "uk"].T).reshape(T, H, d), (c @ w[p + "uv"].T).reshape(T, H, e)
    gate = torch.sigmoid(h @ w[p + "g"].T)
    see = visible(T, None)
    heads = []
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + qr[:, a] @ r.T) * scale
        heads.append(softmax_beside(s, see, w[p + "sink"][a]) @ v[:, a] * gate[:, a: a + 1])
    return torch.cat(heads, dim=1) @ w[p + "o"].T


def decays(h: torch.Tensor, tau: float, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    """[T, heads * dim]: sigmoid(z)^(1/tau), z through the low-rank pair."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def decayed_state(q, k, v, a) -> torch.Tensor:
    """One head, token by token: the rows of S fade by ``a``, k v^T is added, the result is read by q."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = []
    for t in range(q.shape[0]):
        S = a[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def gla(h: torch.Tensor, m: Dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    e = m.get("vdim") or d
    q = (h @ w[p + "q"].T * d ** -0.5).reshape(T, H, d)
    k, v = (h @ w[p + "k"].T).reshape(T, H, d), (h @ w[p + "v"].T).reshape(T, H, e)
    a = decays(h, m.get("tau", 1.0), w, p).reshape(T, H, d)
    heads = [rms_norm(decayed_state(q[:, n], k[:, n], v[:, n], a[:, n]), w[p + "norm"], eps) for n in range(H)]
    g = h @ w[p + "g"].T
    return (torch.cat(heads, dim=1) * g * torch.sigmoid(g)) @ w[p + "o"].T


# ---- feed-forwards --------------------------------------------------------------------------
def squared_relu(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def expert(h: torch.Tensor, limit: Optional[float], w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    if limit is not None:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(z: torch.Tensor, top: int, count: int, keep: int):
    """One token's logits -> [(expert, weight)]: softmax over all, the best groups by their best expert, the
    best experts inside them (the lower index first among equals), weights as the softmax gave them."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    E = len(s)
    per = E // count
    groups = sorted(range(count), key=lambda g: (-float(s[g * per: (g + 1) * per].max()), g))[:keep]
    open_ = [e for e in range(E) if e // per in groups]
    chosen = sorted(open_, key=lambda e: (-float(s[e]), e))[:top]
    return [(e, s[e]) for e in chosen]


def experts(h: torch.Tensor, mlp: Dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[p + "router"].T
    limit = mlp["expert"].get("limit")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in route(z[t], r["top"], groups["count"], groups.get("keep", groups["count"])):
            out[t] += s * expert(h[t: t + 1], limit, w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + expert(h, mlp["shared"].get("limit"), w, p + "shared.")
    return out


# ---- the model --------------------------------------------------------------------------------
def forward(tokens: List[int], cfg: Dict, weights: Dict[str, torch.Tensor], dtype=F, keep_layers: bool = False):
    """Logits [T, vocab]; with ``keep_layers`` also the stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    kept, cached = [], {}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        if spec["type"] == "latent_attention":
            if m.get("kv_from") is None:
                cached[i] = latents(x, m, w, p + "mix.", eps)
                y = latent_attention(x, cached[i], m, w, p + "mix.", eps)
            else:
                y = latent_attention(x, cached[m["kv_from"]], m, w, p + "mix.", eps)
        else:
            y = {"attention": attention, "gla": gla}[spec["type"]](x, m, w, p + "mix.", eps)
        x = x + rms_norm(y, w[p + "norm1"], eps)
        f = spec.get("mlp")
        if f is not None:
            y = squared_relu(x, w, p + "mlp.") if f["kind"] == "dense" else experts(x, f, w, p + "mlp.")
            x = x + rms_norm(y, w[p + "norm2"], eps)
        kept.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
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
