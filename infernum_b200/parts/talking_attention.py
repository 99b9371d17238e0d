"""Grouped-query attention whose heads exchange their scores before the softmax,
over the paged cache.

With ``h`` the mixer's input, H heads over G key/value heads (head a reads
key/value head a // (H / G)), queries and keys of ``dim``, values of ``vdim``:

    q = N_q(W_q h)   k = N_k(W_k h)   v = W_v h      (N: RMS norm over all heads' rows at once)
    q, k <- rotated in the first ``rotary_dim`` dimensions of every head, halves paired
    r_g(i, j) = q_g(i) . k_g(j) * scale * temp[g]
    s_h(i, j) = sum_g talk[h, g] r_g(i, j)
    o_h = softmax_j(s_h) v_h * sigmoid(W_g h)_h
    out = W_o concat_heads(o)

Query i sees keys j <= i; with ``chunk`` only those of its own run of ``chunk``
positions, counted from the sequence's start; with ``window`` only the last
``window``.  Norms, angles, scores, their exchange and the softmax are 32-bit.
One product makes q, k, v and the gate's logits.

Parameters: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``dim``, ``vdim``,
``scale``, ``chunk`` (0: none), ``window`` (0: none), ``rotary`` (None or {"dims",
"theta", "scaling"}), ``prefix``, and tensors behind the prefix: ``names`` for
``q``, ``k``, ``v``, ``o``; ``qk_norm`` (None or {"q", "k", "eps"}); ``talk`` [H, H],
``temp`` [H], ``gate`` [H, hidden] (each a name, or None for none).
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..errors import ConfigError
from ..ops import attention_talk, core
from .base import MIXERS, Mixer, PagedCacheSpec, Runtime, WeightSpec
from .linear import Linear
from .rope import rotary_inv_freq


@MIXERS.register("talking_attention")
class TalkingAttention(Mixer):
    def __init__(self, params, rt: Runtime):
        super().__init__(params, rt)
        self.hidden_size, self.heads = int(params["hidden_size"]), int(params["num_heads"])
        self.kv_heads = int(params.get("num_kv_heads") or self.heads)
        self.dim = int(params["dim"])
        self.vdim = int(params.get("vdim") or self.dim)
        scale = params.get("scale")
        self.scale = float(scale) if scale is not None else self.dim ** -0.5
        self.chunk, self.window = int(params.get("chunk") or 0), int(params.get("window") or 0)
        if self.heads % self.kv_heads:
            raise ConfigError(f"talking attention: {self.heads} heads are not a multiple of {self.kv_heads} key/value heads")
        if attention_talk.plain_floats(self.heads, self.dim, self.vdim) * 4 > attention_talk.PLAIN_SMEM:
            raise ConfigError(f"talking attention: {self.heads} heads of {self.dim} and {self.vdim} are more than a "
                              "row's shared memory holds")
        rot = params.get("rotary") or {}
        self.rotary_dim = int(rot.get("dims") or 0)
        if self.rotary_dim % 2 or self.rotary_dim > self.dim:
            raise ConfigError(f"talking attention: {self.rotary_dim} rotated dimensions must be even and at most {self.dim}")
        self.inv_freq = None
        if self.rotary_dim:
            freqs = rotary_inv_freq(self.rotary_dim, float(rot.get("theta", 10000.0)), rot.get("scaling"))
            self.inv_freq = torch.tensor(freqs, dtype=torch.float64).to(torch.float32).to(rt.device)
        p = params.get("prefix", "")
        self.prefix = p
        names = params.get("names") or {}
        self.names = {k: p + names.get(k, k) for k in ("q", "k", "v", "o")}
        norm = params.get("qk_norm")
        self.norm_names = (p + norm["q"], p + norm["k"]) if norm else None
        self.eps = float(norm["eps"]) if norm else 0.0
        self.talk_name, self.temp_name, self.gate_name = (p + params[k] if params.get(k) else None
                                                          for k in ("talk", "temp", "gate"))
        self.qkv: Optional[Linear] = None
        self.o: Optional[Linear] = None
        self.q_norm = self.k_norm = self.talk = self.q_scale = None
        self.talk_exact = True

    # ---- declarations -----------------------------------------------------
    def cache_spec(self) -> Optional[PagedCacheSpec]:
        return PagedCacheSpec(self.kv_heads, self.dim, self.window, v_head_dim=self.vdim, chunk=self.chunk)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        D, H, G = self.hidden_size, self.heads, self.kv_heads
        specs = {self.names["q"]: WeightSpec((H * self.dim, D)), self.names["k"]: WeightSpec((G * self.dim, D)),
                 self.names["v"]: WeightSpec((G * self.vdim, D)), self.names["o"]: WeightSpec((D, H * self.vdim))}
        if self.norm_names:
            specs[self.norm_names[0]] = WeightSpec((H * self.dim,), init="norm")
            specs[self.norm_names[1]] = WeightSpec((G * self.dim,), init="norm")
        if self.talk_name:
            specs[self.talk_name] = WeightSpec((H, H), std=H ** -0.5)
        if self.temp_name:
            specs[self.temp_name] = WeightSpec((H,), init="norm")
        if self.gate_name:
            specs[self.gate_name] = WeightSpec((H, D))
        return specs

    def bind(self, weights) -> None:
        mats = [weights[self.names[n]] for n in ("q", "k", "v")]
        if self.gate_name:
            mats.append(weights[self.gate_name])
        if len({m.dtype for m in mats}) != 1:
            raise ConfigError(f"{self.prefix}: q, k, v and the gate are stored in different dtypes")
        rows = sum(m.shape[0] for m in mats)
        if rows % 8:  # rows of the product 16 bytes apart
            mats.append(torch.zeros((8 - rows % 8, self.hidden_size), dtype=mats[0].dtype, device=mats[0].device))
        self.qkv = Linear(torch.cat(mats, dim=0), self.rt)
        self.o = Linear(weights[self.names["o"]], self.rt)
        f32 = lambda name: weights[name].to(torch.float32).contiguous() if name else None  # noqa: E731
        if self.norm_names:
            self.q_norm, self.k_norm = (weights[n].contiguous() for n in self.norm_names)
            if self.q_norm.dtype != self.k_norm.dtype:
                self.q_norm, self.k_norm = self.q_norm.float(), self.k_norm.float()
        self.talk = f32(self.talk_name)
        # the scores' scale and the heads' temperatures go into the queries, before these are rounded
        temp = f32(self.temp_name) if self.temp_name else torch.ones(self.heads, device=self.qkv.weight.device)
        self.q_scale = (temp * self.scale).contiguous()
        # the tensor cores take the exchange's weights in bfloat16: those of a bfloat16 checkpoint are
        self.talk_exact = self.talk is None or bool((self.talk == self.talk.to(torch.bfloat16).float()).all())

    def weight_bytes(self) -> int:
        return self.qkv.nbytes + self.o.nbytes

    # ---- the step -----------------------------------------------------------
    @property
    def out_proj(self) -> Linear:
        """The product that ends the sub-layer."""
        return self.o

    def forward(self, x: torch.Tensor, ctx, cache) -> torch.Tensor:
        out = torch.empty((x.shape[0], self.heads * self.vdim), dtype=x.dtype, device=x.device)
        self.forward_hidden(x, ctx, cache, out)
        return self.o(out)

    def forward_hidden(self, x: torch.Tensor, ctx, cache, out: torch.Tensor) -> None:
        """What the last product reads, into ``out`` [N, heads * vdim] (may lie in wider rows)."""
        if not cache.owner:
            raise ConfigError("talking attention must own its cache")
        tables = ctx.block_tables[cache.group]
        rows = self.qkv(x)
        core.qk_row_norm_append(rows, self.q_norm, self.k_norm, self.eps, self.q_scale, self.inv_freq, self.rotary_dim,
                                self.heads, self.kv_heads, self.dim, self.vdim, ctx.positions, ctx.row_entry, tables,
                                cache.k_pool, cache.v_pool, self.rt.err)
        gate = None
        if self.gate_name:
            g0 = (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim
            gate = rows[:, g0: g0 + self.heads]
        # bfloat16 with sizes that have a variant: the tensor-core kernel; everything else the plain 32-bit one
        if not (self.talk_exact and attention_talk.run(rows, cache.k_pool, cache.v_pool, out, ctx, tables, self.heads,
                                                       self.talk, gate, self.chunk, self.window, self.rt)):
            core.attention_talk(rows, cache.k_pool, cache.v_pool, out, ctx, tables, self.heads, self.talk, gate,
                                self.chunk, self.window, self.rt.err)
