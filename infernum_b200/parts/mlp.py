"""Feed-forwards.

``mlp``: without a gate, ``y = act(W_up x) W_down^T``.  Parameters: ``hidden_size``,
``intermediate_size``, ``prefix``, ``names`` (of the two tensors behind the prefix: ``up``,
``down``), ``activation``: "relu2", the square of what relu leaves.

``swiglu``: SwiGLU feed-forward: ``d = (silu(x Wg^T) * (x Wu^T)) Wd^T`` with
``silu(g) = g / (1 + exp(-g))`` evaluated in 32-bit
(infernum-llama/src/graph_builder.rs:498-501; infernum-cuda/kernels/silu.cu:105-116).
Gate and up are one product.  When the intermediate size is a multiple of 64
the fused weight interleaves them 64 rows by 64 rows ([g0..g63, u0..u63,
g64..g127, u64..u127, ...]), so that one 128-row tile of the tcgen05 product
holds gates and their ups and SiLU(gate) * up can be applied in its epilogue;
otherwise it is the plain concatenation ``[Wg; Wu]``.  Only the fused copy is
kept.

Parameters: ``hidden_size``, ``intermediate_size``, ``prefix`` (checkpoint
prefix, e.g. "model.layers.0.mlp."), ``names`` (the three tensors' names
behind the prefix, default gate_proj.weight / up_proj.weight /
down_proj.weight), ``activation`` of the gate: "silu" (default),
"gelu_tanh", ``0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3)))``, or "clamped_swish",
``g' sigmoid(alpha g') (u' + 1)`` for the whole with ``g' = min(g, limit)`` and ``u'`` the
up held to [-limit, limit] (parameters ``limit``, None for none, and ``alpha``).
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..errors import ConfigError
from ..ops import core
from .base import FEED_FORWARDS, FeedForward, Runtime, WeightSpec
from .linear import Linear, matmul_nt


@FEED_FORWARDS.register("mlp")
class Mlp(FeedForward):
    def __init__(self, params, rt: Runtime):
        super().__init__(params, rt)
        self.hidden_size = int(params["hidden_size"])
        self.intermediate_size = int(params["intermediate_size"])
        prefix, names = params.get("prefix", ""), params.get("names") or {}
        self.names = {k: prefix + names.get(k, k) for k in ("up", "down")}
        self.activation = params.get("activation", "relu2")
        if self.activation != "relu2":
            raise ConfigError(f"feed-forward: unknown activation {self.activation!r}; known: relu2")
        self.up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        h, i = self.hidden_size, self.intermediate_size
        return {self.names["up"]: WeightSpec((i, h)), self.names["down"]: WeightSpec((h, i))}

    def bind(self, weights) -> None:
        self.up, self.down = (Linear(weights[self.names[k]], self.rt) for k in ("up", "down"))

    def weight_bytes(self) -> int:
        return self.up.nbytes + self.down.nbytes

    @property
    def out_proj(self) -> Linear:
        return self.down

    def forward(self, x: torch.Tensor, ctx=None) -> torch.Tensor:
        act = torch.empty((x.shape[0], self.intermediate_size), dtype=x.dtype, device=x.device)
        if x.dtype == torch.bfloat16 and self.up.weight.dtype == torch.bfloat16:
            from ..ops import gemm_tc

            # the activation in the product's epilogue, where the product is the package's own
            if gemm_tc.act_route(x, self.up.weight, act, self.activation, err=self.up.err):
                return self.down(act)
        matmul_nt(x, self.up.weight, out=act, err=self.up.err)
        core.pointwise(act, None, self.activation)
        return self.down(act)


@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    def __init__(self, params, rt: Runtime):
        super().__init__(params, rt)
        self.hidden_size = int(params["hidden_size"])
        self.intermediate_size = int(params["intermediate_size"])
        self.prefix = params.get("prefix", "")
        names = params.get("names") or {}
        self.names = {k: self.prefix + names.get(k, f"{k}_proj.weight") for k in ("gate", "up", "down")}
        self.activation = params.get("activation", "silu")
        if self.activation not in core.ACTIVATIONS:
            raise ConfigError(f"gated feed-forward: unknown activation {self.activation!r}; "
                              f"known: {sorted(core.ACTIVATIONS)}")
        limit = params.get("limit")
        self.act_args = {"limit": float("inf") if limit is None else float(limit), "alpha": float(params.get("alpha", 1.0))}
        self.gate_up: Optional[Linear] = None
        self.down: Optional[Linear] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        h, i = self.hidden_size, self.intermediate_size
        return {
            self.names["gate"]: WeightSpec((i, h)),
            self.names["up"]: WeightSpec((i, h)),
            self.names["down"]: WeightSpec((h, i)),
        }

    def bind(self, weights) -> None:
        gate = weights[self.names["gate"]]
        up = weights[self.names["up"]]
        if gate.dtype != up.dtype:
            raise ConfigError(f"{self.prefix}: gate and up projections are stored in different dtypes")
        i, h = self.intermediate_size, self.hidden_size
        self.block = None  # None: [all gates | all ups]; 64: interleaved 64 by 64
        if i % 64 == 0:
            fused = torch.stack([gate.view(i // 64, 64, h), up.view(i // 64, 64, h)], dim=1)
            self.gate_up = Linear(fused.reshape(2 * i, h), self.rt)
            self.block = 64
        else:
            self.gate_up = Linear(torch.cat([gate, up], dim=0), self.rt)
        self.down = Linear(weights[self.names["down"]], self.rt)

    def weight_bytes(self) -> int:
        return self.gate_up.nbytes + self.down.nbytes

    # the product that ends the sub-layer, for arrangements that end two sub-layers in one product
    @property
    def out_proj(self) -> Linear:
        return self.down

    def forward(self, x: torch.Tensor, ctx=None) -> torch.Tensor:
        act = torch.empty((x.shape[0], self.intermediate_size), dtype=x.dtype, device=x.device)
        self.forward_hidden(x, ctx, act)
        return self.down(act)

    def forward_hidden(self, x: torch.Tensor, ctx, act: torch.Tensor) -> None:
        """What the last product reads, into ``act`` [N, intermediate] (may lie in wider rows)."""
        fused = False
        if self.block == 64 and x.dtype == torch.bfloat16 and self.gate_up.weight.dtype == torch.bfloat16:
            from ..ops import gemm_tc

            fused = gemm_tc.swiglu_route(x, self.gate_up.weight, act, self.gate_up.err,
                                         activation=self.activation, act_limit=self.act_args["limit"],
                                         act_alpha=self.act_args["alpha"])
        if not fused:
            core.gated_act(self.gate_up(x), act, self.activation, block=self.block, **self.act_args)
