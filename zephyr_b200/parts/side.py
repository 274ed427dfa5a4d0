"""Parts that join the stream behind a layer's mixer and feed-forward, made from the stream itself.

``token_gate``: y = P (gelu(G x) * e), joined as x + N(y), where e is the layer's part (``dim`` values from ``offset`` on)
of the token's row in a table that all such layers share, gelu is the tanh form and N an RMS norm with a scale.  The
two products run in the model's type with float32 sums; the gate and its product with e are float32 with one rounding,
in the first product's epilogue for few rows, one pass over its sums otherwise.
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..config.errors import ConfigError
from ..config.spec import SideSpec
from ..kernels import ops
from ..weights.loader import ROLE_EMBEDDING, ROLE_LINEAR, WeightDecl
from .base import NORMS, DeferredSum, SidePart, StepContext, lookup, register_side


class TokenGate(SidePart):
    graph_safe = True

    def __init__(self, spec: SideSpec, weights: Mapping[str, torch.Tensor], dtype: torch.dtype):
        p = spec.params
        self.dim, self.offset = int(p["dim"]), int(p["offset"])
        self.table = weights[p["table"]]
        if self.dim <= 0 or self.offset < 0 or self.offset + self.dim > self.table.shape[1]:
            raise ConfigError("a layer's part lies inside a row of the table")
        self.w_gate, self.w_proj = weights[p["gate"]], weights[p["proj"]]
        self.norm = lookup(NORMS, "norm", p["norm"].kind)(p["norm"], weights, dtype)
        if not hasattr(self.norm, "add_scaled"):
            raise ConfigError("the norm behind a token gate joins the stream as it norms (add_scaled)")

    @staticmethod
    def weight_decls(spec: SideSpec) -> dict[str, WeightDecl]:
        p = spec.params
        hidden, dim = int(p["hidden_size"]), int(p["dim"])
        decls = dict(lookup(NORMS, "norm", p["norm"].kind).weight_decls(p["norm"]))
        decls[p["table"]] = WeightDecl((int(p["vocab_size"]), int(p["row"])), ROLE_EMBEDDING)
        decls[p["gate"]] = WeightDecl((dim, hidden), ROLE_LINEAR)
        decls[p["proj"]] = WeightDecl((hidden, dim), ROLE_LINEAR)
        return decls

    def weights_read(self) -> list[torch.Tensor]:
        return [self.w_gate, self.w_proj, *self.norm.weights_read()]      # a step gathers a few rows of the table

    def forward(self, x: torch.Tensor, ctx: StepContext) -> DeferredSum:
        if x.shape[0] <= ops.SMALL_GEMM_ROWS and ops.gemm_small_supported(x, self.w_gate):
            gated = ops.gemm_small_token_gate(x, self.w_gate, self.table, self.offset, ctx.token_ids, ctx.status)
        else:
            gate = ops.linear(x, self.w_gate, out_dtype=torch.float32)
            gated = ops.token_gate(gate, self.table, self.offset, ctx.token_ids, ctx.status)
        return DeferredSum(ops.linear(gated, self.w_proj), self.norm, 1.0)


register_side("token_gate", TokenGate)
