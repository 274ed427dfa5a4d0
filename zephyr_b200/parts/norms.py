"""RMSNorm: y = x * rsqrt(mean(x^2) + eps) * w, statistics in float32, the scale multiplied after
the normalisation and not as (1 + w) (reference: src/layer/normalization.cpp:10-18,
deps/ttl/src/kernels/normalization/normalization.cu:76-139).

With ``groups`` > 1 each of that many equal consecutive parts of the row is divided by its own root mean square; the
scale stays one vector over the whole row.  Such a norm reads a float32 stream (``forward``, ``sum_forward``).

LayerNorm: mean and variance of the row, a scale and (where the spec names one) a shift."""

from __future__ import annotations

from typing import Mapping

import torch

from ..config.errors import ConfigError
from ..config.spec import NormSpec
from ..kernels import ops
from ..weights.loader import ROLE_NORM, ROLE_ZERO, WeightDecl
from .base import Norm, register_norm


class RMSNorm(Norm):
    graph_safe = True

    def __init__(self, spec: NormSpec, weights: Mapping[str, torch.Tensor], dtype: torch.dtype):
        self.size = spec.size
        self.eps = float(spec.eps)
        self.groups = int(spec.groups)
        if self.groups <= 0 or spec.size % self.groups != 0:
            raise ConfigError(f"a norm's groups divide its {spec.size} values evenly, {self.groups} do not")
        self.dtype = dtype
        self.weight = weights[spec.weight]
        self._scale32 = self.weight.float().contiguous()     # what the fused residual form reads

    @staticmethod
    def weight_decls(spec: NormSpec) -> dict[str, WeightDecl]:
        return {spec.weight: WeightDecl((spec.size,), ROLE_NORM)}

    def weights_read(self) -> list[torch.Tensor]:
        return [self.weight]          # (the float32 copy of the scales stands in for them, not beside them)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        if x.dtype == torch.float32 and (self.dtype != torch.float32 or self.groups > 1):
            return ops.sum_rms_norm(x, None, None, self.weight, self.eps, out_dtype=self.dtype, groups=self.groups)    # a float32 stream
        self._needs_one_group("a norm of rows in the model's type")
        return ops.rmsnorm(x, self.weight, self.eps)

    @staticmethod
    def _two_summands(stream: torch.Tensor, summands: tuple):
        """(a, b, shift) of a tuple of summands; what goes beyond two rows and a shift joins the stream here."""
        rows = [s for s in summands if s.dim() == 2]
        shifts = [s for s in summands if s.dim() == 1]
        for more in rows[2:]:
            stream.add_(more)
        shift = None
        if shifts and rows:
            shift = shifts[0] if len(shifts) == 1 else torch.stack(shifts).sum(0)
        elif shifts:
            stream.add_(torch.stack(shifts).sum(0))
        a = rows[0] if len(rows) > 0 else None
        b = rows[1] if len(rows) > 1 else None
        return a, b, shift

    def sum_forward(self, stream: torch.Tensor, summands: tuple) -> torch.Tensor:
        """stream (float32) += (the summands added to each other), in place and in float32; returns the norm
        of the sum in the model's type.  A summand is [rows, H], or a float32 [H] shift that goes on every
        row.  Two summands and a shift take one kernel for the sums and the norm."""
        a, b, shift = self._two_summands(stream, summands)
        return ops.sum_rms_norm(stream, a, b, self.weight, self.eps, out_dtype=self.dtype, bias=shift, groups=self.groups)

    def sum_rounded(self, stream: torch.Tensor, summands: tuple) -> torch.Tensor:
        """The same sums without the norm: stream += the summands; returns the stream's value in the model's type
        (in float32 the stream itself)."""
        a, b, shift = self._two_summands(stream, summands)
        rounded = self.dtype != torch.float32
        out = ops.sum_rms_norm(stream, a, b, None, 0.0, out_dtype=self.dtype, bias=shift, rounded_sum=rounded)
        return out if rounded else stream

    def _needs_one_group(self, what: str) -> None:
        if self.groups > 1:
            raise ConfigError(f"a norm in groups reads a float32 stream: {what} is not built")

    def add_forward(self, residual: torch.Tensor, delta: torch.Tensor) -> torch.Tensor:
        self._needs_one_group("the sum in the model's type")
        return ops.add_rmsnorm(residual, delta, self.weight, self.eps)

    def add_scaled(self, residual: torch.Tensor, delta: torch.Tensor, mult: float,
                   then: "RMSNorm | None" = None, rounded_sum: bool = False) -> torch.Tensor | None:
        """residual (float32) += mult * norm(delta), in place and in one kernel; with ``then`` also returns
        then(residual), with ``rounded_sum`` the sum itself in delta's type: the form a block with norms
        behind its parts uses."""
        self._needs_one_group("the norm of a part's output")
        if then is None:
            return ops.residual_rms_norm(residual, delta, self._scale32, self.eps, mult, rounded_sum=rounded_sum)
        return ops.residual_rms_norm(residual, delta, self._scale32, self.eps, mult, then._scale32, then.eps)

    def as_rms_scale(self) -> tuple[torch.Tensor, float] | None:
        return (self.weight, self.eps) if self.groups == 1 else None


class LayerNorm(Norm):
    """y = (x - mean) / sqrt(var + eps) * w + b, the variance being the mean of the squared deviations;
    statistics, scale and shift in float32.  The input may be a float32 residual stream or a tensor of
    the model's type; the output has the model's type.  ``add_scaled`` is the fused form a block with
    norms behind its parts uses: residual += m * this_norm(delta), then the next norm of the sum."""

    graph_safe = True

    def __init__(self, spec: NormSpec, weights: Mapping[str, torch.Tensor], dtype: torch.dtype):
        self.size = spec.size
        self.eps = float(spec.eps)
        self.dtype = dtype
        self.weight = weights[spec.weight].float().contiguous()
        self.bias = weights[spec.bias].float().contiguous() if spec.bias is not None else None

    @staticmethod
    def weight_decls(spec: NormSpec) -> dict[str, WeightDecl]:
        decls = {spec.weight: WeightDecl((spec.size,), ROLE_NORM)}
        if spec.bias is not None:           # a spec without the name of a shift: scale only
            decls[spec.bias] = WeightDecl((spec.size,), ROLE_ZERO)
        return decls

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.layer_norm(x, self.weight, self.bias, self.eps, out_dtype=self.dtype)

    def add_scaled(self, residual: torch.Tensor, delta: torch.Tensor, mult: float,
                   then: "LayerNorm | None" = None, rounded_sum: bool = False) -> torch.Tensor | None:
        """residual (float32) += mult * norm(delta), in place; with ``then`` also returns then(residual),
        with ``rounded_sum`` the sum itself in delta's type."""
        if then is None:
            return ops.residual_layer_norm(residual, delta, self.weight, self.bias, self.eps, mult,
                                           rounded_sum=rounded_sum)
        return ops.residual_layer_norm(residual, delta, self.weight, self.bias, self.eps, mult,
                                       then.weight, then.bias, then.eps)


register_norm("rmsnorm", RMSNorm)
register_norm("layernorm", LayerNorm)
