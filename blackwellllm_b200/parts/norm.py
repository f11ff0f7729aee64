"""RMSNorm: y = x * rsqrt(mean(x^2) + eps) * w, the sum and the scaling in float32.

Formula of the reference: src/kernels/rmsnorm.cu:107-120,133-138 (it sums in
double and rounds twice through bfloat16; here: one float32 computation and one
rounding on store).  ``rows`` normalises only the named rows (final norm on the
positions whose logits are wanted, src/core/engine.cpp:1029-1035).  With the spec's ``offset`` the gain is
``offset + w`` (a weight stored around zero with offset 1), made once at load in float32.

:class:`LayerNorm`: (x - mean) / sqrt(mean((x - mean)^2) + eps) * w, no bias, everything float32.

:class:`DynamicTanh`: tanh(alpha x) * w + b with a number alpha and a vector b stored beside the weight; no statistic of the row.

All describe themselves to kernels that norm a row inside another pass over it (``row_norm``: the kind, the float32
gain and eps, or for the last one (kind, gain, alpha, bias), as ``ops.row_step`` takes them).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import BuildContext, Norm, ParamSpec, register_norm


class RMSNorm(Norm):
    adds_pending = True

    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.eps = float(spec.eps)
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.param = getattr(spec, "param", "weight")
        self.offset = float(getattr(spec, "offset", 0.0))
        self.weight: Optional[torch.Tensor] = None
        self._gain_f32: Optional[torch.Tensor] = None

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.param, (self.hidden_size,), role="gain", init="ones" if self.offset == 0.0 else "bias_normal")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        w = tensors[self.param]
        if self.offset != 0.0:
            w = w.float() + self.offset     # the gain itself, float32
        self.weight = w.contiguous()
        self._gain_f32 = None

    def gain_f32(self) -> torch.Tensor:
        """The gain as a float32 vector (for kernels that norm inside another pass over the row)."""
        if self._gain_f32 is None:
            self._gain_f32 = self.weight.float().contiguous()
        return self._gain_f32

    def row_norm(self) -> tuple:
        return ops.NORM_RMS, self.gain_f32(), self.eps

    def add_to(self, x: torch.Tensor, stream: torch.Tensor) -> None:
        """``stream += norm(x)`` (float32 both): the norm of a sublayer's output on its way into the stream."""
        ops.rmsnorm_add(x, self.weight, self.eps, stream)

    def add_to_then(self, x: torch.Tensor, stream: torch.Tensor, then: "Norm") -> torch.Tensor:
        """``stream += norm(x)``, then ``then.forward(stream)``: one kernel when ``then`` is an RMS norm too."""
        if type(then) is RMSNorm and then.weight.dtype == self.weight.dtype:
            return ops.rmsnorm_add_norm(x, self.weight, self.eps, stream, then.weight, then.eps, self.ctx.dtype)
        self.add_to(x, stream)
        return then.forward(stream)

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.rmsnorm(x, self.weight, self.eps, self.ctx.dtype, rows=rows)


class LayerNorm(Norm):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.eps = float(spec.eps)
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.param = getattr(spec, "param", "weight")
        self.gain: Optional[torch.Tensor] = None

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.param, (self.hidden_size,), role="gain", init="ones")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.gain = tensors[self.param].float().contiguous()

    def row_norm(self) -> tuple:
        return ops.NORM_LAYER, self.gain, self.eps

    def add_to(self, x: torch.Tensor, stream: torch.Tensor) -> None:
        ops.row_step(stream, x, post=self.row_norm())

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.row_step(x, then=self.row_norm(), rows=rows, out_dtype=self.ctx.dtype)


class DynamicTanh(Norm):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.names = (spec.param, spec.alpha_param, spec.bias_param)
        self.gain: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None
        self.alpha = 1.0

    def param_specs(self) -> List[ParamSpec]:
        w, alpha, b = self.names
        return [ParamSpec(w, (self.hidden_size,), role="gain", init="ones"), ParamSpec(alpha, (), role="gain", init="ones"),
                ParamSpec(b, (self.hidden_size,), role="bias", init="bias_normal")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        w, alpha, b = self.names
        self.gain, self.bias = tensors[w].float().contiguous(), tensors[b].float().contiguous()
        self.alpha = float(tensors[alpha])

    def row_norm(self) -> tuple:
        return ops.NORM_TANH, self.gain, self.alpha, self.bias

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        return ops.row_step(x, then=self.row_norm(), rows=rows, out_dtype=self.ctx.dtype)


register_norm("rmsnorm", RMSNorm)
register_norm("layernorm", LayerNorm)
register_norm("dynamic_tanh", DynamicTanh)
