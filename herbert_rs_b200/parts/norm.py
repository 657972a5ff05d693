"""Norms.  RMSNorm: y = (x / sqrt(mean(x^2) + eps)) * w, in float
(crates/backends/backend_common/src/kernels.rs:54-64), the layer norm with a weight and, if the spec asks, a bias, and a
"norm" without statistics, tanh(alpha * x) * w + b.
A spec with `weight_offset` c stores w - c (weights around zero with c = 1); the offset is added once,
in float, when the tensor is loaded, so every kernel and the norm shared between two products see w."""

from __future__ import annotations

from .. import ops
from ..errors import ConfigError
from ..registry import register_part
from .base import Norm, ParamSpec


class RMSNorm(Norm):
    kind = "rmsnorm"

    def __init__(self, spec, rt):
        self.dim, self.eps, self.rt = spec.dim, spec.eps, rt
        self.name = getattr(spec, "weight_name", "weight")
        self.offset = float(getattr(spec, "weight_offset", 0.0))
        self.groups = int(getattr(spec, "groups", 1))
        if self.groups < 1 or self.dim % self.groups:
            raise ConfigError(f"a norm over {self.dim} channels cannot be cut into {self.groups} equal parts")
        self.weight = None

    def param_specs(self):
        # random weights lie around 1 - offset: the factor the kernels see is around 1 either way
        return {self.name: ParamSpec((self.dim,), role="vector", init="ones_noise" if self.offset == 0.0 else "zeros_noise")}

    def load(self, tensors):
        w = tensors[self.name]
        self.weight = (w + self.offset if self.offset != 0.0 else w).contiguous()

    def weight_bytes(self):
        return self.dim * 4

    def forward(self, x, out, rows=None):
        if self.groups > 1:
            ops.group_rmsnorm(x, self.weight, out, self.eps, self.groups, rows)
        else:
            ops.rmsnorm(x, self.weight, out, self.eps, rows)

    def scale_result(self, factor):
        self.weight = self.weight * factor
        return True

    def shareable(self):
        return (self.weight, self.eps) if self.groups == 1 else None

    def as_stream_norm(self):
        return (self.weight, None, self.eps, True) if self.groups == 1 else None


class LayerNorm(RMSNorm):
    """y = (x - mean(x)) / sqrt(var(x) + eps) * w (+ b), in float (var: mean of squared deviations)."""

    kind = "layernorm"

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.bias_name = self.name + spec.bias_suffix if getattr(spec, "bias", False) else None
        self.bias = None

    def param_specs(self):
        p = super().param_specs()
        if self.bias_name:
            p[self.bias_name] = ParamSpec((self.dim,), role="vector", init="zeros_noise")
        return p

    def load(self, tensors):
        super().load(tensors)
        if self.bias_name:
            self.bias = tensors[self.bias_name].contiguous()

    def weight_bytes(self):
        return self.dim * (8 if self.bias_name else 4)

    def forward(self, x, out, rows=None):
        ops.layernorm(x, self.weight, out, self.eps, rows, bias=self.bias)

    def scale_result(self, factor):
        super().scale_result(factor)
        if self.bias is not None:
            self.bias = self.bias * factor
        return True

    def shareable(self):
        return None         # the products' shared norm is the RMS form only

    def as_stream_norm(self):
        return self.weight, self.bias, self.eps, False


class DynamicTanh(Norm):
    """y = tanh(alpha * x) * w + b, channel by channel; alpha is one number, read from its tensor when it is loaded."""

    def __init__(self, spec, rt):
        self.dim, self.rt = spec.dim, rt
        self.name, self.bias_name, self.alpha_name = spec.weight_name, spec.weight_name + spec.bias_suffix, spec.weight_name + spec.alpha_suffix
        self.alpha = self.weight = self.bias = None

    def param_specs(self):
        return {self.name: ParamSpec((self.dim,), role="vector", init="ones_noise"),
                self.bias_name: ParamSpec((self.dim,), role="vector", init="zeros_noise"),
                self.alpha_name: ParamSpec((), role="vector", init="ones_noise")}

    def load(self, tensors):
        self.alpha = float(tensors[self.alpha_name])
        self.weight, self.bias = tensors[self.name].contiguous(), tensors[self.bias_name].contiguous()

    def weight_bytes(self):
        return self.dim * 8

    def forward(self, x, out, rows=None):
        ops.residual_tanh(x, [(self.as_pointwise(), out)], rows=rows)

    def scale_result(self, factor):
        self.weight, self.bias = self.weight * factor, self.bias * factor
        return True

    def as_pointwise(self):
        return self.alpha, self.weight, self.bias


register_part("norm", "dynamic_tanh", DynamicTanh)
register_part("norm", "rmsnorm", RMSNorm)
register_part("norm", "layernorm", LayerNorm)
