"""The Mamba-2 mixer: a state-space recurrence with one decay and one step size per token and head.

    [z | x | B | C | r] = W h                     z, x: H dv;  B, C: G N;  r: H
    [x | B | C] <- silu(conv([x | B | C]) + b)    a short causal convolution over time, channel by channel
    dt = softplus(r + dt_bias);   a = exp(-exp(A_log) dt)                      one of each per token and head
    S <- a S + dt B x^T;   y = S^T C + D x        per head, S is [N, dv]; head h reads group h / (H / G) of B and C
    out = Wo ( N(y * silu(z)) * w )               N: RMS norm in `norm_groups` equal parts of the row, after the gate

The state matrices and the convolution's last taps - 1 inputs are the sequence's slot of the cache's fixed-size region.
The product leaves float rows; the convolution's result is in the activation dtype, everything from the step sizes to
the norm is float.  Long bfloat16 prompts run the recurrence chunk by chunk on the tensor cores (`ops.ssd_scan`).
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache import CacheNeed, StateNeed
from ..errors import ConfigError
from ..registry import register_part
from .base import Mixer, ParamSpec

_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A_log": "A_log", "D": "D", "norm": "norm",
          "out": "o"}


class Mamba2Mixer(Mixer):
    can_store = True

    def __init__(self, spec, rt):
        self.spec, self.rt = spec, rt
        self.H, self.dv, self.N, self.G, self.taps = spec.num_heads, spec.value_dim, spec.state_dim, spec.groups, spec.conv_taps
        self.inner = self.H * self.dv
        if self.H % self.G:
            raise ConfigError(f"{self.H} heads are no multiple of {self.G} groups")
        if self.inner % spec.norm_groups:
            raise ConfigError(f"a norm over {self.inner} channels cannot be cut into {spec.norm_groups} equal parts")
        if self.taps < 1:
            raise ConfigError("a convolution has at least one tap")
        self.conv_channels = self.inner + 2 * self.G * self.N
        self.n = dict(_NAMES)
        self.n.update(dict(spec.names))

    def param_specs(self):
        s, n, H = self.spec, self.n, self.H
        return {
            n["in"]: ParamSpec((self.inner + self.conv_channels + H, s.hidden_size)),
            n["conv"]: ParamSpec((self.conv_channels, self.taps), role="vector", init="wide"),
            n["conv_bias"]: ParamSpec((self.conv_channels,), role="vector", init="zeros_noise"),
            n["dt_bias"]: ParamSpec((H,), role="vector", init="wide"),
            n["A_log"]: ParamSpec((H,), role="vector", init="zeros_noise"),
            n["D"]: ParamSpec((H,), role="vector", init="ones_noise"),
            n["norm"]: ParamSpec((self.inner,), role="vector", init="ones_noise"),
            n["out"]: ParamSpec((s.hidden_size, self.inner)),
        }

    def load(self, t):
        n = self.n
        self.w_in = t[n["in"]].contiguous()
        self.w_conv, self.b_conv = t[n["conv"]].contiguous(), t[n["conv_bias"]].contiguous()
        self.dt_bias, self.a_log, self.d_skip = t[n["dt_bias"]].contiguous(), t[n["A_log"]].contiguous(), t[n["D"]].contiguous()
        self.norm = t[n["norm"]].contiguous()
        self.w_out = t[n["out"]].contiguous()

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_conv, self.w_out))

    def cache_need(self):
        states = ()
        if self.taps > 1:
            states = (("conv", StateNeed((self.taps - 1, self.conv_channels), torch.float32)),)
        return CacheNeed(state=StateNeed((self.H, self.N, self.dv), torch.float32), states=states)

    def forward(self, h, residual, batch, cache, accumulate=True):
        s, ws, T = self.spec, self.rt.workspace, h.shape[0]
        inner, C = self.inner, self.conv_channels
        proj = ws.take((T, inner + C + self.H), torch.float32)
        ops.gemm(h, self.w_in, proj, ops.EPI_STORE_F32, scratch=ws.take)
        xbc = ws.take((T, (C + 7) // 8 * 8), h.dtype)          # rows that start on 16 bytes
        ops.short_conv(proj[:, inner:inner + C], self.w_conv, cache.states.get("conv"), batch, xbc, silu=True, bias=self.b_conv)
        y = ws.take((T, inner), torch.float32)
        ops.ssd_scan(xbc, inner, inner + self.G * self.N, proj[:, inner + C:], self.dt_bias, self.a_log, self.d_skip, cache.state, batch,
                     y, self.H, self.G, self.N, self.dv, ws.take)
        g = ws.take((T, inner), h.dtype)
        ops.gated_rmsnorm(y, self.norm, s.norm_eps, proj[:, :inner], g, s.norm_groups, inner // s.norm_groups, gate_first=True)
        ops.gemm(g, self.w_out, residual, ops.EPI_RESIDUAL if accumulate else ops.EPI_STORE_F32, scratch=ws.take)


register_part("mixer", "mamba2", Mamba2Mixer)
