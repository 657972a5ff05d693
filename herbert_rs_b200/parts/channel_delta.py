"""The delta rule with a decay per key channel: a float matrix of state per head whose rows decay each at a rate of its own,
corrected toward the token's value along its key, and read with the query.

    q, k = silu(conv(Wq h)), silu(conv(Wk h))   ([G, dk], G query/key heads);   v = silu(conv(Wv h))   ([H, dv])
    q <- q / sqrt(sum q^2 + 1e-6) * dk^-1/2,  k <- k / sqrt(sum k^2 + 1e-6)      per head
    beta = sigmoid(Wb h)  one per head;   g = exp(-exp(A_log) * softplus(A2 A1 h + dt_bias))  one per head and key channel
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q           head h reads q/k head h / (H / G)
    out = Wo ( RMSNorm_head(o) * w * sigmoid(G2 G1 h) )                          w: dv numbers for all heads

conv is a short causal convolution over time on each channel whose last taps - 1 inputs are kept per sequence, beside the state
matrix, in the cache's fixed-size region of the sequence's slot.  The six products that read h are one matrix (rows q, k, v, A1, G1,
b) that leaves float sums; unit vectors, beta, decays, the state and the norm are float on both paths.  A2 and G2 are one matrix too,
over the inner rows of both; on the bfloat16 path A1 h enters it as a high and a low part, so that about 16 bits of it reach the
decay.  The recurrence is the generalised delta rule's (`ops.general_delta_scan`), of which this is a case.
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache import CacheNeed, StateNeed
from ..errors import ConfigError, WeightError
from ..registry import register_part
from .base import Mixer, ParamSpec, stack_rows

_NAMES = {"q": "q", "k": "k", "v": "v", "beta": "b", "decay_down": "a1", "decay_up": "a2", "gate_down": "g1", "gate_up": "g2",
          "out": "o", "norm": "norm", "A_log": "A_log", "dt_bias": "dt_bias", "conv_suffix": ".conv"}


class ChannelDeltaMixer(Mixer):
    can_store = True

    def __init__(self, spec, rt):
        self.spec, self.rt = spec, rt
        self.H, self.G, self.dk, self.dv, self.taps = spec.num_heads, spec.qk_heads, spec.key_dim, spec.value_dim, spec.conv_taps
        if self.H % self.G:
            raise ConfigError(f"{self.H} heads are no multiple of {self.G} query/key heads")
        if self.taps < 1:
            raise ConfigError("a convolution has at least one tap")
        self.n = dict(_NAMES)
        self.n.update(dict(spec.names))
        self.conv_channels = 2 * self.G * self.dk + self.H * self.dv

    def param_specs(self):
        s, n, H, G, dk, dv = self.spec, self.n, self.H, self.G, self.dk, self.dv
        c = n["conv_suffix"]
        return {
            n["q"]: ParamSpec((G * dk, s.hidden_size)),
            n["k"]: ParamSpec((G * dk, s.hidden_size)),
            n["v"]: ParamSpec((H * dv, s.hidden_size)),
            n["q"] + c: ParamSpec((G * dk, self.taps), role="vector", init="wide"),
            n["k"] + c: ParamSpec((G * dk, self.taps), role="vector", init="wide"),
            n["v"] + c: ParamSpec((H * dv, self.taps), role="vector", init="wide"),
            n["beta"]: ParamSpec((H, s.hidden_size)),
            n["decay_down"]: ParamSpec((-1, s.hidden_size), free_size=s.low_rank),       # the inner widths are the stored tensors'
            n["decay_up"]: ParamSpec((H * dk, -1), init="wide", free_size=s.low_rank),
            n["gate_down"]: ParamSpec((-1, s.hidden_size), free_size=s.low_rank),
            n["gate_up"]: ParamSpec((H * dv, -1), init="wide", free_size=s.low_rank),
            n["A_log"]: ParamSpec((H,), role="vector", init="zeros_noise"),
            n["dt_bias"]: ParamSpec((H * dk,), role="vector", init="wide"),
            n["norm"]: ParamSpec((dv,), role="vector", init="ones_noise"),
            n["out"]: ParamSpec((s.hidden_size, H * dv)),
        }

    def load(self, t):
        n = self.n
        c = n["conv_suffix"]
        for down, up in (("decay_down", "decay_up"), ("gate_down", "gate_up")):
            if t[n[down]].shape[0] != t[n[up]].shape[1]:
                raise WeightError(f"{n[down]} has {t[n[down]].shape[0]} rows but {n[up]} has {t[n[up]].shape[1]} columns")
        self.rank, self.gate_rank = t[n["decay_down"]].shape[0], t[n["gate_down"]].shape[0]
        self.w_in = stack_rows([t[n[r]] for r in ("q", "k", "v", "decay_down", "gate_down", "beta")])
        self.w_conv = torch.cat([t[n["q"] + c], t[n["k"] + c], t[n["v"] + c]], dim=0).contiguous()
        # [A2 | 0; 0 | G2] over [A1 h | G1 h]; bfloat16: [A2 | A2 | 0; 0 | 0 | G2] over [high | low | G1 h], a multiple of 8 columns
        decay, gate = t[n["decay_up"]], t[n["gate_up"]]
        self.parts = 2 if self.rt.dtype == torch.bfloat16 else 1
        columns = self.parts * self.rank + self.gate_rank
        self.w_low = torch.zeros((decay.shape[0] + gate.shape[0], (columns + 7) // 8 * 8 if self.parts > 1 else columns), dtype=decay.dtype,
                                 device=decay.device)
        for p in range(self.parts):
            self.w_low[:decay.shape[0], p * self.rank:(p + 1) * self.rank] = decay
        self.w_low[decay.shape[0]:, self.parts * self.rank:columns] = gate
        self.a_log, self.dt_bias = t[n["A_log"]].contiguous(), t[n["dt_bias"]].contiguous()
        self.norm = t[n["norm"]].contiguous()
        self.w_out = t[n["out"]].contiguous()

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_conv, self.w_low, self.w_out))

    def cache_need(self):
        states = ()
        if self.taps > 1:
            states = (("conv", StateNeed((self.taps - 1, self.conv_channels), torch.float32)),)
        return CacheNeed(state=StateNeed((self.H, self.dk, self.dv), torch.float32), states=states)

    def forward(self, h, residual, batch, cache, accumulate=True):
        s, ws, T, H, G, dk, dv = self.spec, self.rt.workspace, h.shape[0], self.H, self.G, self.dk, self.dv
        f32 = torch.float32
        proj = ws.take((T, self.w_in.shape[0]), f32)
        ops.gemm(h, self.w_in, proj, ops.EPI_STORE_F32, scratch=ws.take)
        C = self.conv_channels
        v_off, low_off, b_off = 2 * G * dk, C, C + self.rank + self.gate_rank
        qkv = ws.take((T, C), f32)
        ops.short_conv(proj[:, :C], self.w_conv, cache.states.get("conv"), batch, qkv, add_input=False, silu=True)
        low = proj[:, low_off:b_off]
        if self.parts > 1:
            low = ws.take((T, self.w_low.shape[1]), h.dtype)
            ops.operand_parts(proj[:, low_off:b_off], self.rank, self.gate_rank, low)
        wide = ws.take((T, self.w_low.shape[0]), f32)
        ops.gemm(low, self.w_low, wide, ops.EPI_STORE_F32, scratch=ws.take)
        prep = ws.take((T, H, 5, dk), f32)
        ops.channel_delta_prepare(qkv, 0, G * dk, wide[:, :H * dk], proj[:, b_off:b_off + H], self.dt_bias, self.a_log, s.unit_eps,
                                  dk ** -0.5, prep, H, G, dk)
        o = ws.take((T, H * dv), f32)
        ops.general_delta_scan(prep, qkv[:, v_off:], cache.state, batch, o, H, dk, dv)
        y = ws.take((T, H * dv), h.dtype)
        ops.gated_rmsnorm(o, self.norm, s.norm_eps, wide[:, H * dk:], y, H, dv, sigmoid_gate=True)
        ops.gemm(y, self.w_out, residual, ops.EPI_RESIDUAL if accumulate else ops.EPI_STORE_F32, scratch=ws.take)


register_part("mixer", "channel_delta", ChannelDeltaMixer)
