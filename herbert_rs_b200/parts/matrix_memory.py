"""The matrix-memory mixer (mLSTM): a float matrix and a float vector of state per head, with an input and a forget gate per
token and head that are exponentials kept in range by a running maximum.

    q = Wq h * dk^-1/2,  k = Wk h  ([H, dk]),   v = Wv h  ([H, dv])
    i = c tanh((Wi h + bi) / c),   f = log sigmoid(c tanh((Wf h + bf) / c))      logs of the gates, one of each per head
    m_t = max(f + m_(t-1), i)                                                    m starts at 0
    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T;   n_t likewise with k alone;   both start at zero
    o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)
    out = Wo ( concat_h(o_h / rms(o_h)) * w * sigmoid(Wg h) )                    w: one number per head and channel

The values carry a column of ones, so that n is a column of S and n . q a column of S^T q: the recurrence is the state-space
kernels' with a decay and a weight per token and head (`ops.ssd_scan`: token by token, or 64 tokens at a time on the tensor cores
for bfloat16 prompts), and the division opens the norm behind it.  The six products that read h are one matrix (rows q, k, v, g,
i, f) that leaves float sums; gates, running maximum, state, division and norm are float on both paths.  S and m are the
sequence's slot of the cache's fixed-size region.
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache import CacheNeed, StateNeed
from ..errors import ConfigError
from ..registry import register_part
from .base import Mixer, ParamSpec, stack_rows

_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "input": "i", "forget": "f", "input_bias": "i.b", "forget_bias": "f.b",
          "norm": "norm", "out": "o"}
_MAX = "running_max"


class MatrixMemoryMixer(Mixer):
    can_store = True

    def __init__(self, spec, rt):
        self.spec, self.rt = spec, rt
        self.H, self.dk, self.dv = spec.num_heads, spec.key_dim, spec.value_dim
        self.dvp = (self.dv + 1 + 7) // 8 * 8          # a head's values, the column of ones, zeros
        if not spec.gate_cap > 0.0:
            raise ConfigError(f"the cap on the gates must be > 0, got {spec.gate_cap}")
        self.n = dict(_NAMES)
        self.n.update(dict(spec.names))

    def param_specs(self):
        s, n, H, dk, dv = self.spec, self.n, self.H, self.dk, self.dv
        return {
            n["q"]: ParamSpec((H * dk, s.hidden_size)),
            n["k"]: ParamSpec((H * dk, s.hidden_size)),
            n["v"]: ParamSpec((H * dv, s.hidden_size)),
            n["gate"]: ParamSpec((H * dv, s.hidden_size)),
            n["input"]: ParamSpec((H, s.hidden_size)),
            n["forget"]: ParamSpec((H, s.hidden_size)),
            n["input_bias"]: ParamSpec((H,), role="vector", init="wide"),
            n["forget_bias"]: ParamSpec((H,), role="vector", init="wide"),
            n["norm"]: ParamSpec((H * dv,), role="vector", init="ones_noise"),
            n["out"]: ParamSpec((s.hidden_size, H * dv)),
        }

    def load(self, t):
        n = self.n
        self.w_in = stack_rows([t[n[r]] for r in ("q", "k", "v", "gate", "input", "forget")])
        self.i_bias, self.f_bias = t[n["input_bias"]].contiguous(), t[n["forget_bias"]].contiguous()
        self.norm = t[n["norm"]].contiguous()
        self.w_out = t[n["out"]].contiguous()

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_out))

    def cache_need(self):
        return CacheNeed(state=StateNeed((self.H, self.dk, self.dvp), torch.float32), states=((_MAX, StateNeed((self.H,), torch.float32)),))

    def forward(self, h, residual, batch, cache, accumulate=True):
        s, ws, T, H, dk, dv, dvp = self.spec, self.rt.workspace, h.shape[0], self.H, self.dk, self.dv, self.dvp
        f32 = torch.float32
        proj = ws.take((T, self.w_in.shape[0]), f32)
        ops.gemm(h, self.w_in, proj, ops.EPI_STORE_F32, scratch=ws.take)
        k_off, v_off, g_off, i_off = H * dk, 2 * H * dk, 2 * H * dk + H * dv, 2 * H * dk + 2 * H * dv
        packed = ws.take((T, (H * (dvp + 2 * dk) + 7) // 8 * 8), h.dtype)
        logd, weight, floor = (ws.take((T, H), f32) for _ in range(3))
        ops.matrix_memory_prepare(proj, 0, k_off, v_off, i_off, i_off + H, self.i_bias, self.f_bias, s.gate_cap, cache.states[_MAX], batch,
                                  packed, logd, weight, floor, H, dk, dv, dvp)
        o = ws.take((T, H * dvp), f32)
        ops.ssd_scan(packed, H * dvp, H * (dvp + dk), weight, None, None, None, cache.state, batch, o, H, H, dk, dvp, ws.take, logd=logd)
        y = ws.take((T, H * dv), h.dtype)
        ops.gated_rmsnorm(o, self.norm, s.norm_eps, proj[:, g_off:i_off], y, H, dv, sigmoid_gate=True, unit_stride=dvp,
                          divide=(floor, dk ** -0.5, s.read_eps))
        ops.gemm(y, self.w_out, residual, ops.EPI_RESIDUAL if accumulate else ops.EPI_STORE_F32, scratch=ws.take)


register_part("mixer", "matrix_memory", MatrixMemoryMixer)
