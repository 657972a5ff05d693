"""A plain, slow implementation of the Muzasun decoder: whole sequences, no cache, no batching, one
function per mechanism, written from the design's equations.  It shares no code with the library: it
parses config.json and the safetensors file itself and computes with torch on the CPU.

The design in this file's notation (T tokens, D = width; positions count from 0 in a sequence):

  x[t] = E[tok_t];   per layer   x <- x + mu ( M(N1(x)) + F(N2(x)) )      M the mixer, F the feed-forward (a layer may lack it)
  N(x) = tanh(a x) * w + b       a: one number per norm
  logits = c head N(x)

Mixers: "attention" (grouped heads with biases, a norm per head on q and k, half-split rotation, values that every
layer but the first blends with the first one's), "mlstm" (a matrix memory with an input and a forget gate per head,
kept in range by a running maximum) and "channel_delta" (the delta rule with a decay per key channel).
Feed-forwards: dense, or a mixture of experts in which a token's weight multiplies an expert's input.

`dtype` is the dtype of all arithmetic (float64 for a ground truth).  Weights are used as stored
(bfloat16 values widened exactly).  `store`, where given, is applied to every activation that an engine
would keep in its activation dtype between two kernels (`bf16_storage` rounds those to bfloat16): what
the number format alone does to the logits follows from it.
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, Sequence

import numpy as np
import torch

UNIT_EPS = 1e-6
READ_EPS = 1e-6


# ---- reading a model folder ---------------------------------------------------------------------
def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        raw = f.read()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        if info["dtype"] == "BF16":
            u = np.frombuffer(data[b:e], dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(u.view(np.float32).copy())
        elif info["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(data[b:e], dtype="<f4").copy())
        else:
            raise ValueError(f"dtype {info['dtype']} of {name}")
        out[name] = t.reshape(info["shape"])
    return out


def bf16_storage(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


def _keep(t):
    return t


# ---- small functions --------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    """ln(1 + e^z), without overflow."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def squash_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def causal_conv(u, w):
    """y_t = sum_j w[:, j] * u_{t - taps + 1 + j}; u [T, C], w [C, taps]; the last column weighs u_t itself."""
    T, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


# ---- attention --------------------------------------------------------------------------------
def rotate(x, positions, base, dims):
    """x [T, heads, dim]: channels (i, i + dims/2) of the first `dims` turn by p * base^(-2i/dims)."""
    if dims == 0:
        return x
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.tensor([float(p) for p in positions], dtype=x.dtype) * (float(base) ** (-2.0 * i / dims))
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i], out[..., i + half] = u * c - v * s, v * c + u * s
    return out


def softmax_attention(q, k, v, scale):
    """q, k [T, dk], v [T, dv] of one head: query i over the keys 0 .. i."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def blend_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention_mixer(h, W, p, m, positions, eps, first, dtype, store):
    """Returns the mixer's result and the layer's own values before any blending; `first`: the values to blend with, or None."""
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]

    def proj(n):
        return h @ W[p + n].to(dtype).T + W[p + n + ".b"].to(dtype)
    q, k, own = proj("q").reshape(T, H, dk), proj("k").reshape(T, G, dk), proj("v")
    q = unit_rms(q, eps) * W[p + "q.norm"].to(dtype)
    k = unit_rms(k, eps) * W[p + "k.norm"].to(dtype)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = rotate(q, positions, rot["base"], rot["dims"]), rotate(k, positions, rot["base"], rot["dims"])
    v = own if first is None else blend_values(own, first, W[p + "vmix"].to(dtype))
    q, k, v = store(q), store(k), store(v).reshape(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=dtype)
    for hh in range(H):
        g = hh // (H // G)
        out[:, hh] = softmax_attention(q[:, hh], k[:, g], v[:, g], float(m["scale"]))
    return store(out.reshape(T, H * dv)) @ W[p + "o"].to(dtype).T + W[p + "o.b"].to(dtype), own


# ---- the matrix memory --------------------------------------------------------------------------
def capped(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return -softplus(-z)


def matrix_memory(q, k, v, i, f, S=None, n=None, m=None):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H].  Returns the read-outs [T, H, e] and the state (S, n, m)."""
    T, H, d = q.shape
    e = v.shape[2]
    S = torch.zeros(H, d, e, dtype=q.dtype) if S is None else S.clone()
    n = torch.zeros(H, d, dtype=q.dtype) if n is None else n.clone()
    m = torch.zeros(H, dtype=q.dtype) if m is None else m.clone()
    out = torch.zeros(T, H, e, dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * (k[t][:, :, None] * v[t][:, None, :])
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        bottom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + READ_EPS
        out[t] = torch.einsum("hde,hd->he", S, q[t]) / bottom[:, None]
    return out, (S, n, m)


def mlstm_mixer(h, W, p, m, eps, dtype, store):
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    T = h.shape[0]

    def proj(n):
        return h @ W[p + n].to(dtype).T
    q, k, v = store(proj("q")).reshape(T, H, d) * d ** -0.5, store(proj("k")).reshape(T, H, d), store(proj("v")).reshape(T, H, e)
    i = capped(proj("i") + W[p + "i.b"].to(dtype), cap)
    f = log_sigmoid(capped(proj("f") + W[p + "f.b"].to(dtype), cap))
    o, _ = matrix_memory(q, k, v, i, f)
    y = unit_rms(o, eps).reshape(T, H * e) * W[p + "norm"].to(dtype) * sigmoid(proj("g"))
    return store(y) @ W[p + "o"].to(dtype).T


# ---- the delta rule with a decay per channel ------------------------------------------------------
def channel_delta(q, k, v, g, beta, S=None):
    """q, k, g [T, H, d], v [T, H, e], beta [T, H].  Returns o [T, H, e] and S [H, d, e]."""
    T, H, d = q.shape
    e = v.shape[2]
    S = torch.zeros(H, d, e, dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, e, dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out, S


def channel_decay(low, up, A_log, bias, H):
    """exp(-exp(A_log_h) softplus(up low + bias)) [T, H, d]."""
    z = softplus(low @ up.T + bias)
    return torch.exp(-torch.exp(A_log)[:, None] * z.reshape(z.shape[0], H, -1))


def channel_delta_mixer(h, W, p, m, eps, dtype, store):
    H, G, d, e, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    T = h.shape[0]

    def w(n):
        return W[p + n].to(dtype)

    def proj(n):
        return h @ w(n).T
    assert w("q.conv").shape[1] == taps
    q, k, v = (silu(causal_conv(proj(n), w(n + ".conv"))) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, d)) * d ** -0.5
    k = unit_vector(k.reshape(T, G, d))
    grp = [hh // (H // G) for hh in range(H)]
    beta = sigmoid(proj("b"))
    g = channel_decay(proj("a1"), w("a2"), w("A_log"), w("dt_bias"), H)
    o, _ = channel_delta(q[:, grp], k[:, grp], v.reshape(T, H, e), g, beta)
    gate = sigmoid(store(proj("g1")) @ w("g2").T).reshape(T, H, e)
    y = unit_rms(o, eps) * w("norm") * gate
    return store(y.reshape(T, H * e)) @ w("o").T


# ---- feed-forwards ------------------------------------------------------------------------------
def glu_ff(h, W, p, dtype, store):
    return store(silu(h @ W[p + "gate"].to(dtype).T) * (h @ W[p + "up"].to(dtype).T)) @ W[p + "down"].to(dtype).T


def choose(z, top):
    """Scores sigmoid(z) [T, E]; per token the `top` best experts (a tie goes to the lower index) and their scores."""
    s = sigmoid(z)
    idx = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return idx, torch.gather(s, 1, idx)


def mixture_ff(h, W, p, f, dtype, store):
    idx, wts = choose(h @ W[p + "router"].to(dtype).T, f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        rows, place = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += glu_ff(wts[rows, place][:, None] * h[rows], W, f"{p}e{e}.", dtype, store)
    if f.get("shared"):
        out = out + glu_ff(h, W, p + "shared.", dtype, store)
    return out


# ---- the model ----------------------------------------------------------------------------------
class PlainMuzasun:
    def __init__(self, folder: str = None, config: dict = None, tensors: dict = None):
        if folder is not None:
            with open(os.path.join(folder, "config.json")) as f:
                config = json.load(f)
            tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
        self.cfg = config
        self.W = {k: v.float() for k, v in tensors.items()}

    def norm(self, name, x, dtype):
        return squash_norm(x, self.W[name + ".alpha"].to(dtype), self.W[name].to(dtype), self.W[name + ".b"].to(dtype))

    def hidden(self, tokens: Sequence[int], dtype=torch.float64, store=None):
        """The stream after every layer, and the last one."""
        store = store or _keep
        c, W = self.cfg, self.W
        eps, mu = float(c["norm"]["eps"]), float(c["residual_mult"])
        positions = list(range(len(tokens)))
        x = W["embed"].to(dtype)[torch.tensor([int(t) for t in tokens])]
        first, runs = None, []
        for i, L in enumerate(c["layers"]):
            p, m = f"l{i}.mix.", L["mixer"]
            h = store(self.norm(f"l{i}.norm1", x, dtype))
            if L["type"] == "attention":
                mixing = bool(m.get("v_mix"))
                y, own = attention_mixer(h, W, p, m, positions, eps, first if mixing else None, dtype, store)
                if mixing and first is None:
                    first = own
            elif L["type"] == "mlstm":
                y = mlstm_mixer(h, W, p, m, eps, dtype, store)
            else:
                y = channel_delta_mixer(h, W, p, m, eps, dtype, store)
            f = L.get("mlp")
            if f:
                h2 = store(self.norm(f"l{i}.norm2", x, dtype))
                y = y + (glu_ff(h2, W, f"l{i}.mlp.", dtype, store) if f["kind"] == "dense"
                         else mixture_ff(h2, W, f"l{i}.mlp.", f, dtype, store))
            x = x + mu * y
            runs.append(x)
        return runs, x

    def layers(self, tokens: Sequence[int], dtype=torch.float64):
        return self.hidden(tokens, dtype)[0]

    def logits(self, tokens: Sequence[int], dtype=torch.float64, store=None):
        store = store or _keep
        _, x = self.hidden(tokens, dtype, store)
        return store(self.norm("final.norm", x, dtype)) @ self.W["head"].to(dtype).T * float(self.cfg["logit_scale"])
