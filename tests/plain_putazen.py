"""A plain, slow implementation of the Putazen decoder: whole sequences, no cache, no batching, one
function per mechanism, written from the design's equations.  It shares no code with the library: it
parses config.json and the safetensors file itself and computes with torch on the CPU.

The design in this file's notation (T tokens, D = width; positions count from 0 in a sequence):

  X_s[t] = c_e E[tok_t] for every one of n streams s
  one sublayer q of a layer (q = 1 the mixer, q = 2 the feed-forward, which a layer may lack):
      u = sum_s a_s X_s;   y = F( LN(u) );   X_t <- sum_s M[s][t] X_s + b_t y      (all streams from the old ones)
  LN(u) = (u - mean u) / sqrt(mean (u - mean u)^2 + eps) * w + b
  logits = head LN( sum_s X_s )

Order: the layers in the list's order, except that those of a range run several times in a row with the
same weights.  Mixers: "attention" (two attention maps per head over the same values, subtracted),
"latent_attention" (keys and values are products of one small vector per token) and "mamba2" (a state
matrix per head with one decay and one step size per token and head).

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

GLU_SLOPE = 1.702


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


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(u, w, b):
    """y_t = b + sum_j w[:, j] * u_{t - taps + 1 + j}; u [T, C], w [C, taps]; the last column weighs u_t itself."""
    T, C = u.shape
    taps = w.shape[1]
    y = b.expand(T, C).clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


# ---- hyper-connections ------------------------------------------------------------------------
def stream_in(X, a):
    """X [n, T, D], a [n] -> u [T, D]."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + a[s] * X[s]
    return u


def stream_out(X, y, M, b):
    """new X_t = sum_s M[s][t] X_s + b_t y."""
    n = X.shape[0]
    new = []
    for t in range(n):
        z = b[t] * y
        for s in range(n):
            z = z + M[s, t] * X[s]
        new.append(z)
    return torch.stack(new)


# ---- rotation ---------------------------------------------------------------------------------
def frequencies(dims: int, base: float, scaling=None):
    """([f_i], m): f_i = base^(-2i/dims), i < dims/2; with `scaling` (factor, original, fast, slow) they are stretched
    from band to band, and cos and sin are to be multiplied by m."""
    fs = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return fs, 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))
    lo = max(math.floor(place(float(scaling["fast"]))), 0)
    hi = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(fs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, freqs, mscale, dims, interleaved):
    """x [..., T at axis 0, ..., dim]: pairs (i, i + dims/2), or (2i, 2i + 1), of the first `dims` channels."""
    if dims == 0:
        return x
    ang = torch.tensor(positions, dtype=x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :]
    shape = [len(positions)] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = (torch.cos(ang) * mscale).reshape(shape), (torch.sin(ang) * mscale).reshape(shape)
    out = x.clone()
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        out[..., :dims // 2], out[..., dims // 2:dims] = u * c - v * s, v * c + u * s
    return out


# ---- attention --------------------------------------------------------------------------------
def softmax_attention(q, k, v, scale):
    """q, k [T, dk], v [T, dv] of one head: query i over the keys 0 .. i."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def difference_factor(lq1, lk1, lq2, lk2, diff):
    return float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + diff


def combine_maps(a1, a2, lam, diff, eps):
    """a1 - lam a2, each head's dv channels divided by their root mean square, times 1 - diff."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, W, p, m, positions, eps, dtype, store):
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]

    def proj(n):
        return h @ W[p + n].to(dtype).T + W[p + n + ".b"].to(dtype)
    q, k, v = proj("q").reshape(T, H, 2, dk), proj("k").reshape(T, G, 2, dk), store(proj("v")).reshape(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        fs, ms = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q = rotate(q, positions, fs, ms, rot["dims"], False)
        k = rotate(k, positions, fs, ms, rot["dims"], False)
    q, k = store(q), store(k)
    lam = difference_factor(*(W[p + n].to(dtype) for n in ("lq1", "lk1", "lq2", "lk2")), float(m["diff"]))
    out = torch.zeros(T, H, dv, dtype=dtype)
    for hh in range(H):
        g = hh // (H // G)
        a1 = softmax_attention(q[:, hh, 0], k[:, g, 0], v[:, g], float(m["scale"]))
        a2 = softmax_attention(q[:, hh, 1], k[:, g, 1], v[:, g], float(m["scale"]))
        out[:, hh] = combine_maps(a1, a2, lam, float(m["diff"]), eps)
    return store(out.reshape(T, H * dv)) @ W[p + "o"].to(dtype).T


def latent_mixer(h, W, p, m, positions, eps, dtype, store):
    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (h @ W[p + "q"].to(dtype).T).reshape(T, H, dn + dr)
    kv = h @ W[p + "dkv"].to(dtype).T
    c = store(unit_rms(kv[:, :rk], eps) * W[p + "dkv.norm"].to(dtype))
    r = kv[:, rk:]
    qn, qr = q[..., :dn], q[..., dn:]
    if dr:
        fs, ms = frequencies(dr, m["rot"]["base"])
        r = rotate(r, positions, fs, ms, dr, True)
        qr = rotate(qr, positions, fs, ms, dr, True)
    r = store(r)
    out = torch.zeros(T, H, dv, dtype=dtype)
    for hh in range(H):
        k = c @ W[p + "uk"].to(dtype)[hh * dn:(hh + 1) * dn].T
        v = c @ W[p + "uv"].to(dtype)[hh * dv:(hh + 1) * dv].T
        out[:, hh] = softmax_attention(torch.cat([qn[:, hh], qr[:, hh]], -1), torch.cat([k, r], -1), v, float(m["scale"]))
    return store(out.reshape(T, H * dv)) @ W[p + "o"].to(dtype).T


# ---- the state-space mixer ----------------------------------------------------------------------
def state_space_scan(x, B, C, dt, A, D, S=None):
    """x [T, H, v], B, C [T, G, N], dt [T, H], A [H] (> 0), D [H]; head h reads group h / (H / G).
    S_t = exp(-A dt_t) S_{t-1} + dt_t B_t x_t^T;  y_t = S_t^T C_t + D x_t.  Returns y [T, H, v], S [H, N, v]."""
    T, H, nv = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, nv, dtype=x.dtype) if S is None else S.clone()
    y = torch.zeros_like(x)
    grp = torch.tensor([h // (H // G) for h in range(H)])
    for t in range(T):
        S = torch.exp(-A * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t][grp])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, C[t][grp]) + D[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, w, parts, eps):
    """(y * silu(z)), in `parts` equal runs each divided by its own root mean square, times w."""
    T, n = y.shape
    g = (y * silu(z)).reshape(T, parts, n // parts)
    return unit_rms(g, eps).reshape(T, n) * w


def mamba2_mixer(h, W, p, m, eps, dtype, store):
    H, dv, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    T, inner = h.shape[0], H * dv
    proj = h @ W[p + "in"].to(dtype).T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    assert W[p + "conv"].shape[1] == taps
    xbc = silu(causal_conv(xbc, W[p + "conv"].to(dtype), W[p + "conv.b"].to(dtype)))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    dt = softplus(dt + W[p + "dt_bias"].to(dtype))
    y, _ = state_space_scan(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), dt,
                            torch.exp(W[p + "A_log"].to(dtype)), W[p + "D"].to(dtype))
    y = gated_group_norm(y.reshape(T, inner), z, W[p + "norm"].to(dtype), m["norm_groups"], eps)
    return store(y) @ W[p + "o"].to(dtype).T


# ---- feed-forward -------------------------------------------------------------------------------
def clamped_glu(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * sigmoid(GLU_SLOPE * g) * (u + 1.0)


def dense_ff(h, W, p, f, dtype, store):
    y = clamped_glu(h @ W[p + "gate"].to(dtype).T, h @ W[p + "up"].to(dtype).T, float(f["limit"]))
    return store(y) @ W[p + "down"].to(dtype).T


# ---- the model ----------------------------------------------------------------------------------
def order_of_layers(n, loop):
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


class PlainPutazen:
    def __init__(self, folder: str = None, config: dict = None, tensors: dict = None):
        if folder is not None:
            with open(os.path.join(folder, "config.json")) as f:
                config = json.load(f)
            tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
        self.cfg = config
        self.W = {k: v.float() for k, v in tensors.items()}

    def sublayer(self, X, i, q, fn, dtype, store):
        W, p, eps = self.W, f"l{i}.", float(self.cfg["norm"]["eps"])
        a, b, M = (W[f"{p}hc{q}.{n}"].to(dtype) for n in ("in", "out", "mix"))
        h = store(layer_norm(stream_in(X, a), W[f"{p}norm{q}"].to(dtype), W[f"{p}norm{q}.b"].to(dtype), eps))
        return stream_out(X, fn(h), M, b)

    def layer(self, i, X, positions, dtype, store):
        W, L, eps = self.W, self.cfg["layers"][i], float(self.cfg["norm"]["eps"])
        p, m = f"l{i}.mix.", L["mixer"]
        run = {"attention": lambda h: attention_mixer(h, W, p, m, positions, eps, dtype, store),
               "latent_attention": lambda h: latent_mixer(h, W, p, m, positions, eps, dtype, store),
               "mamba2": lambda h: mamba2_mixer(h, W, p, m, eps, dtype, store)}[L["type"]]
        X = self.sublayer(X, i, 1, run, dtype, store)
        if L.get("mlp"):
            X = self.sublayer(X, i, 2, lambda h: dense_ff(h, W, f"l{i}.mlp.", L["mlp"], dtype, store), dtype, store)
        return X

    def hidden(self, tokens: Sequence[int], dtype=torch.float64, store=None):
        """The sum of the streams after every layer run, and the last one."""
        store = store or _keep
        c = self.cfg
        positions = list(range(len(tokens)))
        x = self.W["embed"].to(dtype)[torch.tensor([int(t) for t in tokens])] * float((c.get("embedding") or {}).get("scale", 1.0))
        X = torch.stack([x] * int(c["streams"]))
        runs = []
        for i in order_of_layers(len(c["layers"]), c.get("loop")):
            X = self.layer(i, X, positions, dtype, store)
            runs.append(X.sum(0))
        return runs, X.sum(0)

    def layers(self, tokens: Sequence[int], dtype=torch.float64):
        return self.hidden(tokens, dtype)[0]

    def logits(self, tokens: Sequence[int], dtype=torch.float64, store=None):
        store = store or _keep
        _, x = self.hidden(tokens, dtype, store)
        h = store(layer_norm(x, self.W["final.norm"].to(dtype), self.W["final.norm.b"].to(dtype), float(self.cfg["norm"]["eps"])))
        return h @ self.W["head"].to(dtype).T
