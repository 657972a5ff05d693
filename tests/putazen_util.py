"""Small Putazen configurations and weights for tests.  Nothing here is shared with the library's compute path: tensors
are drawn with torch's generator and written with the container writer.

Weights: matrices N(0, gain^2 / in), norm weights around 1, biases 0.2-0.5 N, convolution taps 0.5 N, step sizes
softplus(N(-1, 1)), decay rates exp(A_log) between 0.3 and 4.  The streams' matrices lie around 0.8 on the diagonal with
noise beside it, so that the copies differ from one another after the first sublayer and the residual stays of one size.
"""
from __future__ import annotations

import copy
import json
import math
import os

import torch

from herbert_rs_b200.weights.safetensors_io import save_file


def attention(heads=4, kv_heads=2, dim=16, vdim=32, rot_dims=None, base=10000.0, scaling="default", scale=None, sharp=1.0, diff=0.4):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": sharp / math.sqrt(dim) if scale is None else scale,
         "diff": diff}
    dims = dim if rot_dims is None else rot_dims
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if scaling == "default":
            scaling = {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 0.5}
        if scaling:
            m["rot"]["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": m}


def latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=32, base=5000.0, sharp=1.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": sharp / math.sqrt(dim + rot_dim)}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
    return {"type": "latent_attention", "mixer": m}


def mamba(heads=4, vdim=16, state=24, groups=2, norm_groups=2, conv=3):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": conv}}


def dense(ff=80, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(layers, vocab=131, width=64, eps=1e-5, streams=3, loop=None, scale=2.0):
    """layers: list of (mixer entry, mlp entry or None); loop: (start, stop, times) or None."""
    c = {"architecture": "Putazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "streams": streams, "layers": [copy.deepcopy(dict(m, mlp=f)) for m, f in layers]}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    D, V, n = cfg["width"], cfg["vocab"], cfg["streams"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def vec(k, mean=0.0, std=0.2):
        return mean + std * torch.randn(k, generator=g)

    w = {"embed": torch.randn(V, D, generator=g), "head": mat(V, D, 2.0), "final.norm": vec(D, 1.0), "final.norm.b": vec(D, 0.0, 0.3)}
    for i, l in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", l["mixer"], f"l{i}.mix."
        for s in (1, 2) if l.get("mlp") else (1,):
            w[f"{p}norm{s}"], w[f"{p}norm{s}.b"] = vec(D, 1.0), vec(D, 0.0, 0.3)
            w[f"{p}hc{s}.in"], w[f"{p}hc{s}.out"] = vec(n, 1.0 / n, 0.25), vec(n, 1.0, 0.4)
            w[f"{p}hc{s}.mix"] = 0.8 * torch.eye(n) + 0.15 * torch.randn(n, n, generator=g)
        if l["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({q + "q": mat(H * 2 * dk, D, 1.5), q + "k": mat(G * 2 * dk, D, 1.5), q + "v": mat(G * dv, D), q + "o": mat(D, H * dv)})
            w.update({q + "q.b": vec(H * 2 * dk, 0.0, 0.5), q + "k.b": vec(G * 2 * dk, 0.0, 0.5), q + "v.b": vec(G * dv, 0.0, 0.5)})
            w.update({q + x: vec(dk, 0.0, 1.0 / math.sqrt(dk)) for x in ("lq1", "lk1", "lq2", "lk2")})
        elif l["type"] == "latent_attention":
            H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w.update({q + "q": mat(H * (dn + dr), D, 1.5), q + "dkv": mat(rk + dr, D, 1.2), q + "dkv.norm": vec(rk, 1.0),
                      q + "uk": mat(H * dn, rk), q + "uv": mat(H * dv, rk), q + "o": mat(D, H * dv)})
        else:
            H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            C = H * dv + 2 * G * N
            w.update({q + "in": mat(H * dv + C + H, D, 1.2), q + "conv": torch.randn(C, m["conv"], generator=g) * 0.6, q + "conv.b": vec(C, 0.0, 0.3),
                      q + "dt_bias": vec(H, -1.0, 1.0), q + "A_log": torch.rand(H, generator=g) * 2.6 - 1.2, q + "D": vec(H, 1.0, 0.5),
                      q + "norm": vec(H * dv, 1.0), q + "o": mat(D, H * dv)})
        f = l.get("mlp")
        if f:      # gains that reach both clamps for some channels
            w.update({p + "mlp.gate": mat(f["ff"], D, 2.0), p + "mlp.up": mat(f["ff"], D, 2.0), p + "mlp.down": mat(D, f["ff"])})
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write(cfg, tensors, folder):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16) for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def make(folder, layers, seed=0, edit=None, **kw):
    """Write a model folder; returns (folder, plain model).  edit(tensors) may change the weights first."""
    import plain_putazen as P
    cfg = config(layers, **kw)
    w = weights(cfg, seed)
    if edit is not None:
        edit(w)
    write(cfg, w, folder)
    return str(folder), P.PlainPutazen(str(folder))
