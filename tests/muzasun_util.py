"""Small Muzasun configurations and weights for tests.  Nothing here is shared with the library's compute path: tensors
are drawn with torch's generator and written with the container writer.

Weights: matrices N(0, gain^2 / in), norm weights around 1, biases 0.2-0.5 N, convolution taps 0.5 N.  The norms' alphas lie
between 0.4 and 1.2, so tanh bends without saturating everywhere.  Input gates of the matrix memory are around 0, forget gates
around sigmoid(2); the delta rule's decays between about 0.5 and 0.99.  Where a model has routed experts, no choice is close:
the first channels of the stream, one per expert, hold levels in an order that the token's id chooses, no layer adds to them,
and a router reads mostly them.
"""
from __future__ import annotations

import copy
import json
import math
import os

import torch

from herbert_rs_b200.weights.safetensors_io import save_file


def attention(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=None, base=10000.0, sharp=1.0, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": sharp / math.sqrt(dim), "v_mix": v_mix}
    dims = dim if rot_dims is None else rot_dims
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return {"type": "attention", "mixer": m}


def mlstm(heads=3, dim=16, vdim=20, cap=8.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, rank=10):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "low_rank": rank}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, shared=48):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def config(layers, vocab=131, width=64, eps=1e-5, mult=0.5, logit_scale=1.5):
    """layers: list of (mixer entry, mlp entry or None)."""
    return {"architecture": "Muzasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_scale": logit_scale, "layers": [copy.deepcopy(dict(m, mlp=f)) for m, f in layers]}


def weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def vec(k, mean=0.0, std=0.2):
        return mean + std * torch.randn(k, generator=g)

    def norm(name):
        w[name], w[name + ".b"] = vec(D, 1.0), vec(D, 0.0, 0.3)
        w[name + ".alpha"] = 0.4 + 0.8 * torch.rand((), generator=g)

    def ff(p, n):
        w.update({p + "gate": mat(n, D, 1.5), p + "up": mat(n, D, 1.5), p + "down": mat(D, n, 1.5)})
    w = {"embed": torch.randn(V, D, generator=g) * 1.5, "head": mat(V, D, 2.0)}
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m, q = f"l{i}.", l["mixer"], f"l{i}.mix."
        norm(p + "norm1")
        if l["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({q + "q": mat(H * dk, D), q + "k": mat(G * dk, D), q + "v": mat(G * dv, D), q + "o": mat(D, H * dv, 1.5)})
            w.update({q + "q.b": vec(H * dk, 0.0, 0.5), q + "k.b": vec(G * dk, 0.0, 0.5), q + "v.b": vec(G * dv, 0.0, 0.5), q + "o.b": vec(D, 0.0, 0.5)})
            w.update({q + "q.norm": vec(dk, 1.2, 0.3), q + "k.norm": vec(dk, 1.2, 0.3)})
            if m.get("v_mix"):
                w[q + "vmix"] = 0.35 + 0.3 * torch.rand((), generator=g)
        elif l["type"] == "mlstm":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            w.update({q + "q": mat(H * d, D), q + "k": mat(H * d, D), q + "v": mat(H * e, D), q + "g": mat(H * e, D), q + "o": mat(D, H * e, 1.5),
                      q + "norm": vec(H * e, 1.0), q + "i": mat(H, D, 2.0), q + "f": mat(H, D, 2.0), q + "i.b": vec(H, 0.0, 1.0), q + "f.b": vec(H, 2.0, 1.0)})
        else:
            H, G, d, e, R = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["low_rank"]
            w.update({q + "q": mat(G * d, D), q + "k": mat(G * d, D), q + "v": mat(H * e, D), q + "b": mat(H, D, 1.5), q + "o": mat(D, H * e, 1.5)})
            w.update({q + n + ".conv": torch.randn(c, m["conv"], generator=g) * 0.6 for n, c in (("q", G * d), ("k", G * d), ("v", H * e))})
            w.update({q + "a1": mat(R, D), q + "a2": mat(H * d, R), q + "g1": mat(R + 3, D), q + "g2": mat(H * e, R + 3),
                      q + "A_log": torch.rand(H, generator=g) * 2.0 - 2.0, q + "dt_bias": vec(H * d, -1.5, 1.0), q + "norm": vec(e, 1.0)})
        f = l.get("mlp")
        if f:
            norm(p + "norm2")
            if f["kind"] == "dense":
                ff(p + "mlp.", f["ff"])
            else:
                E = f["router"]["experts"]
                w[p + "mlp.router"] = mat(E, D, 0.05) + 4.0 * torch.eye(E, D)
                w[p + "norm2"][:E], w[p + "norm2.b"][:E], w[p + "norm2.alpha"] = 1.0, 0.0, torch.tensor(0.3)
                for e in range(f["router"]["experts"]):
                    ff(f"{p}mlp.e{e}.", f["expert"]["ff"])
                if f.get("shared"):
                    ff(p + "mlp.shared.", f["shared"]["ff"])
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l.get("mlp") and l["mlp"]["kind"] == "moe"], default=0)
    if E:
        levels = torch.linspace(4.0, -4.0, E) if E > 1 else torch.tensor([1.0])
        for t in range(V):
            w["embed"][t, :E] = levels[torch.randperm(E, generator=g)]
        for k, v in w.items():
            if k.endswith((".mix.o", ".mix.o.b", ".down")):
                v[:E] = 0.0
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write(cfg, tensors, folder):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16) for k, v in tensors.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def make(folder, layers, seed=0, edit=None, **kw):
    """Write a model folder; returns (folder, plain model).  edit(tensors) may change the weights first."""
    import plain_muzasun as P
    cfg = config(layers, **kw)
    w = weights(cfg, seed)
    if edit is not None:
        edit(w)
    write(cfg, w, folder)
    return str(folder), P.PlainMuzasun(str(folder))
