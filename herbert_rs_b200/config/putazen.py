"""The Putazen decoder's configuration: a list of layers with one of three mixers and a dense feed-forward or none, of
which a run of neighbours may be executed several times, over a residual of several copies.

config.json of this design is nested:

    architecture: "Putazen"      vocab, width      embedding.scale      norm.eps      streams
    loop: {start, stop, times} (optional)
    layers: [{type, mixer: {...}, mlp: {kind: "dense", ff, limit} or null}, ...]
      type "attention":         mixer has heads, kv_heads, dim, vdim, scale, diff, rot.{base, dims, scaling.{factor, original, fast,
                                slow} (optional)} (optional)
      type "latent_attention":  mixer has heads, dim (unrotated), rot_dim (rotated), vdim, kv_rank, scale, rot.{base, dims}
      type "mamba2":            mixer has heads, vdim, state, groups, conv (taps), norm_groups

Tensor names: embed, head, final.norm, final.norm.b, and per layer
l<i>.{norm1, norm1.b, norm2, norm2.b, hc1.{in, out, mix}, hc2.{in, out, mix}, mix.*, mlp.*}.

What the design fixes stands here as constants: the attention's rotation pairs channel i with i + dims/2, the latent
attention's neighbouring channels; the feed-forward's activation.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional

from ..errors import ConfigError
from .base import Reader
from .kebisun import NO_POSITION_LIMIT, _sub
from .specs import (AttentionSpec, BlockSpec, LatentAttentionSpec, Mamba2Spec, ModelSpec, NormSpec, RotaryPairsSpec, ScaledRotarySpec,
                    SwiGLUSpec, looped_schedule)

LATENT_PAIR_LAYOUT = "interleaved"
FF_ACTIVATION = "swish_clamp"


@dataclass
class PutazenConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    streams: int
    loop: Optional[tuple]    # (start, stop, times) or None
    layers: tuple            # of (mixer spec, feed-forward spec or None)
    source: dict             # the config.json it was read from

    @classmethod
    def from_dict(cls, c: dict) -> "PutazenConfig":
        r = Reader(c)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        emb = _sub(r, "embedding", required=False)
        scale = emb.number("scale", 1.0) if emb is not None else 1.0
        eps = _sub(r, "norm").number("eps")
        if not eps > 0.0:
            raise ConfigError("norm.eps must be > 0")
        streams = r.integer("streams", minimum=1)
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw_layers):
            lr = Reader(entry, f"layers[{i}]")
            kind = lr.string("type")
            m = _sub(lr, "mixer")
            if kind == "attention":
                mixer = cls._attention(m, width, eps)
            elif kind == "latent_attention":
                mixer = cls._latent(m, width, eps)
            elif kind == "mamba2":
                mixer = cls._mamba2(m, width, eps)
            else:
                raise ConfigError(f"layers[{i}]: unknown layer type {kind!r} (attention, latent_attention, mamba2)")
            f = _sub(lr, "mlp", required=False)
            layers.append((mixer, cls._ff(f, width) if f is not None else None))
        loop = None
        lp = _sub(r, "loop", required=False)
        if lp is not None:
            loop = (lp.integer("start", minimum=0), lp.integer("stop", minimum=0), lp.integer("times", minimum=1))
            if not loop[0] <= loop[1] <= len(layers):
                raise ConfigError(f"loop: layers {loop[0]} .. {loop[1]} are not a range of the {len(layers)} layers")
        return cls(vocab, width, float(scale), float(eps), streams, loop, tuple(layers), copy.deepcopy(c))

    @staticmethod
    def _attention(m: Reader, width: int, eps: float) -> AttentionSpec:
        heads, kv = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
        if heads % kv:
            raise ConfigError(f"{m.where}: heads ({heads}) must be a multiple of kv_heads ({kv})")
        dim, vdim = m.integer("dim", minimum=1), m.integer("vdim", minimum=1)
        position = None
        rot = _sub(m, "rot", required=False)
        if rot is not None:
            dims = rot.integer("dims", minimum=0)
            if dims % 2 or dims > dim:
                raise ConfigError(f"{m.where}: rot.dims ({dims}) must be even and at most dim ({dim})")
            sc = _sub(rot, "scaling", required=False)
            if dims and sc is None:
                position = ScaledRotarySpec(dims, rot.number("base"))
            elif dims:
                position = ScaledRotarySpec(dims, rot.number("base"), sc.number("factor"), sc.number("original"), sc.number("fast"),
                                            sc.number("slow"))
        return AttentionSpec(
            hidden_size=width, num_heads=heads, num_kv_heads=kv, head_dim=dim, scale=m.number("scale"), position=position, bias=True,
            bias_suffix=".b", names=("q", "k", "v", "o", "sink"), value_dim=vdim, difference=m.number("diff"), difference_eps=float(eps),
            difference_names=("lq1", "lk1", "lq2", "lk2"))

    @staticmethod
    def _latent(m: Reader, width: int, eps: float) -> LatentAttentionSpec:
        rope_dim = m.integer("rot_dim", minimum=0)
        position = None
        if rope_dim > 0:
            rot = _sub(m, "rot")
            dims = rot.integer("dims", minimum=2)
            if dims != rope_dim or dims % 2:
                raise ConfigError(f"{m.where}: rot.dims ({dims}) must be even and equal rot_dim ({rope_dim})")
            position = RotaryPairsSpec(dims, rot.number("base"), 1.0, LATENT_PAIR_LAYOUT)
        return LatentAttentionSpec(
            hidden_size=width, num_heads=m.integer("heads", minimum=1), nope_dim=m.integer("dim", minimum=1), rope_dim=rope_dim,
            v_dim=m.integer("vdim", minimum=1), kv_rank=m.integer("kv_rank", minimum=1), scale=m.number("scale"), norm_eps=float(eps),
            position=position, names=(("q_up", "q"),))

    @staticmethod
    def _mamba2(m: Reader, width: int, eps: float) -> Mamba2Spec:
        heads, vdim, groups = m.integer("heads", minimum=1), m.integer("vdim", minimum=1), m.integer("groups", minimum=1)
        parts = m.integer("norm_groups", minimum=1)
        if heads % groups:
            raise ConfigError(f"{m.where}: heads ({heads}) must be a multiple of groups ({groups})")
        if heads * vdim % parts:
            raise ConfigError(f"{m.where}: norm_groups ({parts}) must divide heads * vdim ({heads * vdim})")
        return Mamba2Spec(hidden_size=width, num_heads=heads, value_dim=vdim, state_dim=m.integer("state", minimum=1), groups=groups,
                          conv_taps=m.integer("conv", minimum=1), norm_groups=parts, norm_eps=float(eps))

    @staticmethod
    def _ff(f: Reader, width: int) -> SwiGLUSpec:
        kind = f.string("kind")
        if kind != "dense":
            raise ConfigError(f"{f.where}: unknown feed-forward kind {kind!r} (dense)")
        limit = f.number("limit")
        if not limit > 0.0:
            raise ConfigError(f"{f.where}: limit must be > 0")
        return SwiGLUSpec(width, f.integer("ff", minimum=1), activation=FF_ACTIVATION, names=("gate", "up", "down"), act_limit=float(limit))

    def to_dict(self) -> dict:
        return copy.deepcopy(self.source)

    def model_spec(self) -> ModelSpec:
        def norm(name):
            return NormSpec(self.width, self.norm_eps, kind="layernorm", weight_name=name, bias=True, bias_suffix=".b")
        blocks = [BlockSpec(mixer=mixer, ffn=ff, norm1=norm("norm1"), norm2=norm("norm2"), kind="streams", streams=self.streams,
                            stream_names=("hc{q}.in", "hc{q}.out", "hc{q}.mix"),
                            names=(("norm1", ""), ("mixer", "mix"), ("norm2", ""), ("ffn", "mlp")))
                  for mixer, ff in self.layers]
        start, stop, times = self.loop if self.loop is not None else (0, 0, 1)
        return ModelSpec(
            architecture="Putazen", vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks),
            schedule=looped_schedule(len(blocks), start, stop, times), final_norm=norm("norm"), tie_word_embeddings=False,
            max_position=NO_POSITION_LIMIT, stop_token_ids=(), layer_prefix="l{i}.", embed_name="embed", final_norm_name="final.norm",
            head_name="head", embedding_scale=self.embedding_scale, streams=self.streams)
