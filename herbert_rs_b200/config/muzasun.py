"""The Muzasun decoder's configuration: a list of layers with one of three mixers and a dense or routed feed-forward (or none),
both sublayers side by side on norms of the same stream.

config.json of this design is nested:

    architecture: "Muzasun"      vocab, width      norm.eps      residual_mult      logit_scale
    layers: [{type, mixer: {...}, mlp: {...} or null}, ...]
      type "attention":      mixer has heads, kv_heads, dim, vdim, scale, v_mix, rot.{base, dims} (optional)
      type "mlstm":          mixer has heads, dim, vdim, gate_cap
      type "channel_delta":  mixer has heads, kv_heads, dim, vdim, conv (taps)
      mlp.kind "dense": ff;   mlp.kind "moe": expert.ff, router.{experts, top}, shared.ff (optional)

Tensor names: embed, head, final.norm, and per layer l<i>.{norm1, norm2, mix.*, mlp.*}; a norm also has <name>.b and <name>.alpha.

What the design fixes stands here as constants: the norm, silu as every feed-forward's activation, sigmoid scores as weights of
the experts' inputs, rotated channels in pairs (i, i + dims/2).
"""

from __future__ import annotations

import copy
from dataclasses import dataclass

from ..errors import ConfigError
from .base import Reader
from .kebisun import NO_POSITION_LIMIT, _sub
from .specs import (AttentionSpec, BlockSpec, ChannelDeltaSpec, MatrixMemorySpec, ModelSpec, NormSpec, RoutedFFSpec, ScaledRotarySpec,
                    SwiGLUSpec, identity_schedule)

NORM_KIND = "dynamic_tanh"
FF_ACTIVATION = "silu"
ROUTER_SCORE = "sigmoid"
VALUE_BLEND_NAME = "vmix"


@dataclass
class MuzasunConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    layers: tuple            # of (mixer spec, feed-forward spec or None)
    source: dict             # the config.json it was read from

    @classmethod
    def from_dict(cls, c: dict) -> "MuzasunConfig":
        r = Reader(c)
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        eps = _sub(r, "norm").number("eps")
        if not eps > 0.0:
            raise ConfigError("norm.eps must be > 0")
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers, kept = [], None          # kept: values per token of the first layer whose values later ones blend in
        for i, entry in enumerate(raw_layers):
            lr = Reader(entry, f"layers[{i}]")
            kind = lr.string("type")
            m = _sub(lr, "mixer")
            if kind == "attention":
                blend = None
                if m.boolean("v_mix", False):
                    values = m.integer("kv_heads", minimum=1) * m.integer("vdim", minimum=1)
                    blend = "keep" if kept is None else "blend"
                    if kept is not None and values != kept:
                        raise ConfigError(f"{m.where}: v_mix blends {values} values a token with the {kept} of the first such layer")
                    kept = values
                mixer = cls._attention(m, width, eps, blend)
            elif kind == "mlstm":
                mixer = cls._matrix_memory(m, width, eps)
            elif kind == "channel_delta":
                mixer = cls._channel_delta(m, width, eps)
            else:
                raise ConfigError(f"layers[{i}]: unknown layer type {kind!r} (attention, mlstm, channel_delta)")
            f = _sub(lr, "mlp", required=False)
            layers.append((mixer, cls._ff(f, width) if f is not None else None))
        return cls(vocab, width, float(eps), float(r.number("residual_mult", 1.0)), float(r.number("logit_scale", 1.0)), tuple(layers),
                   copy.deepcopy(c))

    @staticmethod
    def _attention(m: Reader, width: int, eps: float, blend) -> AttentionSpec:
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
            if dims:
                position = ScaledRotarySpec(dims, rot.number("base"))
        return AttentionSpec(
            hidden_size=width, num_heads=heads, num_kv_heads=kv, head_dim=dim, scale=m.number("scale"), position=position, bias=True,
            bias_suffix=".b", output_bias=True, names=("q", "k", "v", "o", "sink"), value_dim=vdim, head_qk_norm=True,
            qk_norm=NormSpec(dim, float(eps)), norm_names=("q.norm", "k.norm"), value_blend=blend, value_blend_name=VALUE_BLEND_NAME)

    @staticmethod
    def _matrix_memory(m: Reader, width: int, eps: float) -> MatrixMemorySpec:
        cap = m.number("gate_cap")
        if not cap > 0.0:
            raise ConfigError(f"{m.where}: gate_cap must be > 0")
        return MatrixMemorySpec(hidden_size=width, num_heads=m.integer("heads", minimum=1), key_dim=m.integer("dim", minimum=1),
                                value_dim=m.integer("vdim", minimum=1), gate_cap=float(cap), norm_eps=float(eps))

    @staticmethod
    def _channel_delta(m: Reader, width: int, eps: float) -> ChannelDeltaSpec:
        heads, kv = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
        if heads % kv:
            raise ConfigError(f"{m.where}: heads ({heads}) must be a multiple of kv_heads ({kv})")
        # the inner widths of the decay and the gate are the tensors' shapes, not keys of the design; "low_rank" is read
        # only so that a configuration can say which size random weights should get
        return ChannelDeltaSpec(hidden_size=width, num_heads=heads, qk_heads=kv, key_dim=m.integer("dim", minimum=1),
                                value_dim=m.integer("vdim", minimum=1), conv_taps=m.integer("conv", minimum=1), norm_eps=float(eps),
                                low_rank=m.integer("low_rank", 16, minimum=1))

    @staticmethod
    def _ff(f: Reader, width: int):
        kind = f.string("kind")
        if kind == "dense":
            return SwiGLUSpec(width, f.integer("ff", minimum=1), activation=FF_ACTIVATION, names=("gate", "up", "down"))
        if kind == "moe":
            router = _sub(f, "router")
            experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
            if top > experts:
                raise ConfigError(f"{f.where}: router.top ({top}) exceeds router.experts ({experts})")
            sh = _sub(f, "shared", required=False)
            shared = None
            if sh is not None:
                shared = SwiGLUSpec(width, sh.integer("ff", minimum=1), activation=FF_ACTIVATION,
                                    names=("shared.gate", "shared.up", "shared.down"))
            return RoutedFFSpec(width, experts, top, _sub(f, "expert").integer("ff", minimum=1), activation=FF_ACTIVATION,
                                renormalize=False, router_name="router", expert_names=("e{e}.gate", "e{e}.up", "e{e}.down"), gated=True,
                                score=ROUTER_SCORE, shared=shared, weigh_input=True)
        raise ConfigError(f"{f.where}: unknown feed-forward kind {kind!r} (dense, moe)")

    def to_dict(self) -> dict:
        return copy.deepcopy(self.source)

    def model_spec(self) -> ModelSpec:
        def norm(name):
            return NormSpec(self.width, self.norm_eps, kind=NORM_KIND, weight_name=name)
        blocks, unused = [], []
        for i, (mixer, ff) in enumerate(self.layers):
            blocks.append(BlockSpec(mixer=mixer, ffn=ff, norm1=norm("norm1"), norm2=norm("norm2") if ff is not None else None,
                                    kind="parallel", residual_mult=self.residual_mult,
                                    names=(("norm1", ""), ("mixer", "mix"), ("norm2", ""), ("ffn", "mlp"))))
            # what a file may hold although the layer makes no use of it
            if ff is None:
                unused += [f"l{i}.norm2", f"l{i}.norm2.b", f"l{i}.norm2.alpha"]
            if isinstance(mixer, AttentionSpec) and mixer.value_blend is None:
                unused.append(f"l{i}.mix.{VALUE_BLEND_NAME}")
        return ModelSpec(
            architecture="Muzasun", vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks),
            schedule=identity_schedule(len(blocks)), final_norm=norm("norm"), tie_word_embeddings=False, max_position=NO_POSITION_LIMIT,
            stop_token_ids=(), layer_prefix="l{i}.", embed_name="embed", final_norm_name="final.norm", head_name="head",
            logit_scale=self.logit_scale, unused_names=tuple(unused))
