"""Models: the generic decoder, and the architectures registered for it."""

from ..config.begupel import BegupelConfig
from ..config.kebisun import KebisunConfig
from ..config.muzasun import MuzasunConfig
from ..config.nefivik import NefivikConfig
from ..config.putazen import PutazenConfig
from ..config.qwen3 import Qwen3Config
from ..config.votapel import VotapelConfig
from ..registry import register_architecture
from .decoder import DecoderModel

# "qwen3" is the reference's family key (crates/core/src/config.rs:93-103).
register_architecture("Qwen3ForCausalLM", Qwen3Config, model_types=("qwen3",), default=True)
# Layers of two mixer kinds (latent attention, gated linear attention) with dense or routed
# feed-forwards; config.json names it under "architecture".
register_architecture("Kebisun", KebisunConfig)
# Parallel blocks (one norm, attention and a routed feed-forward side by side) of attention whose values
# are its keys, with biases, a query temperature, capped scores and a sink; learned position vectors.
register_architecture("Votapel", VotapelConfig)
# Layers of lightning attention (a decaying matrix state per head) and of windowed attention with rotated
# values beside a gated delta rule; an input convolution per layer, RMS norms in groups on the sublayers'
# results, a pair embedding, capped logits.
register_architecture("Begupel", BegupelConfig)
# Layers of sigmoid-weighted windowed attention (convolved projections, a gate per head, keys and values that a
# later layer may read) and of a generalised delta rule, each sublayer between two norms and behind a gate; routed
# experts in groups with a clamped activation; a second input by token id at every layer's end.
register_architecture("Nefivik", NefivikConfig)
# A residual of several mixed copies; layers of differential attention, latent attention and a Mamba-2 state-space mixer,
# a run of them several times with the same weights; clamped dense feed-forwards, layer norms with biases.
register_architecture("Putazen", PutazenConfig)
# Parallel blocks whose two sublayers read norms without statistics of the same stream; layers of a matrix memory with
# exponential gates, of the delta rule with a decay per key channel, or of attention whose values are blended with the
# first such layer's; routed experts whose weights multiply their inputs.
register_architecture("Muzasun", MuzasunConfig)

__all__ = ["DecoderModel"]
