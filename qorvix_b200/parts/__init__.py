from .base import Block, FeedForward, Mixer, Norm, PositionEncoding, Runtime
from .registry import build_part, register_part, registered_parts, unregister_part
from .spec import (ActMLPSpec, AttentionSpec, BiasedAttentionSpec, BigramEmbeddingSpec, ChannelDecaySpec, ChannelDeltaSpec, ConvInputSpec,
                   DeltaRuleSpec, DepthAverageSpec, HeadDeltaSpec, RotNormAttentionSpec,
                   DiffAttentionSpec, GLASpec, LatentAttentionSpec, LayerSpec, LoopSpec, Mamba2Spec, MLSTMSpec, ModelSpec, MoESpec,
                   PositionedEmbeddingSpec, RMSNormSpec, RotarySpec, SideBySideSpec, StreamLinkSpec, StreamsSpec, SwiGLUSpec, TableMoESpec,
                   TalkingAttentionSpec, TanhNormSpec, YarnScaling)
from . import (attention, bias_attention, block, channel_recurrent, conv_input, depth_average, diff_attention, embedding,   # registers the
               latent_attention, loop, mlp, moe, recurrent, rmsnorm, rot_norm_attention, rotary, side_by_side, streams, talking_attention, tanh_norm)  # built-in parts
from .linear import Linear
