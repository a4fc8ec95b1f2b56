from . import standard  # registers the standard parts
from . import dynamic_tanh, delta_rule, latent_attention, routed  # noqa: F401  (more parts)
from . import rms_norm, biased_attention, lightning, paired  # noqa: F401
from . import pooled_attention, rglru  # noqa: F401
from . import retention, span_attention, time_mix, token_side  # noqa: F401
from . import layer_scale, normed_embedding  # noqa: F401
from . import hyper_connection, state_space  # noqa: F401
from .base import (CacheRequest, Embedding, FeedForward, Head, Mixer, Norm, Part,
                   PositionEncoding, TensorRequest, build_part, register_connection,
                   register_embedding,
                   register_feed_forward, register_head, register_mixer, register_norm,
                   register_position, register_scale, registered)
from .model import (Block, CacheGroup, HyperConnectedBlock, Model, OutputNormBlock, ParallelBlock, PreNormBlock,
                    SandwichNormBlock, ScaledParallelBlock, register_arrangement)
from .spec import LayerCall, LayerSpec, ModelSpec, PartSpec

__all__ = [
    "Block", "CacheGroup", "CacheRequest", "Embedding", "FeedForward", "Head",
    "HyperConnectedBlock", "LayerCall",
    "LayerSpec", "Mixer", "Model", "ModelSpec", "Norm", "OutputNormBlock", "Part", "PartSpec", "PositionEncoding",
    "ParallelBlock", "PreNormBlock", "SandwichNormBlock", "ScaledParallelBlock", "TensorRequest", "build_part", "register_arrangement",
    "register_connection", "register_embedding", "register_feed_forward", "register_head", "register_mixer",
    "register_norm", "register_position", "register_scale", "registered",
]
