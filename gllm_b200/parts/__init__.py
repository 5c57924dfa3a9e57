"""Layer parts: mixer, feed-forward, norm, position encoding and block."""

from gllm_b200.parts.base import (
    BLOCKS,
    DEPTH_AVERAGES,
    FEED_FORWARDS,
    INPUT_CONVS,
    MIXERS,
    NORMS,
    POSITION_ENCODINGS,
    Block,
    DepthAverage,
    FeedForward,
    GroupView,
    InputConv,
    KVPageRequirement,
    Mixer,
    MixerCache,
    Norm,
    Part,
    PositionEncoding,
    StateRequirement,
    StepContext,
    TensorExpectation,
    build_part,
    register_block,
    register_depth_average,
    register_feed_forward,
    register_input_conv,
    register_mixer,
    register_norm,
    register_position_encoding,
)
from gllm_b200.parts import (  # noqa: F401  (register the built-in kinds)
    attention, block, conv_attention, delta_rule, depth, differential_attention, distance_attention, experts, hyper,
    latent_attention, mamba, matrix_memory, mlp, norm, parallel, rotary, sigmoid_attention,
)

__all__ = [
    "BLOCKS", "DEPTH_AVERAGES", "FEED_FORWARDS", "INPUT_CONVS", "MIXERS", "NORMS", "POSITION_ENCODINGS",
    "Block", "DepthAverage", "FeedForward", "GroupView", "InputConv", "KVPageRequirement", "Mixer", "MixerCache", "Norm", "Part",
    "PositionEncoding", "StateRequirement", "StepContext", "TensorExpectation", "build_part",
    "register_block", "register_depth_average", "register_feed_forward", "register_input_conv", "register_mixer", "register_norm", "register_position_encoding",
]
