from . import attention, block, feed_forward, latent, norm, position, recurrent, stream  # noqa: F401  (registers the parts)
from .model import DecoderModel, LayerRun
from .registry import (BLOCKS, FEED_FORWARDS, LOGIT_TRANSFORMS, MIXERS, NORMS, POSITION_ENCODINGS, STREAM_INPUTS, BuildContext, build_part,
                       register_block, register_feed_forward, register_logit_transform, register_mixer, register_norm,
                       register_position_encoding, register_stream_input, sub_weights)

__all__ = ["DecoderModel", "LayerRun", "BLOCKS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITION_ENCODINGS",
           "LOGIT_TRANSFORMS", "STREAM_INPUTS", "register_stream_input", "register_logit_transform", "BuildContext", "build_part", "register_block", "register_feed_forward", "register_mixer",
           "register_norm", "register_position_encoding", "sub_weights"]
