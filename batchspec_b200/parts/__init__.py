from .base import (BLOCKS, BRANCH_SCALES, DEPTH_AVERAGES, FEED_FORWARDS, INPUT_PARTS, LOGITS_PARTS, MIXERS, NORMS, POSITION_ENCODINGS, Block, CacheSpec,
                   FeedForward, InputPart, LogitsPart, Mixer, Norm, ParamSpec, Part, PartSpec, PositionEncoding, Runtime,
                   StateSpec, build_part, register_part)
from . import (attention, block, delta_rule, embedding, latent_attention, lightning, logits, matrix_memory, mlp, moe, norm, parallel,
               retention, rope, selective_scan, sink_attention, state_space)  # noqa: F401  (registers the built-in parts)

__all__ = ["BLOCKS", "BRANCH_SCALES", "DEPTH_AVERAGES", "FEED_FORWARDS", "INPUT_PARTS", "LOGITS_PARTS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "Block",
           "CacheSpec", "FeedForward", "InputPart", "LogitsPart", "Mixer", "Norm", "ParamSpec", "Part", "PartSpec", "PositionEncoding", "Runtime", "StateSpec",
           "build_part", "register_part"]
