"""Parts of a layer (mixer, feed-forward, norm, position encoding, arrangement) and the model
that a ModelSpec puts together from them.  Importing this package registers the built-in kinds."""
from .base import (Block, CacheNeed, EmbedPart, FeedForward, Mixer, Norm, Part, Position, StateNeed, StreamAddon, WeightSpec, build_block,
                   build_part, register_part, registered)
from .spec import Application, LayerSpec, ModelSpec, PartSpec
from . import attention, block, delta, depth, embed, latent, linear_attention, mingru, mlp, mlstm, moe, norm, parallel, position, rglru, shift, side, ssm  # noqa: F401  (register the built-in kinds)
from .model import DecoderModel

__all__ = ["Application", "Block", "CacheNeed", "DecoderModel", "EmbedPart", "FeedForward", "LayerSpec", "Mixer", "ModelSpec", "Norm",
           "Part", "PartSpec", "Position", "StateNeed", "StreamAddon", "WeightSpec", "build_block", "build_part", "register_part",
           "registered"]
