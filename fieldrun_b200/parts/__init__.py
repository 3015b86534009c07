"""Parts that layers are put together from.  Importing the package registers the built-in kinds."""
from . import addition, attention, block, connector, embedding, feed_forward, hyper_connections, latent_attention, linear_attention, mixer_pair, norm, position, recurrent, retention, token_shift  # noqa: F401
from .base import (Addition, BiasedRows, Block, Connector, CopiesUpdate, DeferredUpdate, MixerInput, StreamConnection, UpdateSum, WeightedRows, FeedForward, Mixer, Norm, Part, Position, as_tensor, build_block, build_part,
                   build_position, register_part, registered)

__all__ = ["Addition", "BiasedRows", "Block", "Connector", "CopiesUpdate", "DeferredUpdate", "MixerInput", "StreamConnection", "UpdateSum", "WeightedRows", "as_tensor", "FeedForward", "Mixer", "Norm", "Part", "Position", "build_block", "build_part",
           "build_position", "register_part", "registered"]
