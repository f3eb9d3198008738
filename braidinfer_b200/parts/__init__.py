"""Parts that layers are made of.  Importing the package registers the built-in parts."""
from .base import (BLOCKS, CONNECTIONS, EMBEDDINGS, FEED_FORWARDS, HEADS, INJECTIONS, LAYER_INPUTS, MIXERS, NORMS,
                   POSITION_ENCODINGS, STREAMS, Block, Connection, Embedding, FeedForward, Head, Injection, LayerInput, Mixer,
                   Norm, Part, PositionEncoding, Registry, Streams)
from .spec import CacheRequest, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TensorSpec
from .runtime import Runtime
from . import (attention, block, delta, embedding, feedforward, hyper, injection, latent_attention,  # noqa: F401
               linear_attention, mlstm, moe, norm, parallel, rope, ssm, token_input)                                       # (registration)
