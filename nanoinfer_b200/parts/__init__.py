"""The parts a model is put together from.  Importing this package registers the built-in
parts under their names."""
from . import (attention, block, delta_rule, depth_mix, differential, embedding, gated_scan, head, hyper, latent_attention, min_gru, mlp,  # noqa: F401
               mlstm, norm, pooled_attention, position, retention, routed, selective_scan, stream_vectors)  # (registration)
from .base import (CONNECTORS, DEPTH_MIXES, FEED_FORWARDS, HEADS, EMBEDDINGS, MIXERS, NORMS, POSITIONS, STREAM_VECTORS, Connector, DepthMix, Embedding, FeedForward, Head,
                   KVCacheSpec, KVCacheView, Mixer, Norm, ParamSpec, Part, PositionEncoding, StateSpec,
                   StepContext, StreamVectors, TensorRef, TwoProducts, Workspace, register_connector, register_depth_mix, register_embedding, register_feed_forward,
                   register_head, register_mixer, register_norm, register_position, register_stream_vectors)
from .block import BLOCKS, Block, register_block

__all__ = [n for n in dir() if not n.startswith("_")]
