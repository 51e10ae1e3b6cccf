from .base import (
    DeferredProduct, KVRequest, ResidualStream, Runtime, StateRequest, Workspace, part_class,
    register_block, register_embedding, register_feed_forward, register_head, register_mixer, register_norm,
    register_position, register_stream_map,
)
from . import attention, block, conv_attention, embedding, feed_forward, hyper_connection, latent_attention, norm, position, recurrent, side_by_side, stream_map  # noqa: F401  (register the built-in parts)
from .linear import Linear

__all__ = [
    "DeferredProduct", "KVRequest", "Linear", "ResidualStream", "Runtime", "StateRequest", "Workspace", "part_class",
    "register_block", "register_embedding", "register_feed_forward", "register_head", "register_mixer",
    "register_norm", "register_position", "register_stream_map",
]
