from . import (attention, block, capped_attention, chunked_attention, clamped_feed_forward, dense_feed_forward, dynamic_tanh, embedding, feed_forward, gated_block,  # noqa: F401
               gated_delta, head, hyper_block, latent_attention, layer_norm, min_gru, norm, normed_pair, output_norm_block,
               parallel_block, retention, rglru, rope, routed_feed_forward, sandwich_block, side_by_side, sigmoid_attention,
               state_space, stream_join, talking_attention, token_side)  # registers the built-in parts
from .base import MODES, Mixer, Part, Prenormed, RunContext, Runtime, StreamRows, StreamsRead, as_delta
from .linear import add_linear, linear
from .registry import build_part, known_parts, register_part, unregister_part
