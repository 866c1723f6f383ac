from .base import (BLOCKS, CONNECTIONS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, Block, CacheRequest, EMBED_ADDS, EmbedAdd, FeedForward, LayerCache,
                   Mixer, Mixture, Norm, Part, PassEntry, PositionEncoding, PostNormed, Replaced, Runtime, ScaledSum, make_part, register_block, register_feed_forward,
                   Connection, NormedPair, StreamAdd, Streams, register_connection, register_embed_add, register_mixer, register_norm, register_pass_entry, register_position_encoding, to_f32, to_operand)
from . import norm, position, embedding, loop, attention, latent_attention, ssm, delta, retention, time_mix, side_by_side, ffn, side, block   # noqa: F401  (register the built-in parts)
