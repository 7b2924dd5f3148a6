"""Parts that layers are put together from.  Importing the package registers the built-in kinds."""

from . import (attention, bigram, block, channel_delta, depth_average, differential_attention, feed_forward,  # noqa: F401
               latent_attention, linear_recurrence, min_gru, norms, pass_entry, recurrent_heads, rope, routed_experts, side_by_side, time_mix, token_side)
from .base import (BLOCKS, FEED_FORWARDS, LAYER_EXTRAS, MIXERS, NORMS, PASS_ENTRIES, POSITION_ENCODINGS, STREAM_MIXES,  # noqa: F401
                   Block, BuildContext, CacheNeeds, FeedForward, KVNeeds, LayerExtra, LayerSpec, Mixer, ModelSpec, Norm,
                   Part, PartSpec, PositionEncoding, ScheduleEntry, Stage, StateNeeds, StreamMix, TensorSpec)
