"""The parts a model is assembled from.  Importing the package registers the built-in kinds."""
from . import (attention, block, channel_delta, conv_attention, delta_rule, distance_attention, feedforward,  # noqa: F401
               gated_recurrence, latent_attention, matrix_memory, mixed_head_attention, norm, position, retention, rotated_attention,
               routed_experts, selective_scan, side_by_side, sink_attention, state_space)
from .base import (BLOCKS, Block, EMBEDDING, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, ROTATION,  # noqa: F401
                   CacheNeed, ModelContext, Rotation, Part, StepContext, Workspace, register_block, register_feed_forward,
                   register_mixer, register_norm, register_position_encoding)
