"""Parts that layers are put together from.  Importing the package registers the built-in kinds."""
from . import (attention, block, delta_rule, embedding, feed_forward, gate, gated_linear, input_conv,  # noqa: F401
               latent_attention, lightning, mingru, moe, multimap_attention, norm, position, selective_scan, side_by_side,
               sink_attention, sloped_attention, unit_attention, window_attention)
from .base import (Block, CacheView, FeedForward, Mixer, Norm, Part, Product, Runtime, Segment, StepContext,
                   StepPlanner, Workspace)
from .registry import (
    BLOCKS,
    EMBEDDINGS,
    FEED_FORWARDS,
    HEADS,
    MIXERS,
    NORMS,
    POSITIONS,
    register_block,
    register_feed_forward,
    register_mixer,
    register_norm,
    register_position,
)
from .spec import (CacheNeed, LayerSpec, ModelSpec, PagedKVNeed, PagedNeed, PagedRowsNeed, ParamSpec, PartSpec, RunEntry,
                   StateNeed)
