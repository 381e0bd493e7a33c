"""Parts a decoder is assembled from.  Importing this package registers the built-in kinds."""
from . import (attention, block, latent_attention, matrix_memory, min_gru, mlp, moe, norm, retention, rope,  # noqa: F401
               selective_scan, side_by_side, state_space)
from .base import (Block, CacheView, FeedForward, HostBatch, Mixer, Norm, Part, PositionEncoding, StepContext,
                   WeightSpec)
