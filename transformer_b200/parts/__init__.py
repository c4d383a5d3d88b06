"""Parts of a model: embeddings, norms, mixers, feed-forwards, position encodings, heads and the arrangements
of a block, each behind a registry."""
from .base import (ARRANGEMENTS, EMBEDDINGS, FEED_FORWARDS, HEADS, INPUT_FILTERS, JOINTS, MIXERS, NORMS, POSITIONS,
                   RESIDUAL_GATES, CacheNeed, DepthSum, Embedding, FeedForward, GatedDelta, Head, InputFilter, Joint, Mixer, Norm, NormedDelta, PairDelta, ParamDecl, Part,
                   Position, ResidualGate, StateNeed, StreamRows, WeightedRows)
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry
from . import (attention, block, channel_delta, decay_memory, ends, feed_forward, gated_linear, latent_attention,  # noqa: F401
               mlstm, norm, rope, side_by_side, split_delta, stream)      # (registers the built-in kinds)
