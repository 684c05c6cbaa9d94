# importing a module registers the kinds it defines
from . import (attention, embedding, feed_forward, gated_pair, latent_attention,  # noqa: F401
               linear_recurrence, matrix_memory, norm, position, state_space, streams,
               token_shift)
from .base import (BuildContext, GroupView, LayerCache, PagedKvNeed, StateNeed,  # noqa: F401
                   StepContext)
from .block import Block, DecoderModel  # noqa: F401
from .registry import build_part, known, register_part, unregister_part  # noqa: F401
from .specs import (ClampedGluSpec, GroupedRmsNormSpec,  # noqa: F401
                    InterleavedRopeSpec, LatentAttentionSpec, TokenShiftSpec)
from .specs import (AttentionSpec, LayerSpec, ModelSpec, MoeSpec, RmsNormSpec,  # noqa: F401
                    RopeSpec, RunEntry, SwiGluSpec)
