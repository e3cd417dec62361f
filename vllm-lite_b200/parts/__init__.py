"""Model parts: descriptions (`spec`), registries (`registry`) and the standard
implementations, which register themselves when this package is imported."""
from . import spec, registry                      # noqa: F401
from . import norm, rope, attention, mlp, block, embedding, head   # noqa: F401  (registration)
from . import latent_attention, gated_mlp, experts               # noqa: F401  (registration)
from .model import CausalLM, cache_needs, cache_sources, declare_model  # noqa: F401
from .registry import BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITIONS  # noqa: F401
from . import recurrent, parallel, conv_attention, token_shift    # noqa: F401  (registration)
from . import differential_attention, linear_recurrent            # noqa: F401  (registration)
