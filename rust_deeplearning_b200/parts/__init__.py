"""Parts of a model.  Importing the package registers the built-in kinds."""
from . import (attention, decay_attention, delta_rule, feed_forward, head_attention, hyper, latent_attention,  # noqa: F401
               matrix_memory, mixer_pair, model, norm, position, routed_experts, state_space)
