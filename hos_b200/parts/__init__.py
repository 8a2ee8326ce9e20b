"""The parts a layer is put together from.  Importing this package registers them."""
from . import (attention, block, differential_attention, embedding, feedforward, gated_attention, hyper, latent_attention, moe,  # noqa: F401
               norm, parallel_mixers, rope, state_mixers, wkv)
