from .base import (FreeDim, KVNeed, LayerIO, NormedInput, ParamDecl, Part, StateNeed, block_class, feed_forward_class, hook_class,
                   mixer_class, norm_class, position_class, register_block, register_feed_forward, register_hook,
                   register_mixer, register_norm, register_position, unregister)
from .linear import Linear
from . import norm, rope, attention, mlp, block, hooks, latent_attention, recurrent, moe, capped_attention, linear_attention, side_by_side, selective_scan, delta_rule, streams  # noqa: F401  (registers the parts)

__all__ = [
    "FreeDim", "KVNeed", "LayerIO", "ParamDecl", "Part", "StateNeed", "Linear",
    "block_class", "feed_forward_class", "hook_class", "mixer_class", "norm_class", "position_class",
    "register_block", "register_feed_forward", "register_hook", "register_mixer", "register_norm",
    "register_position",
    "unregister",
]
