from . import (attention, block, branches, delta_memory, latent_attention, linear_attention, mlp, mlstm, moe, norm,  # noqa: F401
               normed_attention, rope, token_input)   # (register the built-in parts)
from .base import (BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, TOKEN_INPUTS, Block, BuildContext,
                   FeedForward, Mixer, Norm, PagedKV, PagedLatent, Part, PositionEncoding, RequestState,
                   ResidualStream, TokenInput, register_block, register_feed_forward, register_mixer,
                   register_norm, register_position_encoding, register_token_input)
from .linear import linear, linear_partials, reduce_partials

__all__ = [
    "BLOCKS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "TOKEN_INPUTS", "Block", "BuildContext",
    "FeedForward", "Mixer", "Norm", "PagedKV", "PagedLatent", "Part", "PositionEncoding", "RequestState",
    "ResidualStream", "TokenInput", "linear", "linear_partials", "reduce_partials", "register_block", "register_feed_forward", "register_mixer",
    "register_norm", "register_position_encoding", "register_token_input",
]
