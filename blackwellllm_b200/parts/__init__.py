"""Parts of a decoder: norms, position encodings, mixers, feed-forwards, blocks."""
from .base import (Block, BorrowedCache, BuildContext, FeedForward, FixedStateRequest, Mixer, Norm, PagedKVRequest,
                   ParamSpec, Part, PositionEncoding, build_block, build_ffn, build_mixer, build_norm,
                   build_position, register_block, register_ffn, register_mixer, register_norm,
                   register_position)
from . import (attention, block, diff_attention, gated_delta, gla, latent_attention, mlp, mlstm, moe, norm, rope,  # noqa: F401
               side_by_side, state_space)  # noqa: F401  (registers the built-in parts)
from .linear import Linear
