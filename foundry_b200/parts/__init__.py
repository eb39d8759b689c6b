"""Layer parts and their registries; importing registers the built-in ones."""
from .base import (BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, Part, Registry,
                   register_block, register_feed_forward, register_mixer, register_norm,
                   register_position_encoding)
from . import (attention, block, differential_attention, embedding, junction,  # noqa: F401
               latent_attention, linear, mlp, moe, norm, parallel, recurrent, rope,
               rotary_sink_attention, shared_row_attention, sigmoid_attention, sink_attention,
               window_attention)  # (registration)
from .embedding import EMBEDDINGS, register_embedding
from .junction import JUNCTIONS, register_junction
from .attention import GQAAttention
from .block import PreNormResidualBlock
from .linear import Linear, matmul_nt
from .mlp import SwiGLU
from .norm import LayerNorm, RMSNorm
from .rope import Rope, RopeLlama3, llama3_inv_freq, plain_inv_freq

__all__ = ["BLOCKS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "Part", "Registry",
           "register_block", "register_feed_forward", "register_mixer", "register_norm",
           "register_position_encoding", "EMBEDDINGS", "JUNCTIONS", "register_embedding",
           "register_junction", "LayerNorm", "GQAAttention", "PreNormResidualBlock", "Linear",
           "matmul_nt", "SwiGLU", "RMSNorm", "Rope", "RopeLlama3", "llama3_inv_freq",
           "plain_inv_freq"]
