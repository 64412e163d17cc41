from .attention import MultiHeadAttention
from .attention_utils import create_block_causal_mask, packed_block_causal_mask
from .classifier import classifier_model
from .common_utils import (
    delete_kv_caches,
    disable_kv_cache,
    local_kv_cache,
    reparametrize_as_dtype_state_dict_post_hook,
    slice_str_to_array,
)
from .embedding_utils import resize_token_embeddings
from .cached_mixer import CachedMixer
from .feed_forward import ClampedGLU, FeedForward
from .hyper_connections import HyperConnection, LayerScale
from .kv_cache import KVCache, PassCaches, RowCache, SpanKVCache, StateCache
from .latent_attention import LatentAttention, LatentCache
from .layer_norm import Fp32LayerNorm
from .linear import Linear
from .linear_attention import LightningAttention
from .low_precision import FrozenNF4Linear
from .position_embeddings import (
    HalfSplitRotaryPositionalEmbeddings,
    Llama3ScaledRoPE,
    Llama4ScaledRoPE,
    Phi3RotaryPositionalEmbeddings,
    Qwen2RotaryPositionalEmbeddings,
    RotaryPositionalEmbeddings,
    VisionRotaryPositionalEmbeddings,
)
from .rms_norm import RMSNorm, StreamLayerNorm, StreamRMSNorm, rms_norm
from .span_attention import QueryTemperature, SpanAttention
from .tanh_gate import TanhGate
from .tied_linear import TiedLinear
from .transformer import HyperConnectionLayer, ResidualStreamLayer, TransformerCrossAttentionLayer, TransformerDecoder, TransformerSelfAttentionLayer
from .layer_dropout import LayerDropout, ModuleLayerDropoutWrapper, ScaleType, get_scale, prepare_layer_dropout
from .vq_embeddings import VectorQuantizedEmbeddings
from .vision_transformer import CLSEmbedding, CLSProjection, PatchEmbedding, VisionTransformer

__all__ = [
    "MultiHeadAttention",
    "create_block_causal_mask",
    "packed_block_causal_mask",
    "LayerDropout",
    "ModuleLayerDropoutWrapper",
    "ScaleType",
    "get_scale",
    "prepare_layer_dropout",
    "VectorQuantizedEmbeddings",
    "VisionTransformer",
    "CLSEmbedding",
    "CLSProjection",
    "PatchEmbedding",
    "TanhGate",
    "CachedMixer",
    "ClampedGLU",
    "FeedForward",
    "FrozenNF4Linear",
    "HyperConnection",
    "HyperConnectionLayer",
    "KVCache",
    "LatentAttention",
    "LatentCache",
    "LayerScale",
    "LightningAttention",
    "Linear",
    "RotaryPositionalEmbeddings",
    "VisionRotaryPositionalEmbeddings",
    "Llama3ScaledRoPE",
    "Llama4ScaledRoPE",
    "HalfSplitRotaryPositionalEmbeddings",
    "Qwen2RotaryPositionalEmbeddings",
    "Phi3RotaryPositionalEmbeddings",
    "PassCaches",
    "QueryTemperature",
    "RMSNorm",
    "RowCache",
    "SpanAttention",
    "SpanKVCache",
    "StateCache",
    "StreamLayerNorm",
    "StreamRMSNorm",
    "rms_norm",
    "TiedLinear",
    "Fp32LayerNorm",
    "TransformerDecoder",
    "TransformerSelfAttentionLayer",
    "ResidualStreamLayer",
    "TransformerCrossAttentionLayer",
    "reparametrize_as_dtype_state_dict_post_hook",
    "delete_kv_caches",
    "disable_kv_cache",
    "local_kv_cache",
    "slice_str_to_array",
    "classifier_model",
    "resize_token_embeddings",
]
