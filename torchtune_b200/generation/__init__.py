from ._generation import (
    generate,
    generate_next_token,
    get_causal_mask_from_padding_mask,
    get_position_ids_from_padding_mask,
    last_logits,
    sample,
)
from ._rows import BatchDecoder, DecodeGraph, RowLayout

__all__ = ["generate", "generate_next_token", "get_causal_mask_from_padding_mask", "get_position_ids_from_padding_mask", "sample", "last_logits", "BatchDecoder", "DecodeGraph", "RowLayout"]
