"""Begapel: a small decoder of latent-attention layers.

The architecture is read from a ``config.json`` whose ``layers`` list describes every layer on its own (attention sizes, rotation, score
scale, feed-forward width or none, and whether the layer reads another layer's latents).  Each sublayer is normed on both sides with
gains stored around zero, the residual stream is 32-bit and sublayer outputs enter it multiplied by ``residual_mult``; vocabulary logits
are soft-capped.  Everything is built from shared parts: :class:`~torchtune_b200.modules.LatentAttention`,
:class:`~torchtune_b200.modules.ResidualStreamLayer` and the decoder factory.
"""
from ._component_builders import begapel, lora_begapel  # noqa: F401
from ._convert_weights import begapel_hf_to_tune, begapel_tune_to_hf  # noqa: F401

__all__ = ["begapel", "lora_begapel", "begapel_hf_to_tune", "begapel_tune_to_hf"]
