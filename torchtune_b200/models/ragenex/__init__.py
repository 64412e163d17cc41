"""Ragenex: a small decoder of attention and linear-attention layers on several residual streams.

The architecture is read from a ``config.json`` whose ``layers`` list describes every layer on its own: grouped-query attention without
rotation (norms over the whole query and key projections, a query temperature that grows with the position) or lightning attention (a
recurrent state with one decay per head), each with a clamped gated feed-forward block or none.  Sublayers sit between layer norms and layer
scales on hyper-connected 32-bit streams; positions are learned embeddings; a run of layers may be repeated with the same weights.
Everything is built from shared parts: :class:`~torchtune_b200.modules.SpanAttention`,
:class:`~torchtune_b200.modules.LightningAttention`, :class:`~torchtune_b200.modules.HyperConnectionLayer` and the decoder factory.
"""
from ._component_builders import lora_ragenex, ragenex  # noqa: F401
from ._convert_weights import ragenex_hf_to_tune, ragenex_tune_to_hf  # noqa: F401

__all__ = ["ragenex", "lora_ragenex", "ragenex_hf_to_tune", "ragenex_tune_to_hf"]
