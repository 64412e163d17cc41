"""Base of sequence mixers whose cache belongs to the run of the layer, not to the layer: a layer that runs several times in a forward pass
has one cache per run."""
from __future__ import annotations

import logging
from typing import Any, Dict, List, Optional

import torch
from torch import nn

from ..ops import linear
from ._spans import join, joined, plain
from .kv_cache import PassCaches, RowCache

logger = logging.getLogger(__name__)


class CachedMixer(nn.Module):
    """``num_passes`` is how many times the decoder runs this layer per forward pass; the decoder names the current run in
    ``layer_state["pass"]``.  Subclasses create one cache (:meth:`new_cache`) and list the projections of their input
    (:meth:`input_projections`)."""

    def __init__(self) -> None:
        super().__init__()
        self.num_passes = 1
        self.kv_cache: Optional[PassCaches] = None
        self.cache_enabled = False

    def new_cache(self, batch_size: int, dtype: torch.dtype, max_seq_len: int) -> RowCache:
        raise NotImplementedError

    def input_projections(self) -> List[nn.Module]:
        raise NotImplementedError

    # ------------------------------------------------------------------ cache
    def setup_cache(self, batch_size: int, dtype: torch.dtype, max_seq_len: int) -> None:
        if self.kv_cache is not None:
            logger.warning("Key value caches are already setup. You cannot call ``setup_caches()`` twice. Skipping.")
            return
        with torch.no_grad():
            join(self.input_projections())
        self.kv_cache = PassCaches([self.new_cache(batch_size, dtype, max_seq_len) for _ in range(self.num_passes)])
        home = next((p.device for p in self.parameters() if p.device.type != "meta"), None)
        if home is not None and home.type != "cpu":  # a cache created outside a device context belongs where the weights are
            self.kv_cache.to(home)
        self.cache_enabled = True

    def reset_cache(self) -> None:
        if self.kv_cache is None:
            raise RuntimeError("Key value caches are not setup. Call ``setup_caches()`` first.")
        self.kv_cache.reset()

    def current_cache(self, state: Dict[Any, Any]) -> Optional[RowCache]:
        return self.kv_cache[state.get("pass", 0)] if self.cache_enabled and self.kv_cache is not None else None

    # ------------------------------------------------------------------ projections
    def project(self, x2: torch.Tensor) -> List[torch.Tensor]:
        """Results of the input projections as 2-D tensors with contiguous rows (column blocks of one product where the weights are one
        matrix)."""
        mods = self.input_projections()
        whole = joined(mods)
        if whole is not None:
            return list(linear(x2, whole).split([m.weight.shape[0] for m in mods], dim=1))
        return [linear(x2, m.weight) if plain(m) else m(x2) for m in mods]

    def needs_gradients(self, x: torch.Tensor) -> bool:
        return torch.is_grad_enabled() and (x.requires_grad or any(p.requires_grad for p in self.parameters()))
