"""Grouped-query attention over key ranges of a cache, with separate key and value sizes, norms over the whole query and key projections and
a query temperature that grows with the position.

Its steps are CUDA kernels (``ops/span.py``): one launch between the joined input projection and attention (norms, temperature, cache
write), flash attention on the cache for several queries per row, split-key attention for one.  On CPU and under autograd the module runs
the plain statement."""
from __future__ import annotations

from typing import Any, Dict, List, Optional

import torch
from torch import nn

from .. import ops
from ..ops import reference
from ._spans import dense_visibility, kernel_bounds, positions
from .cached_mixer import CachedMixer
from .kv_cache import SpanKVCache


class QueryTemperature:
    """Queries at position ``p`` are multiplied by ``1 + coef · ln(⌊(p + 1) / every⌋ + 1)``."""

    def __init__(self, coef: float, every: int) -> None:
        if int(every) != every or every < 1:
            raise ValueError(f"the temperature steps every {every} positions: a positive whole number is needed")
        self.coef, self.every = float(coef), int(every)

    def __call__(self, pos: torch.Tensor) -> torch.Tensor:
        steps = torch.div(pos.long() + 1, self.every, rounding_mode="floor")
        return 1.0 + self.coef * torch.log((steps + 1).float())


class SpanAttention(CachedMixer):
    """``num_heads`` query heads share ``num_kv_heads`` keys and values in consecutive groups.  ``q_norm`` / ``k_norm`` (RMS norms of the
    whole projections, before they are split into heads) come together or not at all; positions enter only through ``temperature``."""

    def __init__(self, *, embed_dim: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int, q_proj: nn.Module, k_proj: nn.Module, v_proj: nn.Module,
                 output_proj: nn.Module, scale: float, q_norm: Optional[nn.Module] = None, k_norm: Optional[nn.Module] = None, temperature: Optional[QueryTemperature] = None) -> None:
        super().__init__()
        if num_heads % num_kv_heads != 0:
            raise ValueError(f"num_heads ({num_heads}) must be divisible by num_kv_heads ({num_kv_heads})")
        if (q_norm is None) != (k_norm is None):
            raise ValueError("q and k norm must be set together")
        self.embed_dim, self.num_heads, self.num_kv_heads, self.key_dim, self.value_dim = embed_dim, num_heads, num_kv_heads, key_dim, value_dim
        self.q_proj, self.k_proj, self.v_proj, self.output_proj = q_proj, k_proj, v_proj, output_proj
        self.q_norm, self.k_norm = q_norm, k_norm
        self.scale, self.temperature = float(scale), temperature

    def new_cache(self, batch_size: int, dtype: torch.dtype, max_seq_len: int) -> SpanKVCache:
        return SpanKVCache(batch_size, max_seq_len, self.num_kv_heads, self.key_dim, self.value_dim, dtype)

    def input_projections(self) -> List[nn.Module]:
        return [self.q_proj, self.k_proj, self.v_proj]

    def forward(self, x: torch.Tensor, y: Optional[torch.Tensor] = None, *, mask=None, input_pos: Optional[torch.Tensor] = None,
                layer_state: Optional[Dict[Any, Any]] = None) -> torch.Tensor:
        if y is not None and y is not x:
            raise ValueError("attention over key ranges is self-attention only")
        state = {} if layer_state is None else layer_state
        cache = self.current_cache(state)
        if ops.cuda_ops_enabled(x) and x.dtype in (torch.bfloat16, torch.float32):
            if not self.needs_gradients(x):
                bounds = kernel_bounds(state, mask, x, 0 if cache is None else cache.size)
                if bounds is not None:
                    return self._forward_kernels(x, bounds, input_pos, state, cache)
                ops._fallback("span_attention", "a mask whose rows are not key ranges", x)
            else:
                ops._fallback("span_attention", "gradients", x)
        return self._forward_statement(x, mask, input_pos, cache)

    def _forward_kernels(self, x: torch.Tensor, bounds, input_pos: Optional[torch.Tensor], state: Dict[Any, Any], cache: Optional[SpanKVCache]) -> torch.Tensor:
        from ..ops import span

        b, s, _ = x.shape
        q, k, v = self.project(x.reshape(b * s, -1))
        pos = positions(state, input_pos, b, s)
        if cache is not None:
            first, slot = cache.reserve(b, s), cache.slot
            keys, values = cache.k[:b], cache.v[:b]
        else:
            first, slot = 0, None
            keys = torch.empty(b, s, self.num_kv_heads, self.key_dim, dtype=x.dtype, device=x.device)
            values = torch.empty(b, s, self.num_kv_heads, self.value_dim, dtype=x.dtype, device=x.device)
        decode = s == 1 and cache is not None
        if slot is not None and not decode:
            raise RuntimeError("a cache whose position lives on the device takes one token per step")
        t = self.temperature
        q = span.prepare(q, k, v, None if self.q_norm is None else self.q_norm.scale, None if self.k_norm is None else self.k_norm.scale, keys, values, pos, s=s, slot=slot, slot_host=first,
                         eps=0.0 if self.q_norm is None else self.q_norm.eps, coef=0.0 if t is None else t.coef, every=1 if t is None else t.every)
        if cache is not None:
            cache.advance(s)
        if decode:
            out = span.decode(q.view(b, self.num_heads, self.key_dim), keys, values, scale=self.scale, slot=slot, slot_host=first, bounds=bounds,
                              keys_visible=first + 1 if slot is None else keys.shape[1])
        else:
            out = span.prefill(q, keys, values, b=b, s=s, sk=first + s, slot0=first, heads=self.num_heads, scale=self.scale, bounds=bounds)
        return self.output_proj(out.view(b, s, self.num_heads * self.value_dim))

    def _forward_statement(self, x: torch.Tensor, mask, input_pos: Optional[torch.Tensor], cache: Optional[SpanKVCache]) -> torch.Tensor:
        b, s, _ = x.shape
        q, k, v = self.q_proj(x), self.k_proj(x), self.v_proj(x)
        if self.q_norm is not None:
            q, k = self.q_norm(q), self.k_norm(k)
        first = 0 if cache is None else cache.reserve(b, s)
        if self.temperature is not None:
            pos = torch.arange(first, first + s, device=x.device) if input_pos is None else input_pos.reshape(-1, s)
            q = (q.float() * self.temperature(pos)[..., None]).to(q.dtype)
        k, v = k.view(b, s, self.num_kv_heads, self.key_dim), v.view(b, s, self.num_kv_heads, self.value_dim)
        if cache is not None:
            cache.k[:b, first : first + s], cache.v[:b, first : first + s] = k, v
            cache.advance(s)
            k, v = cache.k[:b, : first + s], cache.v[:b, : first + s]
        visible = dense_visibility(mask, b, s, first + s, first, x.device)
        out = reference.span_attention(q.view(b, s, self.num_heads, self.key_dim), k, v, visible, self.scale)
        return self.output_proj(out.reshape(b, s, self.num_heads * self.value_dim))
