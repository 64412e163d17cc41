"""Linear attention with a fixed decay per head ("lightning attention"): a recurrent state instead of a key/value cache.

Per head ``S_t = λ S_{t-1} + k_t v_tᵀ`` and ``o_t = S_tᵀ q_t``, with SiLU on the three projections; the heads' outputs are normed together and
gated.  The state is kept in fp32.  Several tokens per row run as tensor-core chunks, a single one as one pass over the state
(``ops/recurrent.py``); on CPU and under autograd the module runs the plain statement."""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch
import torch.nn.functional as F
from torch import nn

from .. import ops
from ..ops import reference
from ._spans import row_starts
from .cached_mixer import CachedMixer
from .kv_cache import StateCache


class LightningAttention(CachedMixer):
    def __init__(self, *, embed_dim: int, num_heads: int, key_dim: int, value_dim: int, decay: Sequence[float], q_proj: nn.Module, k_proj: nn.Module, v_proj: nn.Module,
                 gate_proj: nn.Module, norm: nn.Module, output_proj: nn.Module) -> None:
        super().__init__()
        if len(decay) != num_heads or not all(0.0 <= d <= 1.0 for d in decay):
            raise ValueError(f"{num_heads} heads need as many decays between 0 and 1, not {list(decay)}")
        self.embed_dim, self.num_heads, self.key_dim, self.value_dim = embed_dim, num_heads, key_dim, value_dim
        self.decay = tuple(float(d) for d in decay)
        self.q_proj, self.k_proj, self.v_proj, self.gate_proj = q_proj, k_proj, v_proj, gate_proj
        self.norm, self.output_proj = norm, output_proj

    def new_cache(self, batch_size: int, dtype: torch.dtype, max_seq_len: int) -> StateCache:
        return StateCache(batch_size, max_seq_len, self.num_heads, self.key_dim, self.value_dim)

    def input_projections(self) -> List[nn.Module]:
        return [self.q_proj, self.k_proj, self.v_proj, self.gate_proj]

    def forward(self, x: torch.Tensor, y: Optional[torch.Tensor] = None, *, mask=None, input_pos: Optional[torch.Tensor] = None,
                layer_state: Optional[Dict[Any, Any]] = None) -> torch.Tensor:
        if y is not None and y is not x:
            raise ValueError("a recurrent layer reads one sequence")
        state = {} if layer_state is None else layer_state
        cache = self.current_cache(state)
        b, s, _ = x.shape
        first = 0 if cache is None else cache.reserve(b, s)
        starts = row_starts(state, mask, b, s, first, x.device)
        if ops.cuda_ops_enabled(x) and x.dtype in (torch.bfloat16, torch.float32) and not self.needs_gradients(x):
            out = self._forward_kernels(x, first, starts, cache)
        else:
            if ops.cuda_ops_enabled(x):
                ops._fallback("lightning_attention", "gradients", x)
            out = self._forward_statement(x, first, starts, cache)
        if cache is not None:
            cache.advance(s)
        return self.output_proj(out.view(b, s, self.num_heads * self.value_dim))

    def _forward_kernels(self, x: torch.Tensor, first: int, starts: Optional[torch.Tensor], cache: Optional[StateCache]) -> torch.Tensor:
        from ..ops import recurrent

        b, s, _ = x.shape
        q, k, v, gate = self.project(x.reshape(b * s, -1))
        if cache is not None and cache.slot is not None and s != 1:
            raise RuntimeError("a cache whose position lives on the device takes one token per step")
        o = recurrent.lightning(q, k, v, self.decay, None if cache is None else cache.state[:b], b=b, s=s, heads=self.num_heads, dim=self.key_dim, vdim=self.value_dim, fresh=first == 0,
                                starts=None if cache is not None and cache.slot is not None else starts, first=first)
        return recurrent.gated_norm(o, self.norm.scale, gate, self.norm.eps)

    def _forward_statement(self, x: torch.Tensor, first: int, starts: Optional[torch.Tensor], cache: Optional[StateCache]) -> torch.Tensor:
        b, s, _ = x.shape
        q, k = (F.silu(p(x)).view(b, s, self.num_heads, self.key_dim) for p in (self.q_proj, self.k_proj))
        v = F.silu(self.v_proj(x)).view(b, s, self.num_heads, self.value_dim)
        if starts is not None:  # padding leaves nothing in the state
            real = first + torch.arange(s, device=x.device)[None, :] >= starts[:, None]
            k = k * real[:, :, None, None]
        before = None if cache is None or first == 0 else cache.state[:b]
        o, after = reference.lightning_attention(q, k, v, self.decay, before)
        if cache is not None:
            cache.state[:b] = after.detach()
        return reference.gated_norm(o.reshape(b, s, -1), self.norm.scale, self.gate_proj(x), self.norm.eps)
