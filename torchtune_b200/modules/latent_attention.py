"""Multi-head latent attention: keys and values are low-rank functions of one cached latent per token.

Per token the cache holds a normalised latent ``c`` (``kv_rank`` values) and one rotated key part shared by all heads (``rot_dim``
values).  A head's key is ``[W_uk c | shared rotated part]``, its value ``W_uv c``.

Two ways to evaluate it, chosen by the number of queries per row: several queries (prefill) expand keys and values once with one GEMM and
run flash attention on them; a single query (decoding) multiplies ``W_ukᵀ`` into the query instead, attends over the latents themselves —
one key / value stream for all heads — and multiplies ``W_uv`` into the result.  Both, and the step between the input projections and
attention (latent norm, rotation, cache write), are CUDA kernels (``ops/latent.py``); on CPU and under autograd the module runs the
plain statement.

A layer may have no latent of its own and read another layer's (``latent_from``).
"""
from __future__ import annotations

import logging
from typing import Any, Dict, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..ops import reference
from ._spans import dense, dense_visibility, join, joined, kernel_bounds, plain, positions
from .kv_cache import RowCache
from .position_embeddings import RotaryPositionalEmbeddings

logger = logging.getLogger(__name__)


class PreciseRotaryPositionalEmbeddings(RotaryPositionalEmbeddings):
    """The interleaved rotation with the (cos, sin) table evaluated in double precision and stored in fp32."""

    def _frequencies(self, device) -> torch.Tensor:
        exponent = torch.arange(0, self.dim, 2, device=device, dtype=torch.float64) / self.dim
        return float(self.base) ** (-exponent)

    def build_rope_cache(self, max_seq_len: int = 4096) -> None:
        pos = torch.arange(max_seq_len, dtype=torch.float64, device=self.theta.device)
        angles = torch.outer(pos, self._frequencies(self.theta.device))
        self.register_buffer("cache", torch.stack([angles.cos(), angles.sin()], dim=-1).float(), persistent=False)
        self.is_cache_built = True


class LatentCache(RowCache):
    """Latent rows ``[batch, max_seq_len, width]`` of the tokens seen so far."""

    def __init__(self, batch_size: int, max_seq_len: int, width: int, dtype: torch.dtype) -> None:
        super().__init__(batch_size, max_seq_len)
        self.register_buffer("latent", torch.zeros(batch_size, max_seq_len, width, dtype=dtype), persistent=False)

    def _move_row(self, row: int, to: int) -> None:
        self.latent[to, : self._size].copy_(self.latent[row, : self._size])


class LatentAttention(nn.Module):
    def __init__(
        self,
        *,
        embed_dim: int,
        num_heads: int,
        head_dim: int,
        rot_dim: int,
        value_dim: int,
        kv_rank: int,
        q_proj: nn.Module,
        kv_down: Optional[nn.Module],
        kv_norm: Optional[nn.Module],
        k_up: nn.Module,
        v_up: nn.Module,
        output_proj: nn.Module,
        gate_proj: Optional[nn.Module] = None,
        pos_embeddings: RotaryPositionalEmbeddings,
        scale: float,
        layer_index: int,
        latent_from: Optional[int] = None,
    ) -> None:
        super().__init__()
        if (kv_down is None) != (latent_from is not None) or (kv_down is None) != (kv_norm is None):
            raise ValueError("a layer has either its own latent projection and norm or a layer to take the latents from")
        self.embed_dim, self.num_heads = embed_dim, num_heads
        self.head_dim, self.rot_dim, self.value_dim, self.kv_rank = head_dim, rot_dim, value_dim, kv_rank
        self.q_proj, self.kv_down, self.kv_norm, self.k_up, self.v_up = q_proj, kv_down, kv_norm, k_up, v_up
        self.gate_proj, self.output_proj = gate_proj, output_proj
        self.pos_embeddings = pos_embeddings
        self.scale = float(scale)
        self.layer_index, self.latent_from = layer_index, latent_from
        self.kv_cache: Optional[LatentCache] = None
        self.cache_enabled = False

    # ------------------------------------------------------------------ cache
    def setup_cache(self, batch_size: int, dtype: torch.dtype, max_seq_len: int) -> None:
        if self.kv_cache is not None:
            logger.warning("Key value caches are already setup. You cannot call ``setup_caches()`` twice. Skipping.")
            return
        self._join_projections()
        if self.latent_from is not None:
            return
        self.kv_cache = LatentCache(batch_size, max_seq_len, self.kv_rank + self.rot_dim, dtype)
        home = self.q_proj.weight.device
        if home.type not in ("meta", "cpu") and self.kv_cache.latent.device.type == "cpu":
            self.kv_cache.to(home)
        self.cache_enabled = True

    def reset_cache(self) -> None:
        if self.latent_from is not None:
            return
        if self.kv_cache is None:
            raise RuntimeError("Key value caches are not setup. Call ``setup_caches()`` first.")
        self.kv_cache.reset()

    # ------------------------------------------------------------------ joined weights
    def _inputs(self) -> List[nn.Module]:
        return [m for m in (self.q_proj, self.kv_down, self.gate_proj) if m is not None]

    def _join_projections(self) -> None:
        with torch.no_grad():
            join(self._inputs())
            join([self.k_up, self.v_up])

    # ------------------------------------------------------------------ forward
    def forward(self, x: torch.Tensor, y: Optional[torch.Tensor] = None, *, mask=None, input_pos: Optional[torch.Tensor] = None,
                layer_state: Optional[Dict[Any, Any]] = None) -> torch.Tensor:
        """``layer_state`` is the dictionary the decoder hands to every layer of one forward pass: latents by layer index, and what is
        derived once per pass from ``mask`` and ``input_pos``."""
        if y is not None and y is not x:
            raise ValueError("latent attention is self-attention only")
        state = {} if layer_state is None else layer_state
        if self.latent_from is not None and ("latent", self.latent_from) not in state:
            raise RuntimeError(f"layer {self.layer_index} reads the latents of layer {self.latent_from}, which has not run in this pass")
        if ops.cuda_ops_enabled(x) and x.dtype in (torch.bfloat16, torch.float32):
            if not (torch.is_grad_enabled() and (x.requires_grad or any(p.requires_grad for p in self.parameters()))):
                bounds = kernel_bounds(state, mask, x, self._first_slot(state))
                if bounds is not None:
                    return self._forward_kernels(x, bounds, input_pos, state)
                ops._fallback("latent_attention", "a mask whose rows are not key ranges", x)
            else:
                ops._fallback("latent_attention", "gradients", x)
        return self._forward_statement(x, mask, input_pos, state)

    def _first_slot(self, state: Dict[Any, Any]) -> int:
        if self.latent_from is not None:
            return state["latent", self.latent_from][1]
        return self.kv_cache.size if self.cache_enabled and self.kv_cache is not None else 0

    def _project(self, x2: torch.Tensor) -> Tuple[torch.Tensor, Optional[torch.Tensor], Optional[torch.Tensor]]:
        """Queries, latent input and gate as 2-D tensors with contiguous rows."""
        mods = self._inputs()
        whole = joined(mods)
        if whole is not None:
            parts = ops.linear(x2, whole).split([m.weight.shape[0] for m in mods], dim=1)
        else:
            parts = [m(x2) for m in mods]
        named = dict(zip((id(m) for m in mods), parts))
        return named[id(self.q_proj)], named.get(id(self.kv_down)), named.get(id(self.gate_proj))

    def _forward_kernels(self, x: torch.Tensor, bounds, input_pos: Optional[torch.Tensor], state: Dict[Any, Any]) -> torch.Tensor:
        from ..ops import latent

        b, s, _ = x.shape
        H, d, r, dv, rank = self.num_heads, self.head_dim, self.rot_dim, self.value_dim, self.kv_rank
        q, kv, gate = self._project(x.reshape(b * s, -1))
        pos = positions(state, input_pos, b, s)
        if self.latent_from is None:
            cache = self.kv_cache if self.cache_enabled else None
            if cache is not None:
                first = cache.reserve(b, s)
                buf, slot = cache.latent[:b], cache.slot
            else:
                first, slot = 0, None
                buf = torch.empty(b, s, rank + r, dtype=x.dtype, device=x.device)
        else:
            buf, first, slot, cache = state["latent", self.latent_from]
        decode = s == 1 and cache is not None
        if slot is not None and not decode:
            raise RuntimeError("a cache whose position lives on the device takes one token per step")
        q_lat = torch.empty(b, H, rank + r, dtype=x.dtype, device=x.device) if decode else None
        latent.prepare(q, kv, None if self.kv_norm is None else self.kv_norm.scale, buf, self.pos_embeddings.cache, pos, s=s, slot=slot, slot_host=first, heads=H, dim=d, rot=r,
                       rot_dims=self.pos_embeddings.dim, rank=rank, eps=0.0 if self.kv_norm is None else self.kv_norm.eps, q_out=q_lat)
        if self.latent_from is None:
            state["latent", self.layer_index] = (buf, first, slot, cache)
            if cache is not None:
                cache.advance(s)
        if decode:
            latent.absorb(q, self.k_up.weight if plain(self.k_up) else dense(self.k_up), q_lat, heads=H, dim=d, rot=r, rank=rank)
            keys = first + 1 if slot is None else buf.shape[1]
            o, ml = latent.decode(q_lat, buf, rank=rank, rot=r, scale=self.scale, slot=slot, slot_host=first, bounds=bounds, keys=keys)
            out = latent.value(o, ml, self.v_up.weight if plain(self.v_up) else dense(self.v_up), gate, vdim=dv)
        else:
            sk = first + s
            lat = buf[:, :sk, :rank].reshape(b * sk, rank)
            whole = joined([self.k_up, self.v_up])
            if whole is not None:
                kn, v = ops.linear(lat, whole).split([H * d, H * dv], dim=1)
            else:
                kn, v = self.k_up(lat), self.v_up(lat)
            out = latent.prefill(q, kn, v, buf, gate, b=b, s=s, sk=sk, slot0=first, heads=H, dim=d, rot=r, vdim=dv, rank=rank, scale=self.scale, bounds=bounds)
        return self.output_proj(out.view(b, s, H * dv))

    def _rotate(self, x: torch.Tensor, input_pos: Optional[torch.Tensor], first: int) -> torch.Tensor:
        b, s, dims = x.shape[0], x.shape[1], self.pos_embeddings.dim
        pos = torch.arange(first, first + s, device=x.device) if input_pos is None else input_pos.reshape(-1, s)
        turned = reference.rope_interleaved(x[..., :dims], self.pos_embeddings.cache, pos)
        return turned if dims == x.shape[-1] else torch.cat([turned, x[..., dims:]], dim=-1)

    def _forward_statement(self, x: torch.Tensor, mask, input_pos: Optional[torch.Tensor], state: Dict[Any, Any]) -> torch.Tensor:
        b, s, _ = x.shape
        H, d, r, dv, rank = self.num_heads, self.head_dim, self.rot_dim, self.value_dim, self.kv_rank
        first = self._first_slot(state)
        q = self.q_proj(x).view(b, s, H, d + r)
        q = torch.cat([q[..., :d], self._rotate(q[..., d:], input_pos, first)], dim=-1)
        if self.latent_from is None:
            kv = self.kv_down(x)
            rows = torch.cat([self.kv_norm(kv[..., :rank]), self._rotate(kv[..., rank:].unsqueeze(2), input_pos, first).squeeze(2)], dim=-1)
            cache = self.kv_cache if self.cache_enabled else None
            if cache is not None:
                cache.reserve(b, s)
                cache.latent[:b, first : first + s] = rows
                rows = cache.latent[:b]
                cache.advance(s)
            state["latent", self.layer_index] = (rows, first, None, cache)
        else:
            rows, first, _, cache = state["latent", self.latent_from]
        sk = first + s
        lat, k_rot = rows[:, :sk, :rank], rows[:, :sk, rank:]
        visible = dense_visibility(mask, b, s, sk, first, x.device)
        out = reference.latent_attention(q, self.k_up(lat).view(b, sk, H, d), k_rot, self.v_up(lat).view(b, sk, H, dv), visible, self.scale).reshape(b, s, H * dv)
        if self.gate_proj is not None:
            out = (out.float() * torch.sigmoid(self.gate_proj(x).float())).to(out.dtype)
        return self.output_proj(out)
