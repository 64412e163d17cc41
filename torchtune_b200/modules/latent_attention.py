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
from ..ops.mask import AttentionMask
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


class LatentCache(nn.Module):
    """Latent rows ``[batch, max_seq_len, width]`` of the tokens seen so far; all batch rows append at the same slot.

    ``slot`` is ``None`` (the next slot is known to the host) or a device int32 that holds it, so a captured decode step can be replayed."""

    def __init__(self, batch_size: int, max_seq_len: int, width: int, dtype: torch.dtype) -> None:
        super().__init__()
        self.register_buffer("latent", torch.zeros(batch_size, max_seq_len, width, dtype=dtype), persistent=False)
        self.batch_size = batch_size
        self.max_seq_len = max_seq_len
        self.slot: Optional[torch.Tensor] = None
        self._size = 0

    @property
    def size(self) -> int:
        return self._size

    def reset(self) -> None:
        self._size = 0

    def reserve(self, batch: int, count: int) -> int:
        """Slot of the first of ``count`` new tokens."""
        if batch > self.latent.shape[0]:
            raise ValueError(f"The current cache has been setup with a batch size of {self.latent.shape[0]}, but found new tokens with batch size {batch}!")
        if self._size + count > self.max_seq_len:
            raise AssertionError("KV cache is full: cannot write past max_seq_len")
        return self._size

    def advance(self, count: int) -> None:
        self._size += count

    def rewind(self, size: int) -> None:
        """Forgets the tokens from slot ``size`` on."""
        if not 0 <= size <= self.max_seq_len:
            raise ValueError(f"{size} is outside the cache")
        self._size = size

    def keep_rows(self, rows: List[int]) -> None:
        """Drops every batch row that is not in ``rows`` (increasing) and moves the kept ones to the front."""
        for to, row in enumerate(rows):
            if to != row:
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

    @staticmethod
    def _join(mods: List[nn.Module]) -> None:
        """Lays the weights of plain linears that read the same input out as one matrix (the parameters become views of it), so
        inference multiplies them in one GEMM."""
        weights = [m.weight for m in mods] if all(_plain(m) for m in mods) else []
        if len(weights) < 2 or any(w.device.type == "meta" or hasattr(w, "_grad_buffer") for w in weights) or _joined(mods) is not None:
            return
        whole = torch.cat([w.data for w in weights])
        at = 0
        for w in weights:
            n = w.shape[0]
            w.data = whole[at : at + n]
            at += n

    def _join_projections(self) -> None:
        with torch.no_grad():
            self._join(self._inputs())
            self._join([self.k_up, self.v_up])

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
                bounds = _kernel_bounds(state, mask, x, self._first_slot(state))
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
        whole = _joined(mods)
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
        pos = _positions(state, input_pos, b, s)
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
            latent.absorb(q, self.k_up.weight if _plain(self.k_up) else _dense(self.k_up), q_lat, heads=H, dim=d, rot=r, rank=rank)
            keys = first + 1 if slot is None else buf.shape[1]
            o, ml = latent.decode(q_lat, buf, rank=rank, rot=r, scale=self.scale, slot=slot, slot_host=first, bounds=bounds, keys=keys)
            out = latent.value(o, ml, self.v_up.weight if _plain(self.v_up) else _dense(self.v_up), gate, vdim=dv)
        else:
            sk = first + s
            lat = buf[:, :sk, :rank].reshape(b * sk, rank)
            whole = _joined([self.k_up, self.v_up])
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
        visible = _dense_visibility(mask, b, s, sk, first, x.device)
        out = reference.latent_attention(q, self.k_up(lat).view(b, sk, H, d), k_rot, self.v_up(lat).view(b, sk, H, dv), visible, self.scale).reshape(b, s, H * dv)
        if self.gate_proj is not None:
            out = (out.float() * torch.sigmoid(self.gate_proj(x).float())).to(out.dtype)
        return self.output_proj(out)


def _plain(m: Optional[nn.Module]) -> bool:
    return isinstance(m, nn.Linear) and type(m).__name__ == "Linear" and m.bias is None


def _dense(m: nn.Module) -> torch.Tensor:
    """The matrix an adapted or quantised linear stands for (``[out, in]``)."""
    eye = torch.eye(m.in_dim if hasattr(m, "in_dim") else m.in_features, dtype=next(m.parameters()).dtype, device=next(m.parameters()).device)
    return m(eye).t().contiguous()


def _joined(mods: List[nn.Module]) -> Optional[torch.Tensor]:
    """The one matrix the weights of ``mods`` are consecutive row blocks of, or ``None``."""
    if len(mods) < 2 or not all(_plain(m) for m in mods):
        return None
    w0 = mods[0].weight.data
    at, store = w0.data_ptr(), w0.untyped_storage().data_ptr()
    rows = 0
    for m in mods:
        w = m.weight.data
        if not w.is_contiguous() or w.data_ptr() != at or w.untyped_storage().data_ptr() != store or w.shape[1] != w0.shape[1]:
            return None
        at += w.numel() * w.element_size()
        rows += w.shape[0]
    return torch.as_strided(w0, (rows, w0.shape[1]), (w0.shape[1], 1))


def _positions(state: Dict[Any, Any], input_pos: Optional[torch.Tensor], b: int, s: int) -> Optional[torch.Tensor]:
    if input_pos is None:
        return None
    key = ("positions", input_pos.data_ptr(), tuple(input_pos.shape))
    if key not in state:
        state[key] = (input_pos.reshape(-1, s).expand(b, s).to(torch.int32).contiguous(), input_pos)
    return state[key][0]


def _kernel_bounds(state: Dict[Any, Any], mask, x: torch.Tensor, first: int):
    """Key range of every query for the kernels, once per pass; ``None`` for a boolean mask that is not a set of growing ranges."""
    key = ("bounds", first, id(mask))
    if key not in state:
        state[key] = (_make_bounds(mask, x.shape[0], x.shape[1], first, x.device), mask)
    return state[key][0]


def _make_bounds(mask, b: int, s: int, first: int, device):
    from ..ops._cuda_attention import dense_mask_bounds, lower_bounds
    from ..ops.latent import Bounds

    if mask is None:
        return Bounds()
    if isinstance(mask, AttentionMask) and mask.bool_mask is None:
        if mask.key_start is not None:
            if mask.key_start.numel() != b:
                raise ValueError(f"key_start has {mask.key_start.numel()} rows, the batch has {b}")
            return Bounds(lo=mask.key_start.to(device=device, dtype=torch.int32).contiguous(), lo_row=1)
        if not mask.causal:
            return None
        lo = lower_bounds(mask, b, s, device)
        if lo is None:
            return Bounds()
        return Bounds(lo=lo.contiguous(), lo_row=s, lo_query=1) if first == 0 else None
    dense = mask.bool_mask if isinstance(mask, AttentionMask) else mask
    dense = dense[..., : first + s]
    if dense.dim() == 4 and dense.shape[1] != 1:
        return None
    bits, lo, hi = dense_mask_bounds(dense, b, s, first + s)
    empty = hi < lo
    ranges = bits.sum(-1, dtype=torch.int32) == torch.where(empty, 0, hi - lo + 1)
    growing = ((lo[:, 1:] >= lo[:, :-1]) & (hi[:, 1:] >= hi[:, :-1])).all() if s > 1 else torch.tensor(True, device=device)
    if not bool(ranges.all() & growing):
        return None
    return Bounds(lo=lo, lo_row=s, lo_query=1, hi=hi, hi_row=s, hi_query=1)


def _dense_visibility(mask, b: int, s: int, sk: int, first: int, device) -> torch.Tensor:
    if isinstance(mask, AttentionMask):
        if mask.bool_mask is None and mask.key_start is None and s != sk:
            if mask.doc_ids is not None or mask.chunk > 0 or mask.window > 0:
                raise ValueError("document, chunk and window masks need the whole sequence in one pass")
        else:
            m = mask.dense(b, s, sk, device)
            mask = torch.ones(1, s, sk, dtype=torch.bool, device=device) if m is None else m
    if mask is None or isinstance(mask, AttentionMask):
        return (torch.arange(sk, device=device)[None, :] <= first + torch.arange(s, device=device)[:, None]).unsqueeze(0)
    m = mask[:, 0] if mask.dim() == 4 else mask
    return m[..., :sk]
