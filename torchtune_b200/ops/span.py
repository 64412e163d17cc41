"""CUDA path of grouped-query attention over key ranges of a cache (``csrc/span_steps.cu``, ``csrc/latent_attention.cu``), inference only.

Tensors may be bf16 or fp32.  bf16 with sizes TMA can address runs on the tensor-core kernels; every other size and all of fp32 runs the
kernel for any size.  Key ranges are passed as :class:`~torchtune_b200.ops.latent.Bounds`."""
from __future__ import annotations

from typing import Optional

import torch

from ._lib import check, err_word, lib, stream_ptr
from .latent import Bounds, _p, _pitch, _wide

_SMS = None


def prepare(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, q_gain: Optional[torch.Tensor], k_gain: Optional[torch.Tensor], keys: torch.Tensor, values: torch.Tensor,
            pos: Optional[torch.Tensor], *, s: int, slot: Optional[torch.Tensor], slot_host: int, eps: float, coef: float, every: int) -> torch.Tensor:
    """Norms the projections (``q`` in place, ``k`` into the cache), applies the query temperature ``1 + coef · ln(⌊(pos + 1) / every⌋ + 1)`` and
    writes keys and values ``[b, slots, heads, dim]`` from ``slot`` on.  Returns ``q``."""
    rows, slots = q.shape[0], keys.shape[1]
    kw, vw = keys.shape[2] * keys.shape[3], values.shape[2] * values.shape[3]
    assert k.shape == (rows, kw) and v.shape == (rows, vw) and q.dtype == k.dtype == v.dtype == keys.dtype == values.dtype and keys.is_contiguous() and values.is_contiguous()
    assert keys.shape[0] * s >= rows and values.shape[:2] == keys.shape[:2] and (pos is None or (pos.dtype == torch.int32 and pos.is_contiguous() and pos.numel() == rows))
    assert q_gain is None or (q_gain.numel() == q.shape[1] and k_gain.numel() == kw and q_gain.dtype == k_gain.dtype == q.dtype)
    check(lib().ttb_span_prepare(q.data_ptr(), _pitch(q), k.data_ptr(), _pitch(k), v.data_ptr(), _pitch(v), _p(q_gain), _p(k_gain), keys.data_ptr(), values.data_ptr(), _p(pos), _p(slot),
                                 int(slot_host), rows, s, slots, q.shape[1], kw, vw, float(eps), float(coef), int(every), _wide(q), stream_ptr()), "span_prepare")
    return q


def prefill_supported(q: torch.Tensor, dim: int, vdim: int) -> bool:
    """Sizes the tensor-core prefill kernel takes: bf16, head sizes multiples of 8 (16-byte rows), keys up to 256 and values up to 128 wide."""
    return q.dtype == torch.bfloat16 and dim % 8 == vdim % 8 == 0 and dim <= 256 and vdim <= 128 and _pitch(q) % 8 == 0 and q.data_ptr() % 16 == 0


def prefill(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, *, b: int, s: int, sk: int, slot0: int, heads: int, scale: float, bounds: Bounds) -> torch.Tensor:
    """``softmax(q · k · scale) v`` for ``s`` queries per row in the slots from ``slot0`` on, against the first ``sk`` slots; ``[b·s, heads·vdim]``."""
    slots, G, dim = keys.shape[1:]
    vdim = values.shape[3]
    assert q.shape == (b * s, heads * dim) and heads % G == 0 and sk <= slots and keys.shape[0] == values.shape[0] == b and keys.is_contiguous() and values.is_contiguous()
    out = torch.empty(b * s, heads * vdim, dtype=q.dtype, device=q.device)
    if prefill_supported(q, dim, vdim):
        check(lib().ttb_span_prefill(q.data_ptr(), _pitch(q), keys.data_ptr(), values.data_ptr(), out.data_ptr(), b, s, sk, slots, heads, G, dim, vdim, slot0, _p(bounds.lo), bounds.lo_row,
                                     bounds.lo_query, _p(bounds.hi), bounds.hi_row, bounds.hi_query, float(scale), err_word(q.device).data_ptr(), stream_ptr()), "span_prefill")
        return out
    _any(q.data_ptr(), s * _pitch(q), _pitch(q), keys, values, out, b, s, sk, heads, 0, None, slot0, bounds, scale)
    return out


def _any(q_ptr: int, q_batch: int, q_row: int, keys: torch.Tensor, values: torch.Tensor, out: torch.Tensor, b: int, s: int, sk: int, heads: int, heads_as_rows: int,
         slot: Optional[torch.Tensor], slot_host: int, bounds: Bounds, scale: float) -> None:
    slots, G, dim = keys.shape[1:]
    vdim = values.shape[3]
    kp, vp = keys.data_ptr(), values.data_ptr()
    check(lib().ttb_latent_attention_any(q_ptr, q_batch, q_row, dim, kp, slots * G * dim, G * dim, dim, kp, 0, 0, vp, slots * G * vdim, G * vdim, vdim, out.data_ptr(), None, None, 0, b, s, sk,
                                         heads, heads // G, dim, 0, vdim, heads_as_rows, 0, _p(slot), int(slot_host), _p(bounds.lo), bounds.lo_row, bounds.lo_query, _p(bounds.hi),
                                         bounds.hi_row, bounds.hi_query, float(scale), _wide(keys), stream_ptr()), "latent_attention_any (span)")


def decode_supported(q: torch.Tensor, dim: int, vdim: int) -> bool:
    return q.dtype == torch.bfloat16 and dim % 8 == vdim % 8 == 0 and dim <= 256 and vdim <= 512 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0


def split_count(b: int, G: int, group: int, dim: int, vdim: int, keys: int) -> int:
    """Key ranges per (batch row, key head): enough CTAs for one per SM, at least one tile of keys each."""
    global _SMS
    if _SMS is None:
        _SMS = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    ctas = G * (1 if group <= 16 else -(-group // 32))
    return max(1, min(-(-keys // lib().ttb_span_decode_tile(group, dim, vdim)), _SMS // (b * ctas)))


def decode(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, *, scale: float, slot: Optional[torch.Tensor], slot_host: int, bounds: Bounds, keys_visible: int) -> torch.Tensor:
    """One query per batch row, ``q`` ``[b, heads, dim]`` with its own row pitch; ``keys_visible`` bounds the number of visible keys (it sizes the
    split).  Returns ``[b, heads·vdim]``."""
    b, heads, dim = q.shape
    slots, G = keys.shape[1:3]
    vdim = values.shape[3]
    assert heads % G == 0 and keys.shape[0] == b and keys.shape[3] == dim and q.stride(2) == 1 and q.stride(1) == dim and keys.is_contiguous() and values.is_contiguous() and q.dtype == keys.dtype
    out = torch.empty(b, heads * vdim, dtype=q.dtype, device=q.device)
    if decode_supported(q, dim, vdim):
        splits = split_count(b, G, heads // G, dim, vdim, keys_visible)
        o = torch.empty(splits, b, heads, vdim, dtype=torch.float32, device=q.device)
        ml = torch.empty(splits, b, heads, 2, dtype=torch.float32, device=q.device)
        check(lib().ttb_span_decode(q.data_ptr(), q.stride(0), keys.data_ptr(), values.data_ptr(), o.data_ptr(), ml.data_ptr(), b, heads, G, dim, vdim, slots, splits, _p(slot), int(slot_host),
                                    _p(bounds.lo), bounds.lo_row, _p(bounds.hi), bounds.hi_row, float(scale), err_word(q.device).data_ptr(), stream_ptr()), "span_decode")
        check(lib().ttb_latent_combine(o.data_ptr(), ml.data_ptr(), out.data_ptr(), splits, b, heads, vdim, 2, stream_ptr()), "latent_combine")
        return out
    _any(q.data_ptr(), q.stride(0), 0, keys, values, out, b, 1, slots, heads, 1, slot, slot_host, bounds, scale)
    return out
