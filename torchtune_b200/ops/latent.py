"""CUDA path of attention over latent keys (``csrc/latent_attention.cu``, ``csrc/latent_steps.cu``), inference only.

Tensors may be bf16 or fp32 (``wide``).  bf16 with sizes TMA can address runs on the tensor-core kernels; every other size and all
of fp32 runs :func:`attention_any`.  Row bounds are passed as :class:`Bounds`: key slots ``lo .. hi`` of every query, with strides so
that one value per batch row needs no expansion."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ._lib import check, err_word, lib, stream_ptr

_SMS = None
# from this many decoded rows the per-head products run as grouped tensor-core GEMMs
ABSORB_GROUPED_ROWS = 128
VALUE_GROUPED_ROWS = 32


@dataclass
class Bounds:
    lo: Optional[torch.Tensor] = None  # int32, or None: 0
    lo_row: int = 0
    lo_query: int = 0
    hi: Optional[torch.Tensor] = None  # int32, or None: the query's own slot
    hi_row: int = 0
    hi_query: int = 0


def _p(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _wide(t: torch.Tensor) -> int:
    if t.dtype == torch.float32:
        return 1
    if t.dtype == torch.bfloat16:
        return 0
    raise TypeError(f"latent attention kernels take bf16 or fp32 tensors, not {t.dtype}")


def _pitch(t: torch.Tensor) -> int:
    """Row pitch of a 2-D tensor with contiguous rows."""
    assert t.dim() == 2 and t.stride(1) == 1
    return t.stride(0)


def prepare(q: torch.Tensor, kv: Optional[torch.Tensor], kv_gain: Optional[torch.Tensor], buf: torch.Tensor, table: torch.Tensor, pos: Optional[torch.Tensor], *,
            s: int, slot: Optional[torch.Tensor], slot_host: int, heads: int, dim: int, rot: int, rot_dims: int, rank: int, eps: float,
            q_out: Optional[torch.Tensor] = None) -> None:
    """Normalises the latent, rotates the shared key part and the queries' rotated parts (in place, or into ``q_out`` ``[rows, heads,
    rank + rot]``) and writes the latent rows to ``buf`` ``[b, slots, rank + rot]`` from ``slot`` on."""
    rows = q.shape[0]
    if kv is not None:
        assert kv.shape == (rows, rank + rot) and kv.dtype == q.dtype == buf.dtype == kv_gain.dtype and buf.is_contiguous() and kv_gain.numel() == rank
        assert buf.shape[0] * s >= rows and buf.shape[2] == rank + rot
    assert q.shape[1] == heads * (dim + rot) and table.dtype == torch.float32 and table.is_contiguous() and table.shape[1] * 2 == rot_dims
    assert pos is None or (pos.dtype == torch.int32 and pos.is_contiguous() and pos.numel() == rows)
    assert q_out is None or (q_out.is_contiguous() and q_out.shape == (rows, heads, rank + rot) and q_out.dtype == q.dtype)
    check(lib().ttb_latent_prepare(_p(kv), 0 if kv is None else _pitch(kv), _p(kv_gain), q.data_ptr(), _pitch(q), _p(q_out), _p(buf) if kv is not None else None, table.data_ptr(), _p(pos),
                                   _p(slot), int(slot_host), rows, s, buf.shape[1], heads, dim, rot, rot_dims, rank, table.shape[0], float(eps), _wide(q), stream_ptr()),
          "latent_prepare")


def prefill_supported(q: torch.Tensor, dim: int, rot: int, vdim: int, rank: int) -> bool:
    """Sizes the tensor-core prefill kernel takes: bf16, all widths multiples of 8 (16-byte rows), at most four key and two value panels."""
    return (q.dtype == torch.bfloat16 and dim % 8 == rot % 8 == vdim % 8 == rank % 8 == 0 and -(-dim // 64) + -(-rot // 64) <= 4 and vdim <= 128
            and _pitch(q) % 8 == 0 and q.data_ptr() % 16 == 0)


def prefill(q: torch.Tensor, kn: torch.Tensor, v: torch.Tensor, buf: torch.Tensor, gate: Optional[torch.Tensor], *, b: int, s: int, sk: int, slot0: int,
            heads: int, dim: int, rot: int, vdim: int, rank: int, scale: float, bounds: Bounds) -> torch.Tensor:
    """``softmax((q_n · k_n + q_r · k_r) · scale) v``, times the sigmoid of ``gate``.  ``q`` ``[b·s, heads·(dim+rot)]``, ``kn`` / ``v``
    ``[b·sk, heads·dim | heads·vdim]`` (row pitches free), rotated key parts read from ``buf``."""
    assert kn.shape == (b * sk, heads * dim) and v.shape == (b * sk, heads * vdim) and q.shape == (b * s, heads * (dim + rot)) and sk <= buf.shape[1]
    assert gate is None or (gate.shape == (b * s, heads * vdim) and gate.dtype == q.dtype)
    out = torch.empty(b * s, heads * vdim, dtype=q.dtype, device=q.device)
    width = rank + rot
    kr_ptr = buf.data_ptr() + rank * buf.element_size()
    if prefill_supported(q, dim, rot, vdim, rank):
        check(lib().ttb_latent_prefill(q.data_ptr(), _pitch(q), kn.data_ptr(), _pitch(kn), kr_ptr, width, buf.shape[1] * width, v.data_ptr(), _pitch(v), _p(gate),
                                       0 if gate is None else _pitch(gate), out.data_ptr(), b, s, sk, heads, dim, rot, vdim, slot0, _p(bounds.lo), bounds.lo_row, bounds.lo_query,
                                       _p(bounds.hi), bounds.hi_row, bounds.hi_query, float(scale), err_word(q.device).data_ptr(), stream_ptr()), "latent_prefill")
        return out
    check(lib().ttb_latent_attention_any(q.data_ptr(), s * _pitch(q), _pitch(q), dim + rot, kn.data_ptr(), sk * _pitch(kn), _pitch(kn), dim, kr_ptr, buf.shape[1] * width, width,
                                         v.data_ptr(), sk * _pitch(v), _pitch(v), vdim, out.data_ptr(), None, _p(gate), 0 if gate is None else _pitch(gate), b, s, sk, heads, 1, dim, rot, vdim,
                                         0, 0, None, slot0, _p(bounds.lo), bounds.lo_row, bounds.lo_query, _p(bounds.hi), bounds.hi_row, bounds.hi_query, float(scale), _wide(q),
                                         stream_ptr()), "latent_attention_any (prefill)")
    return out


def decode_supported(q: torch.Tensor, rank: int, rot: int) -> bool:
    return q.dtype == torch.bfloat16 and rank % 8 == 0 and rot % 8 == 0 and rank <= 512 and rot <= 128


def split_count(b: int, heads: int, rank: int, rot: int, keys: int) -> int:
    """Key ranges per (batch row, head group): enough CTAs for one per SM, at least one tile of keys each."""
    global _SMS
    if _SMS is None:
        _SMS = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    groups = 1 if heads <= 16 else -(-heads // 32)
    return max(1, min(-(-keys // lib().ttb_latent_decode_tile(heads, rank, rot)), _SMS // (b * groups)))


def absorb(q: torch.Tensor, w_uk: torch.Tensor, q_lat: torch.Tensor, *, heads: int, dim: int, rot: int, rank: int) -> None:
    """``q_lat[:, h, :rank] = W_uk[h]ᵀ q_n[h]`` for ``q`` ``[rows, heads·(dim+rot)]``."""
    rows = q.shape[0]
    assert w_uk.shape == (heads * dim, rank) and w_uk.is_contiguous() and w_uk.dtype == q.dtype and q_lat.shape == (rows, heads, rank + rot)
    if q.dtype == torch.bfloat16 and rows >= ABSORB_GROUPED_ROWS and dim % 8 == 0 and rank % 8 == 0:
        from ._cuda import _grouped_gemm

        a = q.view(rows, heads, dim + rot)[:, :, :dim].transpose(0, 1).reshape(heads * rows, dim)
        q_lat[:, :, :rank].copy_(_grouped_gemm(a, w_uk.view(heads, dim, rank), _head_counts(heads, rows, q.device), b_mn=True).view(heads, rows, rank).transpose(0, 1))
        return
    check(lib().ttb_latent_absorb(q.data_ptr(), _pitch(q), dim + rot, w_uk.data_ptr(), q_lat.data_ptr(), heads * (rank + rot), rank + rot, rows, heads, dim, rank, _wide(q), stream_ptr()),
          "latent_absorb")


_counts = {}


def _head_counts(heads: int, rows: int, device) -> torch.Tensor:
    key = (heads, rows, device)
    if key not in _counts:
        if len(_counts) > 256:
            _counts.clear()
        _counts[key] = torch.full((heads,), rows, dtype=torch.int64, device=device)
    return _counts[key]


def decode(q_lat: torch.Tensor, buf: torch.Tensor, *, rank: int, rot: int, scale: float, slot: Optional[torch.Tensor], slot_host: int, bounds: Bounds,
           keys: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """One query per batch row against the cached latents.  Returns fp32 partials ``o [splits, b, heads, rank]`` and ``ml [splits, b,
    heads, 2]``; ``keys`` bounds the visible key count (it sizes the split)."""
    b, heads, width = q_lat.shape
    assert width == rank + rot and buf.shape[0] >= b and buf.shape[2] == width and buf.is_contiguous() and buf.dtype == q_lat.dtype and q_lat.is_contiguous()
    slots = buf.shape[1]
    if decode_supported(q_lat, rank, rot):
        splits = split_count(b, heads, rank, rot, keys)
        o = torch.empty(splits, b, heads, rank, dtype=torch.float32, device=q_lat.device)
        ml = torch.empty(splits, b, heads, 2, dtype=torch.float32, device=q_lat.device)
        check(lib().ttb_latent_decode(q_lat.data_ptr(), buf.data_ptr(), o.data_ptr(), ml.data_ptr(), b, heads, rank, rot, slots, splits, _p(slot), int(slot_host), _p(bounds.lo),
                                      bounds.lo_row, _p(bounds.hi), bounds.hi_row, float(scale), err_word(q_lat.device).data_ptr(), stream_ptr()), "latent_decode")
        return o, ml
    o = torch.empty(1, b, heads, rank, dtype=torch.float32, device=q_lat.device)
    ml = torch.empty(1, b, heads, 2, dtype=torch.float32, device=q_lat.device)
    c = buf.data_ptr()
    check(lib().ttb_latent_attention_any(q_lat.data_ptr(), heads * width, 0, width, c, slots * width, width, 0, c + rank * buf.element_size(), slots * width, width, c, slots * width, width, 0,
                                         o.data_ptr(), ml.data_ptr(), None, 0, b, 1, slots, heads, heads, rank, rot, rank, 1, 1, _p(slot), int(slot_host), _p(bounds.lo), bounds.lo_row, 0,
                                         _p(bounds.hi), bounds.hi_row, 0, float(scale), _wide(q_lat), stream_ptr()), "latent_attention_any (decode)")
    return o, ml


def value(o: torch.Tensor, ml: torch.Tensor, w_uv: torch.Tensor, gate: Optional[torch.Tensor], *, vdim: int) -> torch.Tensor:
    """Combines the key ranges and applies ``W_uv`` per head and the gate; ``[rows, heads·vdim]`` in the weight's dtype."""
    splits, rows, heads, rank = o.shape
    assert w_uv.shape == (heads * vdim, rank) and w_uv.is_contiguous() and (gate is None or gate.shape == (rows, heads * vdim))
    out = torch.empty(rows, heads * vdim, dtype=w_uv.dtype, device=o.device)
    gate_ld = 0 if gate is None else _pitch(gate)
    if w_uv.dtype == torch.bfloat16 and rows >= VALUE_GROUPED_ROWS and vdim % 8 == 0 and rank % 8 == 0:
        from ._cuda import _grouped_gemm

        lat = torch.empty(heads * rows, rank, dtype=torch.bfloat16, device=o.device)
        check(lib().ttb_latent_combine(o.data_ptr(), ml.data_ptr(), lat.data_ptr(), splits, rows, heads, rank, 1, stream_ptr()), "latent_combine")
        y = _grouped_gemm(lat, w_uv.view(heads, vdim, rank), _head_counts(heads, rows, o.device), b_mn=False)
        check(lib().ttb_latent_gate_rows(y.data_ptr(), _p(gate), gate_ld, out.data_ptr(), rows, heads, vdim, stream_ptr()), "latent_gate_rows")
        return out
    if splits > 1:
        o1 = torch.empty(rows, heads, rank, dtype=torch.float32, device=o.device)
        check(lib().ttb_latent_combine(o.data_ptr(), ml.data_ptr(), o1.data_ptr(), splits, rows, heads, rank, 0, stream_ptr()), "latent_combine")
        o, ml = o1, None
    check(lib().ttb_latent_value(o.data_ptr(), _p(ml), w_uv.data_ptr(), _p(gate), gate_ld, out.data_ptr(), rows, heads, rank, vdim, _wide(w_uv), stream_ptr()), "latent_value")
    return out


def residual_norm(x: torch.Tensor, y: Optional[torch.Tensor], w_post: Optional[torch.Tensor], w_next: Optional[torch.Tensor], eps: float, mult: float,
                  offset: float) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``x' = x + mult · norm(y; w_post)`` and ``norm(x'; w_next)`` in one pass (``csrc/residual_norm.cu``)."""
    D = x.shape[-1]
    w = w_post if w_post is not None else w_next
    x2 = x.reshape(-1, D)
    x2 = x2 if x2.is_contiguous() else x2.contiguous()
    y2 = None
    if y is not None:
        y2 = y.reshape(-1, D)
        y2 = y2 if y2.is_contiguous() else y2.contiguous()
        assert y2.dtype == w.dtype and y2.shape == x2.shape
    assert x2.dtype == torch.float32 and all(g is None or (g.dtype == w.dtype and g.numel() == D and g.is_contiguous()) for g in (w_post, w_next))
    out = torch.empty_like(x2) if y is not None else x2
    h = torch.empty(x2.shape, dtype=w.dtype, device=x.device) if w_next is not None else None
    check(lib().ttb_residual_norm(x2.data_ptr(), _p(y2), _p(w_post), out.data_ptr(), _p(w_next), _p(h), x2.shape[0], D, float(eps), float(mult), float(offset), _wide(w), stream_ptr()),
          "residual_norm")
    return out.view(x.shape), None if h is None else h.view(x.shape)
