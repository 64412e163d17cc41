"""What the cached mixers (attention over key ranges, recurrent layers) share: joined projection weights, and positions, key ranges and row
starts derived once per forward pass from the mask."""
from __future__ import annotations

from typing import Any, Dict, List, Optional

import torch
from torch import nn

from ..ops.mask import AttentionMask


def plain(m: Optional[nn.Module]) -> bool:
    return isinstance(m, nn.Linear) and type(m).__name__ == "Linear" and m.bias is None


def dense(m: nn.Module) -> torch.Tensor:
    """The matrix an adapted or quantised linear stands for (``[out, in]``)."""
    eye = torch.eye(m.in_dim if hasattr(m, "in_dim") else m.in_features, dtype=next(m.parameters()).dtype, device=next(m.parameters()).device)
    return m(eye).t().contiguous()


def join(mods: List[nn.Module]) -> None:
    """Lays the weights of plain linears that read the same input out as one matrix (the parameters become views of it), so inference
    multiplies them in one GEMM."""
    weights = [m.weight for m in mods] if all(plain(m) for m in mods) else []
    if len(weights) < 2 or any(w.device.type == "meta" or hasattr(w, "_grad_buffer") for w in weights) or joined(mods) is not None:
        return
    whole = torch.cat([w.data for w in weights])
    at = 0
    for w in weights:
        n = w.shape[0]
        w.data = whole[at : at + n]
        at += n


def joined(mods: List[nn.Module]) -> Optional[torch.Tensor]:
    """The one matrix the weights of ``mods`` are consecutive row blocks of, or ``None``."""
    if len(mods) < 2 or not all(plain(m) for m in mods):
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


def positions(state: Dict[Any, Any], input_pos: Optional[torch.Tensor], b: int, s: int) -> Optional[torch.Tensor]:
    if input_pos is None:
        return None
    key = ("positions", input_pos.data_ptr(), tuple(input_pos.shape))
    if key not in state:
        state[key] = (input_pos.reshape(-1, s).expand(b, s).to(torch.int32).contiguous(), input_pos)
    return state[key][0]


def kernel_bounds(state: Dict[Any, Any], mask, x: torch.Tensor, first: int):
    """Key range of every query for the kernels, once per pass; ``None`` for a boolean mask that is not a set of growing ranges."""
    key = ("bounds", first, id(mask))
    if key not in state:
        state[key] = (make_bounds(mask, x.shape[0], x.shape[1], first, x.device), mask)
    return state[key][0]


def make_bounds(mask, b: int, s: int, first: int, device):
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


def dense_visibility(mask, b: int, s: int, sk: int, first: int, device) -> torch.Tensor:
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


def row_starts(state: Dict[Any, Any], mask, b: int, s: int, first: int, device) -> Optional[torch.Tensor]:
    """First own slot of every row (int32), once per pass; ``None``: all rows start at slot 0.  A recurrent layer has no other masks than
    causal ones over left-padded rows."""
    key = ("starts", first, id(mask))
    if key not in state:
        state[key] = (_row_starts(mask, b, s, first, device), mask)
    return state[key][0]


def _row_starts(mask, b: int, s: int, first: int, device) -> Optional[torch.Tensor]:
    if mask is None:
        return None
    if isinstance(mask, AttentionMask) and mask.bool_mask is None:
        if not mask.causal or mask.doc_ids is not None or mask.chunk > 0 or mask.window > 0:
            raise ValueError("a recurrent layer takes causal masks over whole rows only")
        if mask.key_start is None:
            return None
        if mask.key_start.numel() != b:
            raise ValueError(f"key_start has {mask.key_start.numel()} rows, the batch has {b}")
        return mask.key_start.to(device=device, dtype=torch.int32).contiguous()
    m = mask.bool_mask if isinstance(mask, AttentionMask) else mask
    m = (m[:, 0] if m.dim() == 4 else m)[..., : first + s].to(torch.bool).expand(b, s, first + s)
    start = m[:, -1].to(torch.int8).argmax(-1)  # the last token of a row sees the row from its first token on
    j, own = torch.arange(first + s, device=device), first + torch.arange(s, device=device)
    rows = (j[None, None, :] <= own[None, :, None]) & (j[None, None, :] >= start[:, None, None])
    if not bool((m == rows)[own[None, :].expand(b, s) >= start[:, None]].all()):
        raise ValueError("a recurrent layer takes causal masks over whole rows only")
    return start.to(torch.int32)
