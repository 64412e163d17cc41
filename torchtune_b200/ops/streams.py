"""CUDA path of the steps on several residual streams (``csrc/streams.cu``), inference only; tensors may be bf16 or fp32 (``wide``)."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ._lib import check, lib, stream_ptr
from .latent import _p, _wide


def stream_step(x: torch.Tensor, y: Optional[torch.Tensor], gain: Optional[torch.Tensor], mix: Optional[torch.Tensor], out: Optional[torch.Tensor], read: Optional[torch.Tensor],
                w_next: Optional[torch.Tensor], eps: float, centered: bool, offset: float, keep: bool) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
    """``x`` ``[..., S | 1, D]`` fp32; see :func:`torchtune_b200.ops.stream_step`."""
    lead, (given, D) = x.shape[:-2], x.shape[-2:]
    w = w_next if w_next is not None else gain
    S = mix.shape[0] if mix is not None else (read.numel() if read is not None else given)
    x3 = x.reshape(-1, given, D)
    x3 = x3 if x3.is_contiguous() else x3.contiguous()
    rows = x3.shape[0]
    assert given in (1, S) and all(t is None or (t.dtype == w.dtype and t.is_contiguous()) for t in (gain, mix, out, read, w_next))
    assert (gain is None or gain.numel() == D) and (w_next is None or w_next.numel() == D) and (out is None or out.numel() == S) and (mix is None or mix.shape == (S, S))
    after = x3
    if y is not None:
        y = y.reshape(rows, D)
        y = y if y.is_contiguous() else y.contiguous()
        after = torch.empty(rows, S, D, dtype=torch.float32, device=x.device) if keep or w_next is None else None
    h = None if w_next is None else torch.empty(rows, D, dtype=w.dtype, device=x.device)
    check(lib().ttb_stream_step(x3.data_ptr(), given, _p(y), _p(gain), _p(mix), _p(out), None if y is None else _p(after), _p(read), _p(w_next), _p(h), rows, D, S, float(eps),
                                float(offset), int(centered), _wide(w), stream_ptr()), "stream_step")
    return None if after is None else after.view(*lead, after.shape[1], D), None if h is None else h.view(*lead, D)


def embed_positions(tokens: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, pos_table: torch.Tensor) -> torch.Tensor:
    n, D = tokens.numel(), table.shape[1]
    assert table.is_contiguous() and pos_table.is_contiguous() and pos_table.shape[1] == D and positions.numel() == n
    ids, pos = tokens.to(torch.int64).contiguous(), positions.to(torch.int64).contiguous()
    out = torch.empty(n, D, dtype=torch.float32, device=table.device)
    check(lib().ttb_embed_positions(ids.data_ptr(), pos.data_ptr(), table.data_ptr(), pos_table.data_ptr(), out.data_ptr(), n, D, table.shape[0], pos_table.shape[0], _wide(table),
                                    stream_ptr()), "embed_positions")
    return out.view(*tokens.shape, D)


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float, alpha: float) -> torch.Tensor:
    H = gate.shape[-1]
    g, u = gate.reshape(-1, H), up.reshape(-1, H)
    assert g.stride(1) == 1 and u.stride(1) == 1
    out = torch.empty(g.shape, dtype=g.dtype, device=g.device)
    check(lib().ttb_clamped_glu(g.data_ptr(), u.data_ptr(), out.data_ptr(), g.shape[0], H, g.stride(0), u.stride(0), float(limit), float(alpha), _wide(g), stream_ptr()), "clamped_glu")
    return out.view(gate.shape)
