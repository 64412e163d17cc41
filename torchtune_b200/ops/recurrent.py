"""CUDA path of linear attention with a fixed decay per head (``csrc/lightning.cu``), inference only.

Several tokens per row run in tensor-core chunks (bf16, head sizes multiples of 8 up to 128); every other size, few tokens and all of fp32
run token by token with the state in registers."""
from __future__ import annotations

from typing import Dict, Optional, Sequence, Tuple

import torch

from . import reference
from ._lib import check, err_word, lib, stream_ptr
from .latent import _p, _pitch, _wide

CHUNK = 128
# from this many tokens per row the chunked kernels run
MIN_CHUNKED = 17
_SMS = None
_tables: Dict[Tuple, torch.Tensor] = {}


def _table(decay: Sequence[float], step: int, count: int, device: torch.device) -> torch.Tensor:
    """``decay ** (0, step, 2·step, …)`` per head as fp32 ``[heads, count]``, evaluated in double precision."""
    key = (tuple(decay), step, count, device)
    if key not in _tables:
        if len(_tables) > 512:
            _tables.clear()
        _tables[key] = reference.decay_powers([d**step for d in decay], count).float().to(device).contiguous()
    return _tables[key]


def _decays(decay: Sequence[float], device: torch.device) -> torch.Tensor:
    key = (tuple(decay), device)
    if key not in _tables:
        _tables[key] = torch.tensor(decay, dtype=torch.float64).float().to(device)
    return _tables[key]


def chunks_supported(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, dim: int, vdim: int) -> bool:
    return q.dtype == torch.bfloat16 and dim % 8 == vdim % 8 == 0 and dim <= 128 and vdim <= 128 and all(_pitch(t) % 8 == 0 and t.data_ptr() % 16 == 0 for t in (q, k, v))


def run_chunks(b: int, s: int, heads: int) -> int:
    """Chunks per run: as many runs as fit on the SMs at once."""
    global _SMS
    if _SMS is None:
        _SMS = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    chunks = -(-s // CHUNK)
    return -(-chunks // max(1, _SMS // (b * heads)))


def _silu(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> None:
    """In place; one launch when the three are column blocks of one matrix."""
    size, ld = q.element_size(), _pitch(q)
    together = ld == _pitch(k) == _pitch(v) and k.data_ptr() == q.data_ptr() + q.shape[1] * size and v.data_ptr() == k.data_ptr() + k.shape[1] * size
    for t, width in [(q, q.shape[1] + k.shape[1] + v.shape[1])] if together else [(t, t.shape[1]) for t in (q, k, v)]:
        check(lib().ttb_silu_rows(t.data_ptr(), t.shape[0], _pitch(t), width, stream_ptr()), "silu_rows")


def lightning(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: Sequence[float], state: Optional[torch.Tensor], *, b: int, s: int, heads: int, dim: int, vdim: int, fresh: bool,
              starts: Optional[torch.Tensor], first: int) -> torch.Tensor:
    """SiLU of the three projections (in place where the chunked kernels run), then the recurrence: ``q`` / ``k`` ``[b·s, heads·dim]``, ``v``
    ``[b·s, heads·vdim]``, ``state`` ``[b, heads, dim, vdim]`` fp32 read (unless ``fresh``) and replaced.  Tokens in slots in front of ``starts`` leave
    nothing in the state; token 0 sits in slot ``first``.  Returns ``[b·s, heads·vdim]``, fp32 from the token-by-token kernel, else bf16."""
    assert q.shape == k.shape == (b * s, heads * dim) and v.shape == (b * s, heads * vdim) and q.dtype == k.dtype == v.dtype and len(decay) == heads
    assert state is None or (state.shape == (b, heads, dim, vdim) and state.dtype == torch.float32 and state.is_contiguous())
    assert state is not None or fresh
    if s >= MIN_CHUNKED and chunks_supported(q, k, v, dim, vdim):
        _silu(q, k, v)
        per = run_chunks(b, s, heads)
        runs = -(-(-(-s // CHUNK)) // per)
        powers, chunk_powers = _table(decay, 1, CHUNK + 1, q.device), _table(decay, CHUNK, per + 1, q.device)
        work = torch.empty(b, heads, runs, dim, vdim, dtype=torch.float32, device=q.device) if runs > 1 else None
        out = torch.empty(b * s, heads * vdim, dtype=q.dtype, device=q.device)
        check(lib().ttb_lightning_chunks(q.data_ptr(), _pitch(q), k.data_ptr(), _pitch(k), v.data_ptr(), _pitch(v), powers.data_ptr(), chunk_powers.data_ptr(), _p(state), _p(work),
                                         out.data_ptr(), b, s, heads, dim, vdim, per, int(fresh), _p(starts), int(first), err_word(q.device).data_ptr(), stream_ptr()), "lightning_chunks")
        return out
    out = torch.empty(b * s, heads * vdim, dtype=torch.float32, device=q.device)
    check(lib().ttb_lightning_recurrent(q.data_ptr(), _pitch(q), k.data_ptr(), _pitch(k), v.data_ptr(), _pitch(v), _decays(decay, q.device).data_ptr(), _p(state),
                                        out.data_ptr(), b, s, heads, dim, vdim, int(fresh), _p(starts), int(first), _wide(q), stream_ptr()), "lightning_recurrent")
    return out


def gated_norm(o: torch.Tensor, gain: torch.Tensor, gate: torch.Tensor, eps: float) -> torch.Tensor:
    """``o / rms(o) · gain · sigmoid(gate)`` in the gain's dtype; ``o`` ``[rows, width]`` fp32 or of that dtype."""
    rows, width = o.shape
    assert o.is_contiguous() and gain.numel() == width and gate.shape == (rows, width) and gate.dtype == gain.dtype and o.dtype in (torch.float32, gain.dtype)
    out = torch.empty(rows, width, dtype=gain.dtype, device=o.device)
    check(lib().ttb_gated_norm(o.data_ptr(), int(o.dtype == torch.float32), gain.data_ptr(), gate.data_ptr(), _pitch(gate), out.data_ptr(), rows, width, float(eps), _wide(gain),
                               stream_ptr()), "gated_norm")
    return out
