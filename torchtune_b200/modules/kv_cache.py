"""Key/value cache for incremental decoding (parity: torchtune/modules/kv_cache.py:11-116).

Buffers are laid out ``[batch, max_seq_len, num_kv_heads, head_dim]`` — the layout the
attention kernels consume — rather than head-major.
"""
from __future__ import annotations

from typing import Any, Iterator, List, Optional, Sequence, Tuple

import torch
from torch import nn


class KVCache(nn.Module):
    def __init__(self, batch_size: int, max_seq_len: int, num_kv_heads: int, head_dim: int, dtype: torch.dtype) -> None:
        super().__init__()
        shape = (batch_size, max_seq_len, num_kv_heads, head_dim)
        self.register_buffer("k_cache", torch.zeros(shape, dtype=dtype), persistent=False)
        self.register_buffer("v_cache", torch.zeros(shape, dtype=dtype), persistent=False)
        # positions of the *next* writes; kept as a tensor so updates are pure tensor ops
        self.register_buffer("cache_pos", torch.arange(0, max_seq_len), persistent=False)
        self.batch_size = batch_size
        self.max_seq_len = max_seq_len

    def reset(self) -> None:
        self.k_cache.zero_()
        self.v_cache.zero_()
        self.cache_pos -= self.size

    @property
    def size(self) -> int:
        return int(self.cache_pos[0].item())

    def update(self, k_val: torch.Tensor, v_val: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """Append ``[b, s, n_kv, d]`` keys/values and return the full buffers."""
        bsz, seq_len = k_val.shape[0], k_val.shape[1]
        if bsz > self.k_cache.shape[0]:
            raise ValueError(
                f"The current cache has been setup with a batch size of {self.k_cache.shape[0]}"
                f", but found new key tensors with batch size {bsz}!"
            )
        if self.cache_pos[0] + seq_len > self.max_seq_len:
            raise AssertionError("KV cache is full: cannot write past max_seq_len")
        where = self.cache_pos[:seq_len]
        self.k_cache[:bsz].index_copy_(1, where, k_val)
        self.v_cache[:bsz].index_copy_(1, where, v_val)
        self.cache_pos.add_(seq_len)
        return self.k_cache[:bsz], self.v_cache[:bsz]


class RowCache(nn.Module):
    """What a layer keeps of the tokens seen so far, for batch rows that all append at the same slot.

    ``slot`` is ``None`` (the next slot is known to the host) or a device int32 that holds it, so a captured decode step can be replayed.
    Subclasses say how one row is moved to another place and, where appending changes more than new slots, how to save and restore it."""

    def __init__(self, batch_size: int, max_seq_len: int) -> None:
        super().__init__()
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
        if batch > self.batch_size:
            raise ValueError(f"The current cache has been setup with a batch size of {self.batch_size}, but found new tokens with batch size {batch}!")
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

    def snapshot(self) -> Any:
        """What :meth:`restore` needs to undo the steps taken in between."""
        return self._size

    def restore(self, saved: Any) -> None:
        self._size = saved

    def keep_rows(self, rows: Sequence[int]) -> None:
        """Drops every batch row that is not in ``rows`` (increasing) and moves the kept ones to the front."""
        for to, row in enumerate(rows):
            if to != row:
                self._move_row(row, to)

    def _move_row(self, row: int, to: int) -> None:
        raise NotImplementedError


class SpanKVCache(RowCache):
    """Keys ``[batch, max_seq_len, kv_heads, key_dim]`` and values ``[..., value_dim]`` read as key ranges."""

    def __init__(self, batch_size: int, max_seq_len: int, num_kv_heads: int, key_dim: int, value_dim: int, dtype: torch.dtype) -> None:
        super().__init__(batch_size, max_seq_len)
        self.register_buffer("k", torch.zeros(batch_size, max_seq_len, num_kv_heads, key_dim, dtype=dtype), persistent=False)
        self.register_buffer("v", torch.zeros(batch_size, max_seq_len, num_kv_heads, value_dim, dtype=dtype), persistent=False)

    def _move_row(self, row: int, to: int) -> None:
        for t in (self.k, self.v):
            t[to, : self._size].copy_(t[row, : self._size])


class StateCache(RowCache):
    """The 32-bit state ``[batch, heads, key_dim, value_dim]`` of a recurrent layer.  A cache of size 0 stands for a state of zeros,
    whatever the buffer holds."""

    def __init__(self, batch_size: int, max_seq_len: int, num_heads: int, key_dim: int, value_dim: int) -> None:
        super().__init__(batch_size, max_seq_len)
        self.register_buffer("state", torch.zeros(batch_size, num_heads, key_dim, value_dim, dtype=torch.float32), persistent=False)

    def rewind(self, size: int) -> None:
        if size not in (0, self._size):
            raise ValueError("a recurrent state cannot forget single tokens")
        self._size = size

    def snapshot(self) -> Any:
        return self._size, self.state.clone()

    def restore(self, saved: Any) -> None:
        self._size = saved[0]
        self.state.copy_(saved[1])

    def _move_row(self, row: int, to: int) -> None:
        self.state[to].copy_(self.state[row])


class PassCaches(nn.Module):
    """One cache for each time a layer runs in a forward pass (a looped layer has several); they all hold the same tokens."""

    def __init__(self, caches: Sequence[RowCache]) -> None:
        super().__init__()
        self.passes = nn.ModuleList(caches)

    def __getitem__(self, index: int) -> RowCache:
        return self.passes[index]

    def __iter__(self) -> Iterator[RowCache]:
        return iter(self.passes)

    @property
    def size(self) -> int:
        return self.passes[0].size

    @property
    def slot(self) -> Optional[torch.Tensor]:
        return self.passes[0].slot

    @slot.setter
    def slot(self, value: Optional[torch.Tensor]) -> None:
        for c in self.passes:
            c.slot = value

    def reset(self) -> None:
        for c in self.passes:
            c.reset()

    def reserve(self, batch: int, count: int) -> int:
        return self.passes[0].reserve(batch, count)

    def advance(self, count: int) -> None:
        for c in self.passes:
            c.advance(count)

    def rewind(self, size: int) -> None:
        for c in self.passes:
            c.rewind(size)

    def snapshot(self) -> List[Any]:
        return [c.snapshot() for c in self.passes]

    def restore(self, saved: List[Any]) -> None:
        for c, s in zip(self.passes, saved):
            c.restore(s)

    def keep_rows(self, rows: Sequence[int]) -> None:
        for c in self.passes:
            c.keep_rows(rows)
