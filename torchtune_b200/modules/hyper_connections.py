"""Hyper-connections: several residual streams instead of one, read, mixed and written by learned weights around every sublayer."""
from __future__ import annotations

from typing import NamedTuple, Optional, Tuple

import torch
from torch import nn

from .. import ops
from .rms_norm import StreamLayerNorm


class LayerScale(nn.Module):
    """Element-wise gain of a sublayer's output."""

    def __init__(self, dim: int, init: float = 1.0) -> None:
        super().__init__()
        self.scale = nn.Parameter(torch.full((dim,), float(init)))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return x * self.scale


class StreamEntry(NamedTuple):
    """How the next reader takes its input from the streams: read weights (``None``: their sum), its norm, and whether the streams are
    needed afterwards."""

    read: Optional[torch.Tensor]
    norm: StreamLayerNorm
    keep: bool = True


class HyperConnection(nn.Module):
    """Weights of one sublayer: its input is ``Σ_s read[s] x_s``; its output ``y`` turns the streams into
    ``x_t = Σ_s mix[s, t] x_s + write[t] y``.  Streams are ``[b, s, streams, dim]`` fp32; one stream stands for that many equal ones."""

    def __init__(self, streams: int) -> None:
        super().__init__()
        self.streams = streams
        self.read = nn.Parameter(torch.full((streams,), 1.0 / streams))
        self.write = nn.Parameter(torch.ones(streams))
        self.mix = nn.Parameter(torch.eye(streams))

    @staticmethod
    def enter(x: torch.Tensor, entry: StreamEntry) -> torch.Tensor:
        return ops.stream_step(x, None, None, None, None, entry.read, entry.norm.scale, eps=entry.norm.eps, centered=True)[1]

    def step(self, x: torch.Tensor, y: torch.Tensor, gain: LayerScale, following: Optional[StreamEntry]) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
        """The streams after the sublayer and the next reader's normed input, in one pass."""
        if following is None:
            return ops.stream_step(x, y, gain.scale, self.mix, self.write, None, None, eps=0.0, centered=True)
        return ops.stream_step(x, y, gain.scale, self.mix, self.write, following.read, following.norm.scale, eps=following.norm.eps, centered=True, keep=following.keep)
