"""RMS normalisation (parity: torchtune/modules/rms_norm.py:11-60)."""
from __future__ import annotations

from typing import Optional, Tuple

import torch
from torch import nn

from .. import ops


class RMSNorm(nn.Module):
    """``x * rsqrt(mean(x^2) + eps) * scale`` with fp32 statistics; the learnable
    parameter is called ``scale``."""

    def __init__(self, dim: int, eps: float = 1e-6) -> None:
        super().__init__()
        self.normalized_shape = (dim,)
        self.eps = eps
        self.scale = nn.Parameter(torch.ones(dim))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.rms_norm(x, self.scale, self.eps)

    def extra_repr(self) -> str:
        return f"dim={self.normalized_shape[0]}, eps={self.eps}"


class StreamRMSNorm(nn.Module):
    """RMS norm between a 32-bit residual stream and a sublayer: fp32 in, the gain's dtype out, one rounding.  With ``zero_centered`` the
    gain is ``1 + scale`` and ``scale`` starts at zero.

    :meth:`chain` is the fused step from one sublayer to the next."""

    def __init__(self, dim: int, eps: float = 1e-6, zero_centered: bool = False) -> None:
        super().__init__()
        self.normalized_shape = (dim,)
        self.eps = eps
        self.offset = 1.0 if zero_centered else 0.0
        self.scale = nn.Parameter(torch.zeros(dim) if zero_centered else torch.ones(dim))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.residual_norm(x.float(), None, None, self.scale, eps=self.eps, offset=self.offset)[1]

    @staticmethod
    def chain(x: torch.Tensor, y: torch.Tensor, post: "StreamRMSNorm", mult: float, following: Optional["StreamRMSNorm"]) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """``(x + mult · post(y), following(that))``; ``following=None`` leaves the second out."""
        if following is not None and (following.eps != post.eps or following.offset != post.offset):
            x, _ = ops.residual_norm(x, y, post.scale, None, eps=post.eps, mult=mult, offset=post.offset)
            return x, following(x)
        return ops.residual_norm(x, y, post.scale, None if following is None else following.scale, eps=post.eps, mult=mult, offset=post.offset)

    def extra_repr(self) -> str:
        return f"dim={self.normalized_shape[0]}, eps={self.eps}, offset={self.offset}"


class StreamLayerNorm(nn.Module):
    """Layer norm with a gain and no bias between a 32-bit residual stream and a sublayer: fp32 in, the gain's dtype out, one rounding."""

    def __init__(self, dim: int, eps: float = 1e-5) -> None:
        super().__init__()
        self.normalized_shape = (dim,)
        self.eps = eps
        self.scale = nn.Parameter(torch.ones(dim))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.stream_step(x.float().unsqueeze(-2), None, None, None, None, None, self.scale, eps=self.eps, centered=True)[1]

    def extra_repr(self) -> str:
        return f"dim={self.normalized_shape[0]}, eps={self.eps}"


def rms_norm(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    """Weight-less RMS norm over the last dimension (Llama-4 q/k normalisation)."""
    return ops.rms_norm(x, None, eps)
