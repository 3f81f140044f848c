"""RMSNorm with the reference's constructor, parameters and forward signature
(complexity_deep/core/normalization.py:17-35), computed by the N1 CUDA kernel."""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from ._cache import DerivedCache
from .padding import pad_vector


class RMSNorm(nn.Module):
    """y = weight * x * rsqrt(mean(x^2, -1) + eps); state_dict key: ``weight`` [hidden_size]."""

    def __init__(self, hidden_size: int, eps: float = 1e-6):
        super().__init__()
        self.eps = eps
        self.weight = nn.Parameter(torch.ones(hidden_size))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ops.forward_only(x, "RMSNorm")
        return ops.rmsnorm(x.contiguous(), self.weight, self.eps)

    def extra_repr(self) -> str:
        return f"{self.weight.numel()}, eps={self.eps}"


class StreamNorm(nn.Module):
    """RMSNorm of the fp32 residual stream into the weights' dtype:
    y = x / sqrt(mean(x^2) + eps) * (offset + weight); offset 1 for a weight stored around zero.
    centred: layer norm without a bias, the same of x - mean(x)."""

    def __init__(self, hidden_size: int, eps: float, offset: float = 0.0, centred: bool = False):
        super().__init__()
        if centred and offset:
            raise ValueError("a centred norm has a plain weight")
        self.eps, self.offset, self.centred = eps, offset, centred
        self.weight = nn.Parameter(torch.full((hidden_size,), 1.0 - offset))
        self._derived = DerivedCache()

    def forward(self, stream: torch.Tensor) -> torch.Tensor:
        """stream [T, width padded] fp32 -> [T, width padded]; the padding stays zero."""
        w = self._derived.get("weight", (self.weight,),
                              lambda: pad_vector(self.weight.detach(), stream.shape[1]))
        if self.centred:
            return ops.layernorm_f32(stream, w, self.eps, width=self.weight.numel())
        return ops.rmsnorm_f32(stream, w, self.eps, self.offset, width=self.weight.numel())

    def extra_repr(self) -> str:
        return f"{self.weight.numel()}, eps={self.eps}, offset={self.offset}, centred={self.centred}"
