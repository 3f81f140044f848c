"""Dense MLPs on the fused up-projection and down-projection kernels: SwiGLU with the reference's
parameters (complexity_deep/core/mlp.py:19-40), and for designs that keep the residual stream in fp32
the clamped gated unit and the squared relu."""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from ._cache import DerivedCache
from .padding import ROW_ALIGN, pad_rows, round_up


class SwiGLU(nn.Module):
    """out = down_proj(silu(gate_proj(x)) * up_proj(x)); three bias-free nn.Linear."""

    def __init__(self, hidden_size: int, intermediate_size: int):
        super().__init__()
        self.gate_proj = nn.Linear(hidden_size, intermediate_size, bias=False)
        self.up_proj = nn.Linear(hidden_size, intermediate_size, bias=False)
        self.down_proj = nn.Linear(intermediate_size, hidden_size, bias=False)
        self._derived = DerivedCache()

    def _packed(self):
        g, u = self.gate_proj.weight, self.up_proj.weight
        bn = ops.choose_block_n(g.shape[0])
        packed = self._derived.get(
            "gate_up", (g, u),
            lambda: ops.pack_gate_up(g.detach()[None].contiguous(), u.detach()[None].contiguous(), bn))
        return packed, bn

    def _run(self, x2: torch.Tensor, residual=None, residual_lo=None, want_lo: bool = False):
        packed, bn = self._packed()
        width = self.gate_proj.weight.shape[0]
        h = ops.moe_up(x2, None, 1, packed, width, bn)
        wd = self.down_proj.weight.detach()[None]  # [1, H, I]
        return ops.moe_down(h, wd, None, None, None, 1, None, residual, residual_lo, want_lo)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ops.forward_only(x, "SwiGLU")
        shape = x.shape
        return self._run(x.reshape(-1, shape[-1]).contiguous()).view(shape)


class ClampedGLU(nn.Module):
    """down_proj(g * sigmoid(alpha g) * (u + offset)) with g = min(gate_proj(x), limit) and
    u = clamp(up_proj(x), -limit, limit); three bias-free nn.Linear."""

    def __init__(self, hidden_size: int, intermediate_size: int, limit: float, alpha: float = 1.702,
                 offset: float = 1.0):
        super().__init__()
        self.limit, self.alpha, self.offset = limit, alpha, offset
        self.gate_proj = nn.Linear(hidden_size, intermediate_size, bias=False)
        self.up_proj = nn.Linear(hidden_size, intermediate_size, bias=False)
        self.down_proj = nn.Linear(intermediate_size, hidden_size, bias=False)
        self._derived = DerivedCache()

    def _padded(self, width: int):
        g, u = self.gate_proj.weight.detach(), self.up_proj.weight.detach()
        rows = -(-g.shape[0] // 8) * 8
        return pad_rows(g, rows, width), pad_rows(u, rows, width)

    def _up(self, x: torch.Tensor) -> torch.Tensor:
        src = (self.gate_proj.weight, self.up_proj.weight)
        if x.dtype == torch.float32:
            w = self._derived.get("gate_up_f32", src, lambda: torch.cat(self._padded(x.shape[1]), 0).contiguous())
            return ops.glu_f32(ops.project(x, w, tag="glu_up"), self.alpha, self.limit, self.offset)
        rows = -(-self.gate_proj.weight.shape[0] // 8) * 8
        bn = ops.choose_block_n(rows, x.shape[0])

        def make():
            g, u = self._padded(x.shape[1])
            return ops.pack_gate_up(g[None].contiguous(), u[None].contiguous(), bn)

        return ops.glu_up(x, self._derived.get(f"gate_up_{bn}", src, make), rows, bn, self.alpha,
                          self.limit, self.offset)

    def run(self, x: torch.Tensor, stream: torch.Tensor, layer_scale=None, scale: float = 1.0) -> torch.Tensor:
        """stream += scale * layer_scale * mlp(x), in place; x [T, width padded], stream fp32."""
        h = self._up(x)
        w = self._derived.get("down", (self.down_proj.weight,), lambda: pad_rows(
            self.down_proj.weight.detach(), stream.shape[1], h.shape[1]).contiguous())
        return ops.linear_to_f32(h, w, residual=stream, col_scale=layer_scale, inplace=True,
                                 tag="glu_down", scale=scale)


class SquaredReLU(nn.Module):
    """down_proj(relu(up_proj(x))^2); two bias-free nn.Linear."""

    def __init__(self, hidden_size: int, intermediate_size: int):
        super().__init__()
        self.up_proj = nn.Linear(hidden_size, intermediate_size, bias=False)
        self.down_proj = nn.Linear(intermediate_size, hidden_size, bias=False)
        self._derived = DerivedCache()

    def run(self, x: torch.Tensor, stream: torch.Tensor, layer_scale=None, scale: float = 1.0) -> torch.Tensor:
        """stream += scale * layer_scale * mlp(x), in place; x [T, width padded], stream fp32."""
        rows = round_up(self.up_proj.weight.shape[0], ROW_ALIGN)
        up = self._derived.get("up", (self.up_proj.weight,), lambda: pad_rows(
            self.up_proj.weight.detach(), rows, x.shape[1]).contiguous())
        down = self._derived.get("down", (self.down_proj.weight,), lambda: pad_rows(
            self.down_proj.weight.detach(), stream.shape[1], rows).contiguous())
        h = ops.project(x, up, tag="relu2_up", act="relu2")
        return ops.linear_to_f32(h, down, residual=stream, col_scale=layer_scale, inplace=True,
                                 tag="relu2_down", scale=scale)
