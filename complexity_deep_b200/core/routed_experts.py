"""Mixture of experts with a learned router: softmax scores, the best groups of neighbouring experts,
the best experts within them, clamped gated units as experts.  ``TokenRoutedMLP`` is the counterpart
whose routing is a table over token ids."""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from ._cache import DerivedCache
from .padding import ROW_ALIGN, pad_rows, round_up


class RoutedExperts(nn.Module):
    """sum over the chosen experts of weight * expert(x); expert(x) = down(g sigmoid(alpha g) (u + offset))
    with g = min(gate(x), limit), u = clamp(up(x), -limit, limit).  Of `groups` equal groups of experts
    only the `keep` with the largest score can be chosen from; what is chosen is weighted in proportion to
    its softmax score, weights adding up to one."""

    def __init__(self, hidden_size: int, intermediate_size: int, experts: int, top: int, limit: float,
                 groups: int = 1, keep: int = 1, alpha: float = 1.702, offset: float = 1.0):
        super().__init__()
        if experts % groups or not 1 <= keep <= groups:
            raise ValueError("experts must form equal groups of which at least one is kept")
        if not 1 <= top <= keep * (experts // groups):
            raise ValueError("more experts per token than the kept groups hold")
        self.experts, self.top, self.groups, self.keep = experts, top, groups, keep
        self.limit, self.alpha, self.offset = limit, alpha, offset
        self.router = nn.Linear(hidden_size, experts, bias=False)
        self.gate_proj = nn.Parameter(torch.empty(experts, intermediate_size, hidden_size).normal_(std=0.02))
        self.up_proj = nn.Parameter(torch.empty(experts, intermediate_size, hidden_size).normal_(std=0.02))
        self.down_proj = nn.Parameter(torch.empty(experts, hidden_size, intermediate_size).normal_(std=0.02))
        self._derived = DerivedCache()

    @staticmethod
    def _pad(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
        return torch.stack([pad_rows(x, rows, cols) for x in w.detach()]).contiguous()

    def choose(self, x: torch.Tensor):
        """(experts, weights), both [T, top]"""
        w = self._derived.get("router", (self.router.weight,), lambda: pad_rows(
            self.router.weight.detach(), round_up(self.experts, ROW_ALIGN), x.shape[1]).contiguous())
        return ops.route_top(ops.linear_to_f32(x, w, tag="router"), self.experts, self.top, self.groups, self.keep)

    def _up(self, x: torch.Tensor, seg: torch.Tensor) -> torch.Tensor:
        src = (self.gate_proj, self.up_proj)
        rows = round_up(self.gate_proj.shape[1], ROW_ALIGN)
        width = x.shape[1]
        if x.dtype == torch.float32:
            w = self._derived.get("gate_up_f32", src, lambda: torch.cat(
                [self._pad(self.gate_proj, rows, width), self._pad(self.up_proj, rows, width)], 1).contiguous())
            return ops.glu_f32(ops.grouped_linear_f32(x, w, seg, "glu_up_routed"), self.alpha, self.limit, self.offset)
        bn = ops.choose_block_n(rows, x.shape[0], self.experts)
        w = self._derived.get(f"gate_up_{bn}", src, lambda: ops.pack_gate_up(
            self._pad(self.gate_proj, rows, width), self._pad(self.up_proj, rows, width), bn))
        return ops.glu_up(x, w, rows, bn, self.alpha, self.limit, self.offset, seg_offsets=seg)

    def run(self, x: torch.Tensor, stream: torch.Tensor, layer_scale=None, scale: float = 1.0) -> torch.Tensor:
        """stream += scale * experts(x), in place; x [T, width padded], stream fp32."""
        if layer_scale is not None:
            raise NotImplementedError("routed experts take a scalar scale only")
        ids, weights = self.choose(x)
        table = self._derived.get("table", (self.router.weight,), lambda: torch.arange(
            self.experts, dtype=torch.int64, device=x.device))
        r = ops.route(ids, table, self.experts)
        h = self._up(ops.gather_div(x, r.perm, self.top), r.offsets)
        down = self._derived.get("down", (self.down_proj,), lambda: self._pad(
            self.down_proj, stream.shape[1], h.shape[1]))
        if x.dtype == torch.float32:
            y = ops.grouped_linear_f32(h, down, r.offsets, "moe_down")
        else:
            y = ops.moe_down(h, down, None, None, r.offsets, self.experts, None, None)
        return ops.combine_top_(stream, y, r.inv_perm, weights, scale)
