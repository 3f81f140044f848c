"""Token mixers that share one input projection and one output projection.

A mixer declares the rows it needs in the layer's input projection (``projections``), the columns
it contributes to the output projection (``output_weight``) and what it carries from call to call
(``new_state``), and writes its result into its columns of a common buffer (``mix``).
``ParallelMixers`` runs any number of mixers side by side on the same input: one product for all
their projections, the mixers themselves, one product for all their outputs with the residual sum
in its epilogue.  A layer with a single mixer is the case of one branch.

Heads are padded to multiples of 16 and every segment of the projection buffer starts at a multiple
of 16 elements: the zero rows that the padding adds to the weights make the padded positions zero
wherever they are used.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from .. import ops
from ._cache import DerivedCache
from .padding import HEAD_ALIGN, pad_heads, pad_rows, pad_vector, round_up
from .rotary import interleaved_tables
from .state import DecoderState, DeltaState, LatentState, RecurrentState, WindowState


class Mixer(nn.Module):
    """One branch of ``ParallelMixers``."""
    out_width: int                      # columns of the mixers' output buffer (padded)

    def projections(self) -> List[Tuple[str, torch.Tensor]]:
        """(name, padded weight [rows, width]) of every projection of the layer input."""
        raise NotImplementedError

    def sources(self) -> Sequence[torch.Tensor]:
        """Parameters behind ``projections`` and ``output_weight``."""
        raise NotImplementedError

    def output_weight(self) -> torch.Tensor:
        """[width, out_width]"""
        raise NotImplementedError

    def new_state(self, batch: int, device, dtype, capacity: Optional[int] = None):
        """What the mixer carries from call to call; `capacity`: most tokens per sequence, for states
        that grow and must keep their address."""
        raise NotImplementedError

    def mix(self, proj: Dict[str, torch.Tensor], out: torch.Tensor, part, state: DecoderState,
            batch: int, seq_len: int, out_scale: float) -> None:
        """Writes ``out_scale *`` the mixer's result (before its output projection) into `out`;
        `part` is this mixer's share of `state`."""
        raise NotImplementedError


class WindowAttention(Mixer):
    """Softmax attention over a sliding window with kept first tokens, grouped key heads, per-head
    norm of queries and keys, a logarithmic distance bias per head and mixing of the heads' weights
    after the softmax (see cd_window_attn in include/cdeep.h).  Positions enter through the bias
    only."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, window: int,
                 keep_first: int, scale: float, eps: float) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError("query heads must be a multiple of the key/value heads")
        if window < 1 or keep_first < 0:
            raise ValueError("window must be positive and keep_first not negative")
        self.width, self.heads, self.kv_heads = width, heads, kv_heads
        self.dim, self.vdim = dim, vdim
        self.window, self.keep_first, self.scale, self.eps = window, keep_first, scale, eps
        self.key_width, self.value_width = round_up(dim, HEAD_ALIGN), round_up(vdim, HEAD_ALIGN)
        self.out_width = heads * self.value_width
        self.q_proj = nn.Linear(width, heads * dim, bias=False)
        self.k_proj = nn.Linear(width, kv_heads * dim, bias=False)
        self.v_proj = nn.Linear(width, kv_heads * vdim, bias=False)
        self.o_proj = nn.Linear(heads * vdim, width, bias=False)
        self.q_norm = nn.Parameter(torch.ones(dim))
        self.k_norm = nn.Parameter(torch.ones(dim))
        self.r1 = nn.Parameter(torch.zeros(heads))
        self.r2 = nn.Parameter(torch.zeros(heads))
        self.talk = nn.Parameter(torch.eye(heads))
        self._derived = DerivedCache()

    def projections(self):
        return [("q", pad_heads(self.q_proj.weight.detach(), self.heads, self.key_width)),
                ("k", pad_heads(self.k_proj.weight.detach(), self.kv_heads, self.key_width)),
                ("v", pad_heads(self.v_proj.weight.detach(), self.kv_heads, self.value_width))]

    def sources(self):
        return (self.q_proj.weight, self.k_proj.weight, self.v_proj.weight, self.o_proj.weight)

    def output_weight(self):
        return pad_heads(self.o_proj.weight.detach().t().contiguous(), self.heads, self.value_width).t()

    def _weights(self):
        src = (self.q_norm, self.k_norm, self.r1, self.r2, self.talk)
        return self._derived.get("small", src, lambda: {
            "q_norm": pad_vector(self.q_norm.detach(), self.key_width),
            "k_norm": pad_vector(self.k_norm.detach(), self.key_width),
            "r1": self.r1.detach(), "r2": self.r2.detach(), "talk": self.talk.detach().contiguous()})

    def new_state(self, batch, device, dtype, capacity=None):
        return WindowState(batch, self.window, self.keep_first, self.kv_heads, self.key_width,
                           self.value_width, device, dtype)

    def mix(self, proj, out, part, state, batch, seq_len, out_scale):
        ops.window_attention_(
            proj, out, self._weights(), part.k, part.v, batch=batch, seq_len=seq_len, heads=self.heads,
            kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, window=self.window,
            keep=self.keep_first, scale=self.scale, eps=self.eps, out_scale=out_scale,
            pos0=state.length, pos_dev=state.position if state.device_position else None)


class GatedLinearAttention(Mixer):
    """Linear attention with one decay per key channel, a head norm and a silu gate on its output
    (see cd_linear_attn in include/cdeep.h).  The decay comes from a two-step projection whose
    first step is part of the common input projection."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, rank: int, tau: float,
                 eps: float) -> None:
        super().__init__()
        self.width, self.heads, self.dim, self.vdim, self.rank = width, heads, dim, vdim, rank
        self.tau, self.eps = tau, eps
        self.key_width, self.value_width = round_up(dim, HEAD_ALIGN), round_up(vdim, HEAD_ALIGN)
        self.rank_width = round_up(rank, HEAD_ALIGN)
        self.out_width = heads * self.value_width
        self.q_proj = nn.Linear(width, heads * dim, bias=False)
        self.k_proj = nn.Linear(width, heads * dim, bias=False)
        self.v_proj = nn.Linear(width, heads * vdim, bias=False)
        self.g_proj = nn.Linear(width, heads * vdim, bias=False)
        self.o_proj = nn.Linear(heads * vdim, width, bias=False)
        self.a1_proj = nn.Linear(width, rank, bias=False)
        self.a2_proj = nn.Linear(rank, heads * dim, bias=True)
        self.norm = nn.Parameter(torch.ones(vdim))
        self._derived = DerivedCache()

    def projections(self):
        return [("q", pad_heads(self.q_proj.weight.detach(), self.heads, self.key_width)),
                ("k", pad_heads(self.k_proj.weight.detach(), self.heads, self.key_width)),
                ("v", pad_heads(self.v_proj.weight.detach(), self.heads, self.value_width)),
                ("gate", pad_heads(self.g_proj.weight.detach(), self.heads, self.value_width)),
                ("inner", pad_rows(self.a1_proj.weight.detach(), self.rank_width))]

    def sources(self):
        return (self.q_proj.weight, self.k_proj.weight, self.v_proj.weight, self.g_proj.weight,
                self.a1_proj.weight, self.o_proj.weight)

    def output_weight(self):
        return pad_heads(self.o_proj.weight.detach().t().contiguous(), self.heads, self.value_width).t()

    def _weights(self):
        src = (self.a2_proj.weight, self.a2_proj.bias, self.norm)
        return self._derived.get("small", src, lambda: {
            "a2": pad_rows(pad_heads(self.a2_proj.weight.detach(), self.heads, self.key_width),
                           self.heads * self.key_width, self.rank_width).contiguous(),
            "a2_b": pad_heads(self.a2_proj.bias.detach().view(-1, 1), self.heads, self.key_width).reshape(-1),
            "norm": pad_vector(self.norm.detach(), self.value_width)})

    def new_state(self, batch, device, dtype, capacity=None):
        return RecurrentState(batch, self.heads, self.key_width, self.value_width, device)

    def mix(self, proj, out, part, state, batch, seq_len, out_scale):
        ops.linear_attention_(proj, out, self._weights(), part.s, batch=batch, seq_len=seq_len,
                              heads=self.heads, dim=self.dim, vdim=self.vdim, tau=self.tau,
                              eps=self.eps, out_scale=out_scale)


class LatentAttention(Mixer):
    """Softmax attention over a cached low-rank latent beside a rotated key that the heads have in common,
    with a sigmoid gate per head (see cd_latent_attn in include/cdeep.h).  `positions`: most tokens of a
    sequence; `rot_dims` of the `rot` rotated elements turn, with the given base."""

    def __init__(self, width: int, heads: int, dim: int, rot: int, vdim: int, rank: int, scale: float,
                 rot_dims: int, rot_base: float, positions: int, eps: float) -> None:
        super().__init__()
        if rot_dims % 2 or not 0 < rot_dims <= rot:
            raise ValueError("rotated dimensions come in pairs and must lie within the rotated part")
        self.width, self.heads, self.dim, self.rot, self.vdim, self.rank = width, heads, dim, rot, vdim, rank
        self.scale, self.rot_dims, self.rot_base, self.positions, self.eps = scale, rot_dims, rot_base, positions, eps
        self.dim_width, self.rot_width = round_up(dim, HEAD_ALIGN), round_up(rot, HEAD_ALIGN)
        self.rank_width, self.value_width = round_up(rank, HEAD_ALIGN), round_up(vdim, HEAD_ALIGN)
        self.out_width = heads * self.value_width
        self.q_proj = nn.Linear(width, heads * (dim + rot), bias=False)
        self.kv_proj = nn.Linear(width, rank + rot, bias=False)
        self.kv_norm = nn.Parameter(torch.ones(rank))
        self.uk_proj = nn.Linear(rank, heads * dim, bias=False)
        self.uv_proj = nn.Linear(rank, heads * vdim, bias=False)
        self.g_proj = nn.Linear(width, heads, bias=False)
        self.o_proj = nn.Linear(heads * vdim, width, bias=False)
        self._derived = DerivedCache()

    def projections(self):
        q = self.q_proj.weight.detach().view(self.heads, self.dim + self.rot, self.width)
        q = torch.cat([pad_heads(q[:, :self.dim].reshape(-1, self.width), self.heads, self.dim_width).view(
            self.heads, self.dim_width, self.width), pad_heads(q[:, self.dim:].reshape(-1, self.width), self.heads,
                                                               self.rot_width).view(
            self.heads, self.rot_width, self.width)], 1).reshape(-1, self.width)
        kv = self.kv_proj.weight.detach()
        kv = torch.cat([pad_rows(kv[:self.rank], self.rank_width), pad_rows(kv[self.rank:], self.rot_width)], 0)
        return [("q", q), ("kv", kv),
                ("gate", pad_rows(self.g_proj.weight.detach(), round_up(self.heads, HEAD_ALIGN)))]

    def sources(self):
        return (self.q_proj.weight, self.kv_proj.weight, self.g_proj.weight, self.o_proj.weight)

    def output_weight(self):
        return pad_heads(self.o_proj.weight.detach().t().contiguous(), self.heads, self.value_width).t()

    def _weights(self):
        src = (self.kv_norm, self.uk_proj.weight, self.uv_proj.weight)

        def make():
            H = self.heads
            uk, uv = (pad_rows(w.detach(), w.shape[0], self.rank_width)
                      for w in (self.uk_proj.weight, self.uv_proj.weight))
            uv = pad_heads(uv, H, self.value_width).contiguous()
            expand = torch.cat([pad_heads(uk, H, round_up(self.dim, 64)), uv], 0)
            uk = pad_heads(uk, H, self.dim_width).reshape(H, self.dim_width, self.rank_width).contiguous()
            cos, sin = interleaved_tables(self.positions, self.rot_dims, self.rot_width, self.rot_base, uk.device)
            return {"norm": pad_vector(self.kv_norm.detach(), self.rank_width), "uk": uk, "expand": expand,
                    "uk_t": uk.transpose(1, 2).contiguous(), "uv": uv.view(H, self.value_width, self.rank_width),
                    "cos": cos, "sin": sin}

        return self._derived.get("small", src, make)

    def new_state(self, batch, device, dtype, capacity=None):
        return LatentState(batch, self.rank_width + self.rot_width, self.positions, device, dtype, capacity)

    def mix(self, proj, out, part, state, batch, seq_len, out_scale):
        on_device = state.device_position
        cache = part.rows if on_device else part.reserve(state.length + seq_len)
        ops.latent_attention_(
            proj, out, self._weights(), cache, batch=batch, seq_len=seq_len, heads=self.heads, dim=self.dim,
            rot=self.rot, rank=self.rank, vdim=self.vdim, scale=self.scale, eps=self.eps, out_scale=out_scale,
            pos0=0 if on_device else state.length, pos_dev=state.position if on_device else None)


class DeltaRule(Mixer):
    """Gated delta rule whose state decays at a rate per key channel, with short convolutions ahead of q, k and v,
    grouped q / k heads, a head norm and a sigmoid gate on the result (see cd_delta_attn in
    include/cdeep.h).  Decay and gate come from two-step projections of inner width `rank` and
    `gate_rank`, whose first steps are part of the common input projection."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, rank: int,
                 gate_rank: int, eps: float) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of the q / k heads")
        if taps < 1:
            raise ValueError("the convolution needs at least the current token")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.taps, self.rank, self.gate_rank, self.eps = taps, rank, gate_rank, eps
        self.key_width, self.value_width = round_up(dim, HEAD_ALIGN), round_up(vdim, HEAD_ALIGN)
        self.channels = 2 * kv_heads * self.key_width + heads * self.value_width
        self.out_width = heads * self.value_width
        self.q_proj = nn.Linear(width, kv_heads * dim, bias=False)
        self.k_proj = nn.Linear(width, kv_heads * dim, bias=False)
        self.v_proj = nn.Linear(width, heads * vdim, bias=False)
        self.q_conv = nn.Parameter(torch.zeros(kv_heads * dim, taps))
        self.k_conv = nn.Parameter(torch.zeros(kv_heads * dim, taps))
        self.v_conv = nn.Parameter(torch.zeros(heads * vdim, taps))
        self.b_proj = nn.Linear(width, heads, bias=False)
        self.a1_proj = nn.Linear(width, rank, bias=False)
        self.a2_proj = nn.Linear(rank, heads * dim, bias=False)
        self.A_log = nn.Parameter(torch.zeros(heads))
        self.dt_bias = nn.Parameter(torch.zeros(heads * dim))
        self.g1_proj = nn.Linear(width, gate_rank, bias=False)
        self.g2_proj = nn.Linear(gate_rank, heads * vdim, bias=False)
        self.norm = nn.Parameter(torch.ones(vdim))
        self.o_proj = nn.Linear(heads * vdim, width, bias=False)
        self._derived = DerivedCache()

    def projections(self):
        a, g = round_up(self.rank, HEAD_ALIGN), round_up(self.gate_rank, HEAD_ALIGN)
        return [("q", pad_heads(self.q_proj.weight.detach(), self.kv_heads, self.key_width)),
                ("k", pad_heads(self.k_proj.weight.detach(), self.kv_heads, self.key_width)),
                ("v", pad_heads(self.v_proj.weight.detach(), self.heads, self.value_width)),
                ("b", pad_rows(self.b_proj.weight.detach(), round_up(self.heads, HEAD_ALIGN))),
                ("inner", torch.cat([pad_rows(self.a1_proj.weight.detach(), a),
                                     pad_rows(self.g1_proj.weight.detach(), g)], 0))]

    def sources(self):
        return (self.q_proj.weight, self.k_proj.weight, self.v_proj.weight, self.b_proj.weight,
                self.a1_proj.weight, self.g1_proj.weight, self.o_proj.weight)

    def output_weight(self):
        return pad_heads(self.o_proj.weight.detach().t().contiguous(), self.heads, self.value_width).t()

    def _weights(self):
        src = (self.a2_proj.weight, self.g2_proj.weight, self.q_conv, self.k_conv, self.v_conv, self.A_log,
               self.dt_bias, self.norm)

        def make():
            a, g = round_up(self.rank, HEAD_ALIGN), round_up(self.gate_rank, HEAD_ALIGN)
            a2 = pad_heads(self.a2_proj.weight.detach(), self.heads, self.key_width)
            g2 = pad_heads(self.g2_proj.weight.detach(), self.heads, self.value_width)
            inner = a2.new_zeros(a2.shape[0] + g2.shape[0], a + g)      # one product for both second steps
            inner[: a2.shape[0], : self.rank] = a2
            inner[a2.shape[0]:, a: a + self.gate_rank] = g2
            taps = torch.cat([pad_heads(self.q_conv.detach(), self.kv_heads, self.key_width),
                              pad_heads(self.k_conv.detach(), self.kv_heads, self.key_width),
                              pad_heads(self.v_conv.detach(), self.heads, self.value_width)], 0)
            return {"inner": inner, "taps": taps.t().contiguous(), "rate": self.A_log.detach().float().exp(),
                    "dt_bias": pad_heads(self.dt_bias.detach().float().view(-1, 1), self.heads,
                                         self.key_width).reshape(-1).contiguous(),
                    "norm": pad_vector(self.norm.detach(), self.value_width)}

        return self._derived.get("small", src, make)

    def new_state(self, batch, device, dtype, capacity=None):
        return DeltaState(batch, self.heads, self.key_width, self.value_width, self.taps, self.channels, device, dtype)

    def mix(self, proj, out, part, state, batch, seq_len, out_scale):
        on_device = state.device_position
        ops.delta_attention_(
            proj, out, self._weights(), part.ring, part.s, batch=batch, seq_len=seq_len, heads=self.heads,
            kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, eps=self.eps, out_scale=out_scale,
            pos0=0 if on_device else state.length, pos_dev=state.position if on_device else None)


class ParallelMixers(nn.Module):
    """``sum_m scale_m * mixer_m(h)`` over named branches that read the same h."""

    def __init__(self, branches: Dict[str, Mixer], scales: Dict[str, float]) -> None:
        super().__init__()
        self.branches = nn.ModuleDict(branches)
        self.scales = dict(scales)
        self._derived = DerivedCache()

    def _packed(self, width: int):
        """(stacked input projection, {branch: {name: columns}}, stacked output projection)"""
        src = [t for m in self.branches.values() for t in m.sources()]

        def make():
            rows, spans, at = [], {}, 0
            for name, m in self.branches.items():
                spans[name] = {}
                for part, w in m.projections():
                    rows.append(pad_rows(w, w.shape[0], width))
                    spans[name][part] = (at, at + w.shape[0])
                    at += w.shape[0]
            outs = [pad_rows(m.output_weight(), width) for m in self.branches.values()]
            return torch.cat(rows, 0).contiguous(), spans, torch.cat(outs, 1).contiguous()

        return self._derived.get("packed", src, make)

    def new_state(self, batch: int, device, dtype, capacity: Optional[int] = None) -> Dict[str, object]:
        return {name: m.new_state(batch, device, dtype, capacity) for name, m in self.branches.items()}

    def run(self, h: torch.Tensor, x: torch.Tensor, layer_scale: Optional[torch.Tensor],
            parts: Dict[str, object], state: DecoderState, batch: int, seq_len: int,
            scale: float = 1.0) -> torch.Tensor:
        """x += scale * layer_scale * mixers(h), in place; h [T, width padded], x the fp32 stream."""
        w_in, spans, w_out = self._packed(h.shape[1])
        proj = ops.project(h, w_in, tag="mixer_in")
        out = torch.empty(h.shape[0], w_out.shape[1], dtype=h.dtype, device=h.device)
        at = 0
        for name, m in self.branches.items():
            cols = {part: proj[:, a:b] for part, (a, b) in spans[name].items()}
            m.mix(cols, out[:, at:at + m.out_width], parts[name], state, batch, seq_len,
                  self.scales[name])
            at += m.out_width
        return ops.linear_to_f32(out, w_out, residual=x, col_scale=layer_scale, inplace=True,
                                 tag="mixer_out", scale=scale)
