"""Tensor-level wrappers over the libcdeep C ABI.

PyTorch is used for device memory and streams only: each function checks its arguments,
allocates outputs with ``torch.empty`` on the caller's device and enqueues the CUDA kernels
on ``torch.cuda.current_stream()``.  Nothing here computes on the CPU and nothing falls
back to PyTorch operators.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib

BF16 = torch.bfloat16


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _need(t: torch.Tensor, name: str, dtype=BF16) -> None:
    if not isinstance(t, torch.Tensor) or not t.is_cuda:
        raise RuntimeError(
            f"{name}: expected a CUDA tensor; the complexity_deep_b200 kernels have no CPU path")
    if t.dtype != dtype:
        raise RuntimeError(f"{name}: expected dtype {dtype}, got {t.dtype}")
    if not t.is_contiguous():
        raise RuntimeError(f"{name}: expected a contiguous tensor")


def forward_only(x: torch.Tensor, what: str) -> None:
    """The kernels are forward-only.  An activation that carries autograd history would lose
    its gradient silently, so that case is refused instead."""
    if torch.is_grad_enabled() and isinstance(x, torch.Tensor) and x.requires_grad:
        raise RuntimeError(
            f"{what}: the complexity_deep_b200 kernels implement the forward pass only; call the "
            "model under torch.no_grad() / torch.inference_mode() (no backward is available)")


class _Profile:
    """Optional CUDA-event timing of the GEMM entry points (used by bench.py).

    Disabled by default: then `span` costs one attribute check.  When enabled, every call of
    an instrumented entry point records an event before and after its launch on the current
    stream; `collect` synchronises and returns per-entry launch counts and device time.
    """

    def __init__(self) -> None:
        self.enabled = False
        self.events = []
        self.kernel_launches = 0

    def reset(self, enabled: bool) -> None:
        self.enabled = enabled
        self.events = []
        self.kernel_launches = 0

    def collect(self):
        """name -> (calls, total_ms, kernels launched)."""
        torch.cuda.synchronize()
        out = {}
        for name, a, b, n in self.events:
            c, ms, k = out.get(name, (0, 0.0, 0))
            out[name] = (c + 1, ms + a.elapsed_time(b), k + n)
        return out


PROFILE = _Profile()


class _Span:
    def __init__(self, name: str, kernels: int = 1) -> None:
        self.name, self.kernels = name, kernels

    def __enter__(self):
        if PROFILE.enabled:
            self.start = torch.cuda.Event(enable_timing=True)
            self.start.record()
        return self

    def __exit__(self, *exc):
        if PROFILE.enabled:
            end = torch.cuda.Event(enable_timing=True)
            end.record()
            PROFILE.events.append((self.name, self.start, end, self.kernels))
        return False


def status_fetch() -> int:
    """Synchronises and returns the kernels' status word (0 = ok); raises on a timeout."""
    lib = _lib.load()
    st = ctypes.c_int(0)
    _lib.check(lib.cd_status_fetch(ctypes.byref(st)), "cd_status_fetch")
    if st.value == 4:
        raise _lib.CdeepError("checking build: a libcdeep kernel met an index, address or segment "
                              "table out of range and skipped the access")
    if st.value != 0:
        raise _lib.CdeepError("a libcdeep kernel gave up on a bounded wait (pipeline error)")
    return st.value


# --------------------------------------------------------------------------- dispatch
@dataclass
class Routing:
    """Routing artefacts of one batch of token ids (all int32, on the device)."""
    expert_ids: torch.Tensor   # [T]
    counts: torch.Tensor       # [E]
    offsets: torch.Tensor      # [E + 1]
    perm: torch.Tensor         # [T] sorted position -> source row
    inv_perm: torch.Tensor     # [T] source row -> sorted position
    num_experts: int


def route(token_ids: torch.Tensor, table: torch.Tensor, num_experts: int) -> Routing:
    lib = _lib.load()
    ids = token_ids.reshape(-1)
    _need(ids, "token_ids", torch.int64)
    _need(table, "token_to_expert", torch.int64)
    T, V, E = ids.numel(), table.numel(), int(num_experts)
    dev = ids.device
    i32 = dict(dtype=torch.int32, device=dev)
    expert_ids = torch.empty(T, **i32)
    perm = torch.empty(T, **i32)
    inv_perm = torch.empty(T, **i32)
    counts = torch.empty(E, **i32)
    offsets = torch.empty(E + 1, **i32)
    ws_bytes = lib.cd_route_workspace_bytes(T, E)
    ws = torch.empty(max(ws_bytes, 4), dtype=torch.uint8, device=dev)
    with _Span("route", 2):
        _lib.check(lib.cd_route(ids.data_ptr(), table.data_ptr(), V, E, T, expert_ids.data_ptr(),
                                counts.data_ptr(), offsets.data_ptr(), perm.data_ptr(),
                                inv_perm.data_ptr(), ws.data_ptr(), ws.numel(), _stream()),
                   "cd_route")
    return Routing(expert_ids, counts, offsets, perm, inv_perm, E)


# --------------------------------------------------------------------------- row-wise
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float,
            residual: Optional[torch.Tensor] = None, dst_rows: Optional[torch.Tensor] = None,
            want_sum: bool = False, x_lo: Optional[torch.Tensor] = None):
    """``norm(x (+ residual)) * weight``; returns ``out`` or ``(sum, out)`` when want_sum.

    With ``dst_rows`` row i of the result is written to row ``dst_rows[i]``.  With ``x_lo``
    (the low part of a split-bf16 value, see ``SplitStream``) the input is ``x + x_lo`` in fp32.
    """
    lib = _lib.load()
    H = x.shape[-1]
    x2 = x.reshape(-1, H)
    _need(x2, "x")
    _need(weight, "weight")
    T = x2.shape[0]
    if x_lo is not None:
        if residual is not None or want_sum:
            raise RuntimeError("x_lo cannot be combined with residual / want_sum")
        lo2 = x_lo.reshape(-1, H)
        _need(lo2, "x_lo")
        if lo2.shape[0] != T:
            raise RuntimeError("x_lo does not match x")
        if dst_rows is not None:
            _need(dst_rows, "dst_rows", torch.int32)
            if dst_rows.numel() != T:
                raise RuntimeError("dst_rows must have one entry per row")
        out = torch.empty_like(x2)
        with _Span("rmsnorm"):
            _lib.check(lib.cd_rmsnorm_split(x2.data_ptr(), lo2.data_ptr(), weight.data_ptr(),
                                            float(eps), out.data_ptr(), _ptr(dst_rows), T, H,
                                            _stream()), "cd_rmsnorm_split")
        return out.view(x.shape)
    res2 = None
    if residual is not None:
        res2 = residual.reshape(-1, H)
        _need(res2, "residual")
    if dst_rows is not None:
        _need(dst_rows, "dst_rows", torch.int32)
        if dst_rows.numel() != T:
            raise RuntimeError("dst_rows must have one entry per row")
    out = torch.empty_like(x2)
    s = torch.empty_like(x2) if (want_sum and res2 is not None) else None
    with _Span("rmsnorm"):
        _lib.check(lib.cd_rmsnorm(x2.data_ptr(), _ptr(res2), weight.data_ptr(), float(eps),
                                  _ptr(s), out.data_ptr(), _ptr(dst_rows), T, H, _stream()),
                   "cd_rmsnorm")
    out = out.view(x.shape)
    if want_sum:
        return (s.view(x.shape) if s is not None else x), out
    return out


def gather_rows(x: torch.Tensor, src_rows: torch.Tensor) -> torch.Tensor:
    lib = _lib.load()
    H = x.shape[-1]
    x2 = x.reshape(-1, H)
    _need(x2, "x")
    _need(src_rows, "src_rows", torch.int32)
    out = torch.empty_like(x2)
    with _Span("gather_rows"):
        _lib.check(lib.cd_gather_rows(x2.data_ptr(), src_rows.data_ptr(), out.data_ptr(),
                                      x2.shape[0], H, _stream()), "cd_gather_rows")
    return out


def qk_norm_rope_(qkv: torch.Tensor, q_w: Optional[torch.Tensor], k_w: Optional[torch.Tensor],
                  cos: torch.Tensor, sin: torch.Tensor, eps: float, seq_len: int, pos0: int,
                  hq: int, hkv: int, head_dim: int) -> torch.Tensor:
    """In-place Q/K RMSNorm + RoPE on the fused projection buffer [T, (hq + 2 hkv) * D]."""
    lib = _lib.load()
    _need(qkv, "qkv")
    _need(cos, "cos", torch.float32)
    _need(sin, "sin", torch.float32)
    if q_w is not None:
        _need(q_w, "q_norm.weight")
        _need(k_w, "k_norm.weight")
    T = qkv.shape[0]
    if qkv.shape[1] != (hq + 2 * hkv) * head_dim:
        raise RuntimeError("qkv width does not match the head layout")
    if cos.shape[0] < pos0 + seq_len or cos.shape[1] != head_dim:
        raise RuntimeError("cos/sin tables too short for the requested positions")
    with _Span("qk_norm_rope"):
        _lib.check(lib.cd_qk_norm_rope(qkv.data_ptr(), _ptr(q_w), _ptr(k_w), cos.data_ptr(),
                                       sin.data_ptr(), float(eps), T, seq_len, pos0, hq, hkv,
                                       head_dim, _stream()), "cd_qk_norm_rope")
    return qkv


def decode_rope_append(qkv: torch.Tensor, q_w: Optional[torch.Tensor],
                       k_w: Optional[torch.Tensor], cos: torch.Tensor, sin: torch.Tensor,
                       eps: float, hq: int, hkv: int, head_dim: int, k_cache: torch.Tensor,
                       v_cache: torch.Tensor, pos_dev: torch.Tensor) -> torch.Tensor:
    """Decode step (one row of qkv per sequence): Q/K RMSNorm + RoPE in place at the position
    held by the device scalar `pos_dev` (int32), and the row's rotated k and its v written
    into k_cache / v_cache [B, hkv, capacity, D] at that position."""
    lib = _lib.load()
    _need(qkv, "qkv")
    _need(cos, "cos", torch.float32)
    _need(sin, "sin", torch.float32)
    if q_w is not None:
        _need(q_w, "q_norm.weight")
        _need(k_w, "k_norm.weight")
    B, D = qkv.shape[0], head_dim
    cap = k_cache.shape[2]
    if qkv.shape[1] != (hq + 2 * hkv) * D:
        raise RuntimeError("qkv width does not match the head layout")
    for t, name in ((k_cache, "k cache"), (v_cache, "v cache")):
        if not t.is_cuda or t.dtype != BF16 or t.stride(-1) != 1 or tuple(t.shape) != (B, hkv, cap, D):
            raise RuntimeError(f"{name}: expected a CUDA bf16 tensor [B, kv heads, capacity, D]")
    if k_cache.stride() != v_cache.stride():
        raise RuntimeError("k and v caches must share their strides")
    if cos.shape[0] < cap or cos.shape[1] != D or sin.shape != cos.shape:
        raise RuntimeError("cos/sin tables must cover the cache capacity")
    if pos_dev.dtype != torch.int32 or not pos_dev.is_cuda or pos_dev.numel() != 1:
        raise RuntimeError("pos_dev: expected one int32 on the device")
    with _Span("decode_rope_append"):
        _lib.check(lib.cd_decode_rope_append(
            qkv.data_ptr(), _ptr(q_w), _ptr(k_w), cos.data_ptr(), sin.data_ptr(), float(eps), B,
            hq, hkv, D, k_cache.data_ptr(), v_cache.data_ptr(), k_cache.stride(0),
            k_cache.stride(1), k_cache.stride(2), cap, pos_dev.data_ptr(), _stream()),
            "cd_decode_rope_append")
    return qkv


def decode_attention(qkv: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                     mask: Optional[torch.Tensor], hq: int, hkv: int, head_dim: int,
                     kv_len_dev: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Single-query attention: qkv [B, (hq + 2 hkv) * D] (its q columns are used), k / v
    [B, hkv, L, D] views of the cache (any batch / head / token strides, D contiguous),
    mask None or a bf16 additive mask viewable as [B or 1, L].  `kv_len_dev` (one int32 on the
    device): attend only the first min(L, value) cached tokens.  Returns [B, hq * D]."""
    lib = _lib.load()
    B, D = qkv.shape[0], head_dim
    L = k.shape[2]
    for t, name in ((qkv, "qkv"), (k, "k cache"), (v, "v cache")):
        if not t.is_cuda or t.dtype != BF16 or t.stride(-1) != 1:
            raise RuntimeError(f"{name}: expected a CUDA bf16 tensor with a contiguous last dim")
    if tuple(k.shape) != (B, hkv, L, D) or tuple(v.shape) != (B, hkv, L, D):
        raise RuntimeError("cache shapes do not match")
    if k.stride() != v.stride():
        raise RuntimeError("k and v caches must share their strides")
    mptr, mstride = None, 0
    if mask is not None:
        m2 = mask.reshape(-1, L)
        if m2.dtype != BF16 or not m2.is_cuda or m2.stride(1) != 1 or m2.shape[0] not in (1, B):
            raise RuntimeError("mask: expected a CUDA bf16 additive mask of shape [B or 1, 1, 1, L]")
        mptr, mstride = m2.data_ptr(), (m2.stride(0) if m2.shape[0] == B else 0)
    if kv_len_dev is not None and (kv_len_dev.dtype != torch.int32 or not kv_len_dev.is_cuda
                                   or kv_len_dev.numel() != 1):
        raise RuntimeError("kv_len_dev: expected one int32 on the device")
    ws_bytes = lib.cd_decode_attention_workspace_bytes(B, hq, hkv, L, D)
    ws = torch.empty(ws_bytes, dtype=torch.uint8, device=qkv.device)
    out = torch.empty(B, hq * D, dtype=BF16, device=qkv.device)
    with _Span("decode_attention", 2):
        _lib.check(lib.cd_decode_attention(
            qkv.data_ptr(), qkv.stride(0), k.data_ptr(), v.data_ptr(), k.stride(0), k.stride(1),
            k.stride(2), mptr, mstride, float(head_dim) ** -0.5, B, hq, hkv, L, _ptr(kv_len_dev),
            D, out.data_ptr(), ws.data_ptr(), ws_bytes, _stream()), "cd_decode_attention")
    return out


def attention_prefill_supported(B: int, S: int, hq: int, hkv: int, head_dim: int) -> bool:
    return bool(_lib.load().cd_attention_prefill_supported(B, S, hq, hkv, head_dim))


def attention_prefill(qkv: torch.Tensor, batch: int, seq_len: int, hq: int, hkv: int,
                      head_dim: int) -> torch.Tensor:
    """Causal self-attention of a prompt: qkv [B * S, (hq + 2 hkv) * D] (after Q/K norm + RoPE)
    -> [B * S, hq * D]; softmax scale D ** -0.5 as scaled_dot_product_attention's default."""
    lib = _lib.load()
    _need(qkv, "qkv")
    if tuple(qkv.shape) != (batch * seq_len, (hq + 2 * hkv) * head_dim):
        raise RuntimeError("qkv shape does not match batch / sequence / head layout")
    out = torch.empty(batch * seq_len, hq * head_dim, dtype=BF16, device=qkv.device)
    with _Span("attention_prefill"):
        _lib.check(lib.cd_attention_prefill(qkv.data_ptr(), out.data_ptr(), batch, seq_len, hq, hkv,
                                            head_dim, float(head_dim) ** -0.5, _stream()),
                   "cd_attention_prefill")
    return out


# --------------------------------------------------------------------------- weights
def choose_block_n(width: int, rows: Optional[int] = None, groups: int = 1,
                   sm_count: Optional[int] = None) -> int:
    """Accumulator-tile width for the SwiGLU up-projection of an expert `width` wide.

    Many rows (prefill): 256 (128 gate + 128 up columns per tile) unless padding `width` to a
    multiple of 128 would waste more than a quarter of the tile columns; then 128 (64 + 64).
    Measured on B200 at width 704 (padded to 768, 9 % waste): 1146 TFLOP/s with 256-wide tiles
    against 672 TFLOP/s with 128-wide ones, which are bound by shared-memory bandwidth.
    Few rows (decode, `rows` <= 512): a tile is one chain of K/16 dependent MMA instructions
    whose cost hardly depends on the tile width, so the time is set by how many tiles the
    busiest SM runs back to back: the narrowest tile that leaves at most one tile per SM
    (every one of the `groups` experts has at least one row tile), else the widest.
    """
    if rows is not None and rows <= 512:
        if sm_count is None:
            sm_count = (torch.cuda.get_device_properties(torch.cuda.current_device())
                        .multi_processor_count if torch.cuda.is_available() else 148)
        m_tiles = max(groups, -(-rows // 128))
        for bn in (32, 64, 128, 256):
            if m_tiles * -(-width // (bn // 2)) <= sm_count:
                return bn
        return 256
    padded = -(-width // 128) * 128
    return 256 if (padded - width) / width <= 0.25 else 128


def pack_gate_up(gate: torch.Tensor, up: torch.Tensor, block_n: int,
                 feature_major: bool = True) -> torch.Tensor:
    """Interleaves gate and up rows per accumulator tile (cd_pack_gate_up).

    feature_major: gate, up are [G, I, H] (one output feature per row, nn.Linear layout);
    otherwise [G, H, I] (the reference's routed-expert layout ``x @ W[e]``).  Result
    [G, ceil(I / half) * block_n, H] with, for each tile, `half` gate rows then `half` up rows
    (half = block_n / 2); rows past I are zero.
    """
    lib = _lib.load()
    _need(gate, "gate weights")
    _need(up, "up weights")
    if gate.shape != up.shape or gate.dim() != 3:
        raise RuntimeError("gate and up must be 3-D tensors of the same shape")
    G = gate.shape[0]
    I, H = (gate.shape[1], gate.shape[2]) if feature_major else (gate.shape[2], gate.shape[1])
    rows = lib.cd_gate_up_packed_rows(I, block_n)
    packed = torch.empty(G, rows, H, dtype=BF16, device=gate.device)
    _lib.check(lib.cd_pack_gate_up(gate.data_ptr(), up.data_ptr(), packed.data_ptr(), G, I, H,
                                   block_n, 1 if feature_major else 0, _stream()),
               "cd_pack_gate_up")
    return packed


def pack_down(down: torch.Tensor) -> torch.Tensor:
    """[E, I, H] (``h @ W[e]``) -> [E, H, I] (one output feature per row) (cd_pack_down)."""
    lib = _lib.load()
    _need(down, "down weights")
    E, I, H = down.shape
    out = torch.empty(E, H, I, dtype=BF16, device=down.device)
    _lib.check(lib.cd_pack_down(down.data_ptr(), out.data_ptr(), E, I, H, _stream()),
               "cd_pack_down")
    return out


# --------------------------------------------------------------------------- GEMMs
def moe_up(x_sorted: torch.Tensor, seg_offsets: Optional[torch.Tensor], num_groups: int,
           packed_w: torch.Tensor, width: int, block_n: int) -> torch.Tensor:
    lib = _lib.load()
    _need(x_sorted, "x_sorted")
    _need(packed_w, "packed gate/up weights")
    T, H = x_sorted.shape
    rows = lib.cd_gate_up_packed_rows(width, block_n)
    if tuple(packed_w.shape) != (num_groups, rows, H):
        raise RuntimeError(f"packed weights have shape {tuple(packed_w.shape)}, expected "
                           f"{(num_groups, rows, H)}")
    if seg_offsets is not None:
        _need(seg_offsets, "seg_offsets", torch.int32)
    h = torch.empty(T, width, dtype=BF16, device=x_sorted.device)
    with _Span("moe_up_routed" if seg_offsets is not None else "moe_up_shared"):
        _lib.check(lib.cd_moe_up(x_sorted.data_ptr(), _ptr(seg_offsets), num_groups,
                                 packed_w.data_ptr(), h.data_ptr(), T, H, width, block_n,
                                 _stream()), "cd_moe_up")
    return h


def moe_up_pair(x_sorted: torch.Tensor, seg_offsets: torch.Tensor, num_groups: int,
                packed_w: torch.Tensor, width: int, packed_shared: torch.Tensor,
                width_shared: int, block_n: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Routed (grouped) and shared (dense) SwiGLU up-projections of the same rows in one
    launch; returns (h_routed [T, width], h_shared [T, width_shared])."""
    lib = _lib.load()
    _need(x_sorted, "x_sorted")
    _need(packed_w, "packed gate/up weights")
    _need(packed_shared, "packed shared gate/up weights")
    _need(seg_offsets, "seg_offsets", torch.int32)
    T, H = x_sorted.shape
    rows = lib.cd_gate_up_packed_rows(width, block_n)
    rows_s = lib.cd_gate_up_packed_rows(width_shared, block_n)
    if tuple(packed_w.shape) != (num_groups, rows, H) or tuple(packed_shared.shape) != (1, rows_s, H):
        raise RuntimeError("packed weights do not match the widths / tile width")
    h = torch.empty(T, width, dtype=BF16, device=x_sorted.device)
    h_s = torch.empty(T, width_shared, dtype=BF16, device=x_sorted.device)
    with _Span("moe_up_pair"):
        _lib.check(lib.cd_moe_up_pair(x_sorted.data_ptr(), seg_offsets.data_ptr(), num_groups,
                                      packed_w.data_ptr(), h.data_ptr(), width,
                                      packed_shared.data_ptr(), h_s.data_ptr(), width_shared, T, H,
                                      block_n, _stream()), "cd_moe_up_pair")
    return h, h_s


def _split_args(residual, residual_lo, T, H, want_lo, device):
    """Checks the low part of a split residual and allocates the low part of the output."""
    lo2 = None
    if residual_lo is not None:
        if residual is None:
            raise RuntimeError("residual_lo without residual")
        lo2 = residual_lo.reshape(-1, H)
        _need(lo2, "residual_lo")
        if lo2.shape[0] != T:
            raise RuntimeError("residual_lo rows do not match")
    out_lo = torch.empty(T, H, dtype=BF16, device=device) if want_lo else None
    return lo2, out_lo


def moe_down(h_routed: torch.Tensor, wd_routed: torch.Tensor, h_shared: Optional[torch.Tensor],
             wd_shared: Optional[torch.Tensor], seg_offsets: Optional[torch.Tensor],
             num_experts: int, row_map: Optional[torch.Tensor],
             residual: Optional[torch.Tensor], residual_lo: Optional[torch.Tensor] = None,
             want_lo: bool = False):
    """wd_routed: [E, H, I_e] (feature rows, I_e contiguous); wd_shared: [H, I_s].
    `residual_lo` / `want_lo`: split-bf16 residual stream; with want_lo returns (out, out_lo)."""
    lib = _lib.load()
    _need(h_routed, "h_routed")
    _need(wd_routed, "routed down weights")
    T, I_e = h_routed.shape
    E, H, I_e2 = wd_routed.shape
    if E != num_experts or I_e2 != I_e:
        raise RuntimeError("routed down weights do not match h_routed")
    I_s = 0
    if h_shared is not None:
        _need(h_shared, "h_shared")
        _need(wd_shared, "shared down weight")
        I_s = h_shared.shape[1]
        if tuple(wd_shared.shape) != (H, I_s) or h_shared.shape[0] != T:
            raise RuntimeError("shared down weight does not match h_shared")
    if seg_offsets is not None:
        _need(seg_offsets, "seg_offsets", torch.int32)
    if row_map is not None:
        _need(row_map, "row_map", torch.int32)
    res2 = None
    if residual is not None:
        res2 = residual.reshape(-1, H)
        _need(res2, "residual")
        if res2.shape[0] != T:
            raise RuntimeError("residual rows do not match")
    if row_map is not None and row_map.numel() != T:
        raise RuntimeError("row_map must have one entry per row")
    lo2, out_lo = _split_args(res2, residual_lo, T, H, want_lo, h_routed.device)
    out = torch.empty(T, H, dtype=BF16, device=h_routed.device)
    with _Span("moe_down"):
        _lib.check(lib.cd_moe_down(h_routed.data_ptr(), I_e, wd_routed.data_ptr(), _ptr(h_shared),
                                   I_s, _ptr(wd_shared), _ptr(seg_offsets), E, _ptr(row_map),
                                   _ptr(res2), _ptr(lo2), out.data_ptr(), _ptr(out_lo), T, H,
                                   _stream()), "cd_moe_down")
    return (out, out_lo) if want_lo else out


def push_rows(x_sorted: torch.Tensor, offsets: torch.Tensor, push_base: torch.Tensor,
              num_experts: int, experts_per_rank: int, peer_ptrs_dev: int) -> None:
    """Writes every expert-sorted row into the receive buffer of the GPU that owns its expert
    (peer-mapped memory; `peer_ptrs_dev` = device address of the array of buffer addresses)."""
    lib = _lib.load()
    _need(x_sorted, "x_sorted")
    _need(offsets, "offsets", torch.int32)
    _need(push_base, "push_base", torch.int32)
    T, H = x_sorted.shape
    with _Span("push_rows"):
        _lib.check(lib.cd_push_rows(x_sorted.data_ptr(), None, offsets.data_ptr(),
                                    push_base.data_ptr(), num_experts, experts_per_rank,
                                    peer_ptrs_dev, T, H, _stream()), "cd_push_rows")


def peer_put_i32(src: torch.Tensor, peer_bufs: torch.Tensor, world: int, offset: int) -> None:
    """Stores the int32 vector `src` at element `offset` of every rank's (peer-mapped) buffer
    (cd_peer_put_i32); visible to the peers after the next peer_barrier."""
    lib = _lib.load()
    _need(src, "src", torch.int32)
    _need(peer_bufs, "peer buffer addresses", torch.int64)
    with _Span("peer_put"):
        _lib.check(lib.cd_peer_put_i32(src.data_ptr(), src.numel(), peer_bufs.data_ptr(), world,
                                       int(offset), _stream()), "cd_peer_put_i32")


def ep_plan(all_counts: torch.Tensor, rank: int, experts_per_rank: int, ret_ptrs: torch.Tensor,
            row_bytes: int, capacity: int):
    """Exchange plan of the expert-parallel layer from the [ranks, E] count matrix, one launch
    (cd_ep_plan): returns (push_base int32 [E], seg_offsets int32 [El + 1], row_ptrs int64 [capacity])."""
    lib = _lib.load()
    _need(all_counts, "counts of all ranks", torch.int32)
    _need(ret_ptrs, "return buffer addresses", torch.int64)
    G, E = all_counts.shape
    dev = all_counts.device
    push_base = torch.empty(E, dtype=torch.int32, device=dev)
    seg_offsets = torch.empty(experts_per_rank + 1, dtype=torch.int32, device=dev)
    row_ptrs = torch.empty(capacity, dtype=torch.int64, device=dev)
    with _Span("ep_plan"):
        _lib.check(lib.cd_ep_plan(all_counts.data_ptr(), G, E, experts_per_rank, rank,
                                  ret_ptrs.data_ptr(), row_bytes, capacity, push_base.data_ptr(),
                                  seg_offsets.data_ptr(), row_ptrs.data_ptr(), _stream()), "cd_ep_plan")
    return push_base, seg_offsets, row_ptrs


def peer_barrier(flag_ptrs: torch.Tensor, flags: torch.Tensor, rank: int, world: int,
                 limit_ms: int = 2000, tag: str = "peer_barrier") -> None:
    """Cross-GPU barrier kernel (cd_peer_barrier); `flag_ptrs` int64 [world] addresses of the
    ranks' signal pads, `flags` this rank's pad (int32 [>= 1 + world])."""
    lib = _lib.load()
    _need(flag_ptrs, "flag_ptrs", torch.int64)
    _need(flags, "flags", torch.int32)
    if flag_ptrs.numel() != world or flags.numel() < 1 + world:
        raise RuntimeError("signal pad too small for the group")
    with _Span(tag):
        _lib.check(lib.cd_peer_barrier(flag_ptrs.data_ptr(), flags.data_ptr(), rank, world,
                                       int(limit_ms), _stream()), "cd_peer_barrier")


def moe_down_push(h_routed: torch.Tensor, wd_routed: torch.Tensor, seg_offsets: torch.Tensor,
                  num_experts: int, out_row_ptrs: torch.Tensor) -> None:
    """Routed down projection whose epilogue stores each row at its own address."""
    lib = _lib.load()
    _need(h_routed, "h_routed")
    _need(wd_routed, "routed down weights")
    _need(seg_offsets, "seg_offsets", torch.int32)
    _need(out_row_ptrs, "out_row_ptrs", torch.int64)
    T, I_e = h_routed.shape
    E, H, _ = wd_routed.shape
    if E != num_experts or out_row_ptrs.numel() != T:
        raise RuntimeError("moe_down_push: shapes do not match")
    with _Span("moe_down"):
        _lib.check(lib.cd_moe_down_push(h_routed.data_ptr(), I_e, wd_routed.data_ptr(),
                                        seg_offsets.data_ptr(), E, out_row_ptrs.data_ptr(), T, H,
                                        _stream()), "cd_moe_down_push")


def moe_combine(h_shared: torch.Tensor, wd_shared: torch.Tensor,
                routed_sorted: Optional[torch.Tensor], row_map: Optional[torch.Tensor],
                residual: Optional[torch.Tensor], residual_lo: Optional[torch.Tensor] = None,
                want_lo: bool = False):
    """Shared down projection + routed part (sorted order, from the expert GPUs) + residual.
    `residual_lo` / `want_lo` as in moe_down."""
    lib = _lib.load()
    _need(h_shared, "h_shared")
    _need(wd_shared, "shared down weight")
    T, I_s = h_shared.shape
    H = wd_shared.shape[0]
    if wd_shared.shape[1] != I_s:
        raise RuntimeError("shared down weight does not match h_shared")
    if routed_sorted is not None:
        _need(routed_sorted, "routed_sorted")
        if tuple(routed_sorted.shape) != (T, H):
            raise RuntimeError("routed_sorted does not match")
    if row_map is not None:
        _need(row_map, "row_map", torch.int32)
    res2 = None
    if residual is not None:
        res2 = residual.reshape(-1, H)
        _need(res2, "residual")
    lo2, out_lo = _split_args(res2, residual_lo, T, H, want_lo, h_shared.device)
    out = torch.empty(T, H, dtype=BF16, device=h_shared.device)
    with _Span("moe_combine"):
        _lib.check(lib.cd_moe_combine(h_shared.data_ptr(), I_s, wd_shared.data_ptr(),
                                      _ptr(routed_sorted), _ptr(row_map), _ptr(res2), _ptr(lo2),
                                      out.data_ptr(), _ptr(out_lo), T, H, _stream()),
                   "cd_moe_combine")
    return (out, out_lo) if want_lo else out


# device index -> the split-K workspace registered with the library (kept alive here; None =
# switched off by the caller)
_SPLIT_K_WS: dict = {}
_SPLIT_K_ROWS = 512          # calls of more rows never qualify (their tiles fill the SMs)
# the workspace form is opt-in (split_k(True), or CDEEP_SPLIT_K=1 for registration at first use): its
# workspace is shared by every stream of the device; the cluster form needs none and is always on
_SPLIT_K_AUTO = os.environ.get("CDEEP_SPLIT_K", "0") == "1"


def split_k(enable: bool = True, device: Optional[torch.device] = None) -> None:
    """Registers (or withdraws) the workspace that lets the few-row projections of a decode step
    cut their K loop over several CTAs (cd_splitk_workspace_set).  The workspace is shared by
    every call on the device: keep launches that may split on one stream."""
    lib = _lib.load()
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    with torch.cuda.device(dev):
        if enable:
            ws = torch.empty(lib.cd_splitk_workspace_bytes(), dtype=torch.uint8, device=dev)
            _lib.check(lib.cd_splitk_workspace_set(ws.data_ptr(), ws.numel(), _stream()),
                       "cd_splitk_workspace_set")
            _SPLIT_K_WS[dev.index] = ws
        else:
            _lib.check(lib.cd_splitk_workspace_set(None, 0, _stream()), "cd_splitk_workspace_set")
            torch.cuda.current_stream().synchronize()
            _SPLIT_K_WS[dev.index] = None      # stays off: the automatic registration skips this device


def split_k_config(flags: int = -1) -> int:
    """Which forms of split-K the few-row projections may take (cd_splitk_config): bit 0 the
    cluster form, bit 1 the workspace form; negative = query.  Returns the previous flags."""
    return _lib.load().cd_splitk_config(int(flags))


def _split_k_auto(x: torch.Tensor) -> None:
    # first few-row projection on a device: register the workspace (not while a graph is being
    # captured; the model's warm-up pass before the capture comes through here)
    if (_SPLIT_K_AUTO and x.shape[0] <= _SPLIT_K_ROWS and x.device.index not in _SPLIT_K_WS
            and not torch.cuda.is_current_stream_capturing()):
        split_k(True, x.device)


def mu_qkv(x: torch.Tensor, mu_prev: Optional[torch.Tensor], w: torch.Tensor,
           w_mu: Optional[torch.Tensor]) -> torch.Tensor:
    lib = _lib.load()
    _split_k_auto(x)
    _need(x, "x")
    _need(w, "qkv weight")
    T, H = x.shape
    N = w.shape[0]
    if mu_prev is not None:
        _need(mu_prev, "mu_prev")
        _need(w_mu, "mu qkv weight")
        if tuple(mu_prev.shape) != (T, H) or tuple(w_mu.shape) != (N, H):
            raise RuntimeError("mu_prev / mu weights do not match x / qkv weights")
    out = torch.empty(T, N, dtype=BF16, device=x.device)
    with _Span("mu_qkv"):
        _lib.check(lib.cd_mu_qkv(x.data_ptr(), _ptr(mu_prev), w.data_ptr(),
                                 _ptr(w_mu) if mu_prev is not None else None, out.data_ptr(), T,
                                 H, N, _stream()), "cd_mu_qkv")
    return out


def mu_qkv_rope(x: torch.Tensor, mu_prev: Optional[torch.Tensor], w: torch.Tensor,
                w_mu: Optional[torch.Tensor], q_w: Optional[torch.Tensor],
                k_w: Optional[torch.Tensor], cos: torch.Tensor, sin: torch.Tensor, eps: float,
                seq_len: int, pos0: int, hq: int, hkv: int, head_dim: int) -> torch.Tensor:
    """The mu-guided QKV projection with Q/K RMSNorm + RoPE applied before the output is
    rounded: the fused kernel where it applies, else cd_mu_qkv followed by cd_qk_norm_rope."""
    lib = _lib.load()
    T, H = x.shape
    N = w.shape[0]
    if not lib.cd_mu_qkv_rope_supported(T, N, hq, hkv, head_dim):
        qkv = mu_qkv(x, mu_prev, w, w_mu)
        return qk_norm_rope_(qkv, q_w, k_w, cos, sin, eps, seq_len, pos0, hq, hkv, head_dim)
    _need(x, "x")
    _need(w, "qkv weight")
    _need(cos, "cos", torch.float32)
    _need(sin, "sin", torch.float32)
    if mu_prev is not None:
        _need(mu_prev, "mu_prev")
        _need(w_mu, "mu qkv weight")
        if tuple(mu_prev.shape) != (T, H) or tuple(w_mu.shape) != (N, H):
            raise RuntimeError("mu_prev / mu weights do not match x / qkv weights")
    if q_w is not None:
        _need(q_w, "q_norm.weight")
        _need(k_w, "k_norm.weight")
    if cos.shape[0] < pos0 + seq_len or cos.shape[1] != head_dim:
        raise RuntimeError("cos/sin tables too short for the requested positions")
    out = torch.empty(T, N, dtype=BF16, device=x.device)
    with _Span("mu_qkv"):
        _lib.check(lib.cd_mu_qkv_rope(
            x.data_ptr(), _ptr(mu_prev), w.data_ptr(), _ptr(w_mu) if mu_prev is not None else None,
            out.data_ptr(), T, H, N, _ptr(q_w), _ptr(k_w), cos.data_ptr(), sin.data_ptr(),
            float(eps), seq_len, pos0, hq, hkv, head_dim, _stream()), "cd_mu_qkv_rope")
    return out


def mu_proj(h: torch.Tensor, w: torch.Tensor, mu_param: torch.Tensor, mu_min: float,
            mu_max: float, out_clamp: Optional[Tuple[float, float]] = None) -> torch.Tensor:
    lib = _lib.load()
    _need(h, "hidden_states")
    _need(w, "mu_proj.weight")
    _need(mu_param, "mu")
    _split_k_auto(h)
    T, H = h.shape
    out = torch.empty(T, H, dtype=BF16, device=h.device)
    lo, hi = out_clamp if out_clamp is not None else (0.0, 0.0)
    with _Span("mu_proj"):
        _lib.check(lib.cd_mu_proj(h.data_ptr(), w.data_ptr(), mu_param.data_ptr(), float(mu_min),
                                  float(mu_max), 1 if out_clamp is not None else 0, float(lo),
                                  float(hi), out.data_ptr(), T, H, _stream()), "cd_mu_proj")
    return out


def linear(x: torch.Tensor, w: torch.Tensor, residual: Optional[torch.Tensor] = None,
           tag: str = "linear", residual_lo: Optional[torch.Tensor] = None,
           want_lo: bool = False):
    """``x @ w^T (+ residual)``.  `residual_lo` / `want_lo`: split-bf16 residual stream; with
    want_lo returns (out, out_lo)."""
    lib = _lib.load()
    _need(x, "x")
    _need(w, "weight")
    _split_k_auto(x)
    T, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise RuntimeError("weight does not match x")
    if N % 8:
        # rows of the output must stay 16-byte aligned: compute into a padded buffer against
        # zero-padded weight rows and hand back the first N columns (e.g. an lm_head whose
        # vocabulary size is not a multiple of 8)
        if residual is not None or want_lo:
            raise RuntimeError("residual with an output width that is not a multiple of 8")
        pad = 8 - N % 8
        w_pad = torch.cat([w, w.new_zeros(pad, K)], dim=0)
        return linear(x, w_pad, None, tag)[:, :N]
    if residual is not None:
        _need(residual, "residual")
        if tuple(residual.shape) != (T, N):
            raise RuntimeError("residual does not match the output")
    lo2, out_lo = _split_args(residual, residual_lo, T, N, want_lo, x.device)
    out = torch.empty(T, N, dtype=BF16, device=x.device)
    with _Span(tag):
        _lib.check(lib.cd_linear(x.data_ptr(), w.data_ptr(), _ptr(residual), _ptr(lo2),
                                 out.data_ptr(), _ptr(out_lo), T, K, N, _stream()), "cd_linear")
    return (out, out_lo) if want_lo else out


# --------------------------------------------------------------------------- fp32 residual stream
# Decoders that keep the residual stream in fp32.  Operands are bf16, or fp32 when a model runs
# entirely in 32 bits; which one follows from the operand's dtype.
def _storage(t: torch.Tensor, name: str) -> int:
    """Checks an operand of either storage type; returns the C ABI's `fp32` flag."""
    if t.dtype not in (BF16, torch.float32):
        raise RuntimeError(f"{name}: expected dtype {BF16} or {torch.float32}, got {t.dtype}")
    _need(t, name, t.dtype)
    return 1 if t.dtype == torch.float32 else 0


def embed_rows(ids: torch.Tensor, table: torch.Tensor, width: int, ldx: int) -> torch.Tensor:
    """fp32 stream rows [T, ldx] = table[ids] (columns past `width` are zero)."""
    lib = _lib.load()
    ids = ids.reshape(-1).contiguous()
    _need(ids, "token_ids", torch.int64)
    fp32 = _storage(table, "embedding table")
    T = ids.numel()
    x = torch.empty(T, ldx, dtype=torch.float32, device=ids.device)
    with _Span("embed_rows"):
        _lib.check(lib.cd_embed_rows(ids.data_ptr(), table.data_ptr(), x.data_ptr(), T, table.shape[0],
                                     width, table.shape[1], ldx, fp32, _stream()), "cd_embed_rows")
    return x


def embed_positions(ids: torch.Tensor, table: torch.Tensor, pos_table: torch.Tensor, width: int, ldx: int,
                    seq_len: int, pos0: int, pos_dev: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 stream rows [T, ldx] = table[ids] + pos_table[position]; ids [B, seq_len], positions from
    pos0 (or the device scalar pos_dev) in every sequence."""
    lib = _lib.load()
    ids = ids.reshape(-1).contiguous()
    _need(ids, "token_ids", torch.int64)
    fp32 = _storage(table, "embedding table")
    _need(pos_table, "position table", table.dtype)
    if pos_table.shape[1] != table.shape[1]:
        raise RuntimeError("embedding and position tables differ in width")
    if pos_dev is None and pos0 + seq_len > pos_table.shape[0]:
        raise RuntimeError(f"position {pos0 + seq_len - 1} is beyond the {pos_table.shape[0]} learned ones")
    T = ids.numel()
    x = torch.empty(T, ldx, dtype=torch.float32, device=ids.device)
    with _Span("embed_rows"):
        _lib.check(lib.cd_embed_positions(ids.data_ptr(), table.data_ptr(), pos_table.data_ptr(), x.data_ptr(), T,
                                          table.shape[0], pos_table.shape[0], seq_len, pos0, _ptr(pos_dev), width,
                                          table.shape[1], ldx, fp32, _stream()), "cd_embed_positions")
    return x


def layernorm_f32(x: torch.Tensor, weight: torch.Tensor, eps: float, width: Optional[int] = None) -> torch.Tensor:
    """(x - mean) / sqrt(var + eps) * weight of an fp32 stream [T, ldx] into weight's dtype, over the first
    `width` columns (the rest of x and weight must be zero there)."""
    lib = _lib.load()
    _need(x, "x", torch.float32)
    fp32 = _storage(weight, "weight")
    T, ldx = x.shape
    if weight.numel() != ldx:
        raise RuntimeError("norm weight does not match the stream")
    out = torch.empty(T, ldx, dtype=weight.dtype, device=x.device)
    with _Span("layernorm_f32"):
        _lib.check(lib.cd_layernorm_f32(x.data_ptr(), weight.data_ptr(), float(eps), out.data_ptr(), T, width or ldx,
                                        ldx, fp32, _stream()), "cd_layernorm_f32")
    return out


def rmsnorm_f32(x: torch.Tensor, weight: torch.Tensor, eps: float, offset: float = 0.0,
                width: Optional[int] = None) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * (weight + offset) of an fp32 stream [T, ldx] into weight's dtype;
    the mean runs over the first `width` columns (the rest of x and weight must be zero there)."""
    lib = _lib.load()
    _need(x, "x", torch.float32)
    fp32 = _storage(weight, "weight")
    T, ldx = x.shape
    if weight.numel() != ldx:
        raise RuntimeError("norm weight does not match the stream")
    out = torch.empty(T, ldx, dtype=weight.dtype, device=x.device)
    with _Span("rmsnorm_f32"):
        _lib.check(lib.cd_rmsnorm_f32(x.data_ptr(), weight.data_ptr(), float(eps), float(offset),
                                      out.data_ptr(), T, width or ldx, ldx, fp32, _stream()),
                   "cd_rmsnorm_f32")
    return out


def _rows(x: torch.Tensor, name: str) -> int:
    """Checks a matrix whose rows may be columns of a wider buffer; returns the C ABI's `fp32` flag."""
    if not x.is_cuda or x.dim() != 2 or x.dtype not in (BF16, torch.float32) or x.stride(1) != 1:
        raise RuntimeError(f"{name}: expected rows of a CUDA {BF16} or {torch.float32} buffer")
    return 1 if x.dtype == torch.float32 else 0


def linear_to_f32(x: torch.Tensor, w: torch.Tensor, residual: Optional[torch.Tensor] = None,
                  col_scale: Optional[torch.Tensor] = None, inplace: bool = False,
                  tag: str = "linear_f32", scale: float = 1.0) -> torch.Tensor:
    """fp32 ``residual + scale * col_scale * (x @ w^T)``; operands bf16 (tcgen05) or fp32 (FMA pipe); x
    may be columns of a wider buffer.  inplace: the residual buffer itself receives the result."""
    lib = _lib.load()
    fp32 = _rows(x, "x")
    _need(w, "weight", x.dtype)
    T, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise RuntimeError("weight does not match x")
    if residual is not None:
        _need(residual, "residual", torch.float32)
        if tuple(residual.shape) != (T, N):
            raise RuntimeError("residual does not match the output")
    if col_scale is not None:
        _need(col_scale, "col_scale", x.dtype)
        if col_scale.numel() != N:
            raise RuntimeError("col_scale does not match the output")
    if not fp32:
        _split_k_auto(x)
    out = residual if inplace and residual is not None else torch.empty(T, N, dtype=torch.float32,
                                                                        device=x.device)
    with _Span(tag):
        if fp32:
            _lib.check(lib.cd_linear_f32(x.data_ptr(), x.stride(0), w.data_ptr(), _ptr(residual), _ptr(col_scale),
                                         float(scale), 0, out.data_ptr(), None, 1, T, K, N, _stream()), "cd_linear_f32")
        else:
            _lib.check(lib.cd_linear_f32out(x.data_ptr(), x.stride(0), w.data_ptr(), _ptr(residual), _ptr(col_scale),
                                            float(scale), out.data_ptr(), T, K, N, _stream()), "cd_linear_f32out")
    return out


ACTIVATIONS = {None: 0, "relu2": 1}     # codes of the C ABI


def project(x: torch.Tensor, w: torch.Tensor, tag: str = "linear", act: Optional[str] = None,
            out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(x @ w^T)`` in x's dtype (into `out` if given); x may be columns of a wider buffer."""
    lib = _lib.load()
    fp32 = _rows(x, "x")
    _need(w, "weight", x.dtype)
    T, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise RuntimeError("weight does not match x")
    if out is None:
        out = torch.empty(T, N, dtype=x.dtype, device=x.device)
    _need(out, "out", x.dtype)
    if tuple(out.shape) != (T, N):
        raise RuntimeError("out does not match x and the weight")
    if not fp32:
        _split_k_auto(x)
    with _Span(tag):
        if fp32:
            _lib.check(lib.cd_linear_f32(x.data_ptr(), x.stride(0), w.data_ptr(), None, None, 1.0, ACTIVATIONS[act],
                                         out.data_ptr(), None, 1, T, K, N, _stream()), "cd_linear_f32")
        else:
            _lib.check(lib.cd_project(x.data_ptr(), x.stride(0), w.data_ptr(), ACTIVATIONS[act], out.data_ptr(), T, K,
                                      N, _stream()), "cd_project")
    return out


def grouped_linear_f32(x: torch.Tensor, w: torch.Tensor, seg_offsets: torch.Tensor, tag: str) -> torch.Tensor:
    """fp32 ``x[rows of g] @ w[g]^T`` for the row ranges given by seg_offsets; w [G, N, K]."""
    lib = _lib.load()
    _need(x, "x", torch.float32)
    _need(w, "weights", torch.float32)
    _need(seg_offsets, "seg_offsets", torch.int32)
    (T, K), (G, N, K2) = x.shape, w.shape
    if K != K2 or seg_offsets.numel() != G + 1:
        raise RuntimeError("grouped weights do not match x / seg_offsets")
    out = torch.empty(T, N, dtype=torch.float32, device=x.device)
    with _Span(tag):
        _lib.check(lib.cd_linear_f32(x.data_ptr(), K, w.data_ptr(), None, None, 1.0, 0, out.data_ptr(),
                                     seg_offsets.data_ptr(), G, T, K, N, _stream()), "cd_linear_f32")
    return out


def glu_up(x: torch.Tensor, packed_w: torch.Tensor, width: int, block_n: int, alpha: float,
           limit: float, offset: float, seg_offsets: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Clamped gated unit on packed gate / up weights (pack_gate_up); with several groups the row
    ranges of x come from seg_offsets."""
    lib = _lib.load()
    _need(x, "x")
    _need(packed_w, "packed gate/up weights")
    T, H = x.shape
    G = packed_w.shape[0]
    if tuple(packed_w.shape[1:]) != (lib.cd_gate_up_packed_rows(width, block_n), H):
        raise RuntimeError("packed weights do not match the width / tile width")
    if seg_offsets is not None:
        _need(seg_offsets, "seg_offsets", torch.int32)
    if (seg_offsets is None and G != 1) or (seg_offsets is not None and seg_offsets.numel() != G + 1):
        raise RuntimeError("seg_offsets do not match the groups")
    h = torch.empty(T, width, dtype=BF16, device=x.device)
    with _Span("glu_up" if seg_offsets is None else "glu_up_routed"):
        _lib.check(lib.cd_glu_up(x.data_ptr(), _ptr(seg_offsets), G, packed_w.data_ptr(), h.data_ptr(), T, H, width,
                                 block_n, float(alpha), float(limit), float(offset), _stream()), "cd_glu_up")
    return h


def glu_f32(gate_up: torch.Tensor, alpha: float, limit: float, offset: float) -> torch.Tensor:
    """The clamped gated unit of fp32 pre-activations [T, 2 I] (gate columns, then up)."""
    lib = _lib.load()
    _need(gate_up, "gate_up", torch.float32)
    T, I = gate_up.shape[0], gate_up.shape[1] // 2
    h = torch.empty(T, I, dtype=torch.float32, device=gate_up.device)
    with _Span("glu_f32"):
        _lib.check(lib.cd_glu_f32(gate_up.data_ptr(), h.data_ptr(), T, I, float(alpha), float(limit),
                                  float(offset), _stream()), "cd_glu_f32")
    return h


# --------------------------------------------------------------------------- mixers
def _columns(t: torch.Tensor, name: str, dtype) -> int:
    """Address of a column slice of a row-major buffer."""
    if not t.is_cuda or t.dtype != dtype or t.dim() != 2 or t.stride(1) != 1:
        raise RuntimeError(f"{name}: expected columns of a CUDA {dtype} buffer")
    return t.data_ptr()


def window_attention_(proj: dict, out: torch.Tensor, weights: dict, ring_k: torch.Tensor,
                      ring_v: torch.Tensor, *, batch: int, seq_len: int, heads: int, kv_heads: int,
                      dim: int, vdim: int, window: int, keep: int, scale: float, eps: float,
                      out_scale: float, pos0: int, pos_dev: Optional[torch.Tensor] = None) -> None:
    """Attention of `seq_len` new tokens per sequence over a sliding window with kept first tokens
    (cd_window_attn).  proj: 'q', 'k', 'v' column slices of the projection buffer (may be normed in
    place); weights: 'q_norm', 'k_norm', 'r1', 'r2', 'talk'; the rings receive the new
    keys and values; `out` = columns of the mixers' output buffer."""
    lib = _lib.load()
    dt = out.dtype
    fp32 = 1 if dt == torch.float32 else 0
    q, k, v = proj["q"], proj["k"], proj["v"]
    dp, vp = ring_k.shape[3], ring_v.shape[3]
    if (q.shape != (batch * seq_len, heads * dp) or k.shape != (batch * seq_len, kv_heads * dp)
            or v.shape != (batch * seq_len, kv_heads * vp) or out.shape != (batch * seq_len, heads * vp)):
        raise RuntimeError("window attention: projection columns do not match the head layout")
    if q.stride(0) != k.stride(0) or q.stride(0) != v.stride(0):
        raise RuntimeError("window attention: q, k and v must share their row stride")
    _need(ring_k, "key ring", dt)
    _need(ring_v, "value ring", dt)
    for ring in (ring_k, ring_v):
        if tuple(ring.shape[:3]) != (batch, keep + window, kv_heads):
            raise RuntimeError("window attention: ring does not match batch / window / heads")
    for name, n in (("q_norm", dp), ("k_norm", dp), ("r1", heads), ("r2", heads), ("talk", heads * heads)):
        _need(weights[name], name, dt)
        if weights[name].numel() != n:
            raise RuntimeError(f"window attention: {name} has the wrong size")
    if pos_dev is not None and (pos_dev.dtype != torch.int32 or not pos_dev.is_cuda or pos_dev.numel() != 1):
        raise RuntimeError("pos_dev: expected one int32 on the device")
    a = _lib.WindowAttn(
        q=_columns(q, "q", dt), k=_columns(k, "k", dt), v=_columns(v, "v", dt), ldp=q.stride(0),
        q_w=weights["q_norm"].data_ptr(), k_w=weights["k_norm"].data_ptr(), r1=weights["r1"].data_ptr(),
        r2=weights["r2"].data_ptr(), talk=weights["talk"].data_ptr(), ring_k=ring_k.data_ptr(),
        ring_v=ring_v.data_ptr(), out=_columns(out, "out", dt), ldo=out.stride(0), pos_dev=_ptr(pos_dev),
        scale=float(scale), eps=float(eps), out_scale=float(out_scale), B=batch, S=seq_len, H=heads,
        G=kv_heads, dim=dim, dp=dp, vdim=vdim, vp=vp, window=window, keep=keep, pos0=pos0, normed=0)
    ref = ctypes.byref(a)
    ws_bytes = lib.cd_window_attention_decode_workspace_bytes(ref) if seq_len == 1 else 0
    if ws_bytes:
        ws = torch.empty(ws_bytes, dtype=torch.uint8, device=out.device)
        with _Span("window_attention_decode", 3):
            _lib.check(lib.cd_window_attention_decode(ref, ws.data_ptr(), ws_bytes, fp32, _stream()),
                       "cd_window_attention_decode")
        return
    with _Span("head_norm"):
        _lib.check(lib.cd_window_attention_norm(ref, fp32, _stream()), "cd_window_attention_norm")
    a.normed = 1
    if not fp32 and lib.cd_window_attention_prefill_supported(ref):
        with _Span("window_attention_prefill"):
            _lib.check(lib.cd_window_attention_prefill(ref, _stream()), "cd_window_attention_prefill")
    else:
        with _Span("window_attention_rows"):
            _lib.check(lib.cd_window_attention_rows(ref, fp32, _stream()), "cd_window_attention_rows")
    with _Span("window_append"):
        _lib.check(lib.cd_window_attention_append(ref, fp32, _stream()), "cd_window_attention_append")


_GLA_CHUNK_MIN = 16     # shorter portions walk token by token


def linear_attention_(proj: dict, out: torch.Tensor, weights: dict, state: torch.Tensor, *, batch: int,
                      seq_len: int, heads: int, dim: int, vdim: int, tau: float, eps: float,
                      out_scale: float) -> None:
    """Gated linear attention of `seq_len` new tokens per sequence (cd_linear_attn).  proj: 'q', 'k',
    'v', 'gate', 'inner' column slices; weights: 'a2', 'a2_b', 'norm'; `state` [B, heads, dkp, dvp]
    fp32 is carried on in place."""
    lib = _lib.load()
    dt = out.dtype
    fp32 = 1 if dt == torch.float32 else 0
    _need(state, "state", torch.float32)
    dkp, dvp = state.shape[2], state.shape[3]
    T = batch * seq_len
    want = {"q": heads * dkp, "k": heads * dkp, "v": heads * dvp, "gate": heads * dvp,
            "inner": proj["inner"].shape[1]}
    ldp = proj["q"].stride(0)
    for name, n in want.items():
        if tuple(proj[name].shape) != (T, n) or proj[name].stride(0) != ldp:
            raise RuntimeError(f"linear attention: {name} columns do not match the head layout")
    if tuple(out.shape) != (T, heads * dvp) or tuple(state.shape[:2]) != (batch, heads):
        raise RuntimeError("linear attention: output or state does not match the head layout")
    for name, n in (("a2", heads * dkp * want["inner"]), ("a2_b", heads * dkp), ("norm", dvp)):
        _need(weights[name], name, dt)
        if weights[name].numel() != n:
            raise RuntimeError(f"linear attention: {name} has the wrong size")
    a = _lib.LinearAttn(
        q=_columns(proj["q"], "q", dt), k=_columns(proj["k"], "k", dt), v=_columns(proj["v"], "v", dt),
        gate=_columns(proj["gate"], "gate", dt), inner=_columns(proj["inner"], "inner", dt), ldp=ldp,
        a2=weights["a2"].data_ptr(), a2_b=weights["a2_b"].data_ptr(), norm_w=weights["norm"].data_ptr(),
        state=state.data_ptr(), out=_columns(out, "out", dt), ldo=out.stride(0), inv_tau=1.0 / tau,
        eps=float(eps), out_scale=float(out_scale), q_scale=float(dim) ** -0.5, B=batch, S=seq_len,
        H=heads, dk=dim, dkp=dkp, dv=vdim, dvp=dvp, rank=want["inner"])
    ref = ctypes.byref(a)
    if seq_len == 1:
        with _Span("gla_step"):
            _lib.check(lib.cd_gla_step(ref, fp32, _stream()), "cd_gla_step")
        return
    log_decay = torch.empty(T, heads * dkp, dtype=torch.float32, device=out.device)
    a.log_decay = log_decay.data_ptr()
    with _Span("gla_decay"):
        _lib.check(lib.cd_gla_decay(ref, fp32, _stream()), "cd_gla_decay")
    ws_bytes = 0 if fp32 or seq_len < _GLA_CHUNK_MIN else lib.cd_gla_chunk_workspace_bytes(ref)
    if ws_bytes:
        ws = torch.empty(ws_bytes, dtype=torch.uint8, device=out.device)
        with _Span("gla_chunk", 3):
            _lib.check(lib.cd_gla_chunk(ref, ws.data_ptr(), ws_bytes, _stream()), "cd_gla_chunk")
        return
    o_raw = torch.empty(T, heads * dvp, dtype=torch.float32, device=out.device)
    a.o_raw = o_raw.data_ptr()
    with _Span("gla_sequence"):
        _lib.check(lib.cd_gla_sequence(ref, fp32, _stream()), "cd_gla_sequence")
    with _Span("gla_finish"):
        _lib.check(lib.cd_gla_finish(ref, fp32, _stream()), "cd_gla_finish")


def _need_pos_dev(pos_dev: Optional[torch.Tensor]) -> None:
    if pos_dev is not None and (pos_dev.dtype != torch.int32 or not pos_dev.is_cuda or pos_dev.numel() != 1):
        raise RuntimeError("pos_dev: expected one int32 on the device")


_LATENT_EXPAND_MIN = 64     # shorter portions attend in the latent's space


def _expand_latent(kv: torch.Tensor, cache: torch.Tensor, w: torch.Tensor, batch: int, seq_len: int,
                   pos0: int) -> torch.Tensor:
    """Unrotated keys and values [batch * (pos0 + seq_len), N] of all tokens so far: from the call's own
    normed latents where nothing is cached before them, else from the cache."""
    rank = w.shape[1]
    if pos0 == 0:
        return project(kv[:, :rank], w, tag="latent_expand")
    n = pos0 + seq_len
    out = torch.empty(batch * n, w.shape[0], dtype=w.dtype, device=w.device)
    for b in range(batch):
        project(cache[b, :n, :rank], w, tag="latent_expand", out=out[b * n:(b + 1) * n])
    return out


def latent_attention_(proj: dict, out: torch.Tensor, weights: dict, cache: torch.Tensor, *, batch: int, seq_len: int,
                      heads: int, dim: int, rot: int, rank: int, vdim: int, scale: float, eps: float,
                      out_scale: float, pos0: int, pos_dev: Optional[torch.Tensor] = None) -> None:
    """Latent attention of `seq_len` new tokens per sequence (cd_latent_attn).  proj: 'q', 'kv', 'gate'
    column slices (q and kv are changed in place); weights: 'norm', 'cos', 'sin', 'uk' [H, dimp, rankp],
    'uk_t' [H, rankp, dimp], 'uv' [H, vp, rankp], 'expand' [H * d64 + H * vp, rankp] (d64: dim rounded up to
    64, zero rows beyond dim); cache [B, capacity, rankp + rotp] receives the new rows."""
    lib = _lib.load()
    dt = out.dtype
    fp32 = 1 if dt == torch.float32 else 0
    q, kv, gate = proj["q"], proj["kv"], proj["gate"]
    uk, uk_t, uv = weights["uk"], weights["uk_t"], weights["uv"]
    dimp, rankp, vp = uk.shape[1], uk.shape[2], uv.shape[1]
    rotp = kv.shape[1] - rankp
    T = batch * seq_len
    if (tuple(q.shape) != (T, heads * (dimp + rotp)) or kv.shape[0] != T or rotp < rot or gate.shape[0] != T
            or gate.shape[1] < heads or tuple(out.shape) != (T, heads * vp)):
        raise RuntimeError("latent attention: projection columns do not match the head layout")
    if q.stride(0) != kv.stride(0) or q.stride(0) != gate.stride(0):
        raise RuntimeError("latent attention: q, kv and gate must share their row stride")
    for name, shape in (("uk", (heads, dimp, rankp)), ("uk_t", (heads, rankp, dimp)), ("uv", (heads, vp, rankp)),
                        ("norm", (rankp,))):
        _need(weights[name], name, dt)
        if tuple(weights[name].shape) != shape:
            raise RuntimeError(f"latent attention: {name} has the wrong shape")
    for name in ("cos", "sin"):
        _need(weights[name], name, torch.float32)
        if weights[name].shape[1] != rotp // 2:
            raise RuntimeError(f"latent attention: {name} does not match the rotated part")
    _need(weights["expand"], "expand", dt)
    if tuple(weights["expand"].shape) != (heads * (-(-dim // 64) * 64 + vp), rankp):
        raise RuntimeError("latent attention: expand has the wrong shape")
    _need(cache, "latent cache", dt)
    if cache.shape[0] != batch or cache.shape[2] != rankp + rotp:
        raise RuntimeError("latent attention: cache does not match batch / widths")
    _need_pos_dev(pos_dev)
    if pos_dev is None and pos0 + seq_len > min(cache.shape[1], weights["cos"].shape[0]):
        raise RuntimeError("latent attention: more tokens than the cache or the position tables hold")
    a = _lib.LatentAttn(
        q=_columns(q, "q", dt), kv=_columns(kv, "kv", dt), gate=_columns(gate, "gate", dt), ldp=q.stride(0),
        norm_w=weights["norm"].data_ptr(), cos_t=weights["cos"].data_ptr(), sin_t=weights["sin"].data_ptr(),
        uk=uk.data_ptr(), uk_t=uk_t.data_ptr(), uv=uv.data_ptr(), cache=cache.data_ptr(),
        out=_columns(out, "out", dt), ldo=out.stride(0), pos_dev=_ptr(pos_dev), scale=float(scale), eps=float(eps),
        out_scale=float(out_scale), B=batch, S=seq_len, H=heads, dim=dim, dimp=dimp, rot=rot, rotp=rotp, rank=rank,
        rankp=rankp, vdim=vdim, vp=vp, capacity=cache.shape[1], positions=weights["cos"].shape[0], pos0=pos0)
    ref = ctypes.byref(a)
    with _Span("latent_prepare"):
        _lib.check(lib.cd_latent_prepare(ref, fp32, _stream()), "cd_latent_prepare")
    if not fp32 and seq_len >= _LATENT_EXPAND_MIN and lib.cd_latent_prefill_supported(ref):
        expanded = _expand_latent(kv, cache, weights["expand"], batch, seq_len, pos0)
        with _Span("latent_prefill"):
            _lib.check(lib.cd_latent_prefill(ref, expanded.data_ptr(), _stream()), "cd_latent_prefill")
        return
    ws_bytes = 0 if fp32 else lib.cd_latent_decode_workspace_bytes(ref)
    if ws_bytes:
        ws = torch.empty(ws_bytes, dtype=torch.uint8, device=out.device)
        with _Span("latent_decode", 3):
            _lib.check(lib.cd_latent_decode(ref, ws.data_ptr(), ws_bytes, _stream()), "cd_latent_decode")
        return
    with _Span("latent_rows"):
        _lib.check(lib.cd_latent_rows(ref, fp32, _stream()), "cd_latent_rows")


_DELTA_CHUNK_MIN = 16       # shorter portions walk token by token


def delta_attention_(proj: dict, out: torch.Tensor, weights: dict, ring: torch.Tensor, state: torch.Tensor, *,
                     batch: int, seq_len: int, heads: int, kv_heads: int, dim: int, vdim: int, eps: float,
                     out_scale: float, pos0: int, pos_dev: Optional[torch.Tensor] = None) -> None:
    """Delta rule with per-channel decay over `seq_len` new tokens per sequence (cd_delta_attn).  proj: 'q',
    'k', 'v', 'b' and 'inner' column slices; weights: 'inner' [H * dkp + H * dvp, inner width] (from the
    inner projection to decay and gate inputs), 'taps' [taps, C], 'rate', 'dt_bias' (fp32), 'norm'; `ring`
    [B, taps, C] and `state` [B, H, dkp, dvp] fp32 are carried on in place."""
    lib = _lib.load()
    dt = out.dtype
    fp32 = 1 if dt == torch.float32 else 0
    _need(state, "state", torch.float32)
    _need(ring, "convolution ring", dt)
    dkp, dvp, taps = state.shape[2], state.shape[3], ring.shape[1]
    T, C = batch * seq_len, 2 * kv_heads * dkp + heads * dvp
    for name, n in (("q", kv_heads * dkp), ("k", kv_heads * dkp), ("v", heads * dvp)):
        if tuple(proj[name].shape) != (T, n) or proj[name].stride(0) != proj["b"].stride(0):
            raise RuntimeError(f"delta rule: {name} columns do not match the head layout")
    if proj["b"].shape[0] != T or proj["b"].shape[1] < heads or tuple(out.shape) != (T, heads * dvp):
        raise RuntimeError("delta rule: columns do not match the head layout")
    if tuple(state.shape[:2]) != (batch, heads) or ring.shape[0] != batch or ring.shape[2] != C:
        raise RuntimeError("delta rule: state or ring does not match the head layout")
    for name, n, d in (("taps", taps * C, dt), ("rate", heads, torch.float32),
                       ("dt_bias", heads * dkp, torch.float32), ("norm", dvp, dt)):
        _need(weights[name], name, d)
        if weights[name].numel() != n:
            raise RuntimeError(f"delta rule: {name} has the wrong size")
    if weights["inner"].shape[0] != heads * (dkp + dvp):
        raise RuntimeError("delta rule: inner weights do not match the head layout")
    _need_pos_dev(pos_dev)
    zg = linear_to_f32(proj["inner"], weights["inner"], tag="delta_inner")
    a = _lib.DeltaAttn(
        q=_columns(proj["q"], "q", dt), k=_columns(proj["k"], "k", dt), v=_columns(proj["v"], "v", dt),
        b=_columns(proj["b"], "b", dt), ldp=proj["b"].stride(0), zg=zg.data_ptr(), ldz=zg.shape[1],
        taps_w=weights["taps"].data_ptr(), rate=weights["rate"].data_ptr(), dt_bias=weights["dt_bias"].data_ptr(),
        norm_w=weights["norm"].data_ptr(), ring=ring.data_ptr(), state=state.data_ptr(),
        out=_columns(out, "out", dt), ldo=out.stride(0), pos_dev=_ptr(pos_dev), eps=float(eps), out_scale=float(out_scale), B=batch,
        S=seq_len, H=heads, G=kv_heads, dk=dim, dkp=dkp, dv=vdim, dvp=dvp, taps=taps, pos0=pos0)
    ref = ctypes.byref(a)
    if seq_len == 1 and lib.cd_delta_step_supported(ref):
        with _Span("delta_step"):
            _lib.check(lib.cd_delta_step(ref, fp32, _stream()), "cd_delta_step")
        return
    act = torch.empty(T, C, dtype=dt, device=out.device)
    inv = torch.empty(T, 2 * kv_heads, dtype=torch.float32, device=out.device)
    o_raw = torch.empty(T, heads * dvp, dtype=torch.float32, device=out.device)
    a.act, a.inv, a.o_raw = act.data_ptr(), inv.data_ptr(), o_raw.data_ptr()
    with _Span("delta_prepare"):
        _lib.check(lib.cd_delta_prepare(ref, fp32, _stream()), "cd_delta_prepare")
    ws_bytes = 0 if fp32 or seq_len < _DELTA_CHUNK_MIN else lib.cd_delta_chunk_workspace_bytes(ref)
    if ws_bytes:
        ws = torch.empty(ws_bytes, dtype=torch.uint8, device=out.device)
        with _Span("delta_chunk", 2):
            _lib.check(lib.cd_delta_chunk(ref, ws.data_ptr(), ws_bytes, _stream()), "cd_delta_chunk")
        with _Span("delta_finish"):
            _lib.check(lib.cd_delta_finish(ref, fp32, _stream()), "cd_delta_finish")
        return
    with _Span("delta_sequence"):
        _lib.check(lib.cd_delta_sequence(ref, fp32, _stream()), "cd_delta_sequence")
    with _Span("delta_finish"):
        _lib.check(lib.cd_delta_finish(ref, fp32, _stream()), "cd_delta_finish")


# --------------------------------------------------------------------------- learned routing
def route_top(logits: torch.Tensor, experts: int, top: int, groups: int = 1, keep: int = 1):
    """Experts [T, top] (int64) and weights [T, top] (fp32) from fp32 logits [T, >= experts] (cd_route_top)."""
    lib = _lib.load()
    _need(logits, "router logits", torch.float32)
    T = logits.shape[0]
    ids = torch.empty(T, top, dtype=torch.int64, device=logits.device)
    weights = torch.empty(T, top, dtype=torch.float32, device=logits.device)
    with _Span("route_top"):
        _lib.check(lib.cd_route_top(logits.data_ptr(), logits.shape[1], T, experts, groups, keep, top, ids.data_ptr(),
                                    weights.data_ptr(), _stream()), "cd_route_top")
    return ids, weights


def gather_div(x: torch.Tensor, perm: torch.Tensor, div: int) -> torch.Tensor:
    """out[i] = x[perm[i] // div]"""
    lib = _lib.load()
    _storage(x, "x")
    _need(perm, "perm", torch.int32)
    out = torch.empty(perm.numel(), x.shape[1], dtype=x.dtype, device=x.device)
    with _Span("gather_div"):
        _lib.check(lib.cd_gather_div(x.data_ptr(), perm.data_ptr(), div, out.data_ptr(), perm.numel(), x.shape[0],
                                     x.shape[1] * x.element_size(), _stream()), "cd_gather_div")
    return out


def combine_top_(stream: torch.Tensor, y: torch.Tensor, inv_perm: torch.Tensor, weights: torch.Tensor,
                 scale: float) -> torch.Tensor:
    """stream[t] += scale * sum_j weights[t, j] * y[inv_perm[t * top + j]]"""
    lib = _lib.load()
    fp32 = _storage(y, "y")
    _need(stream, "stream", torch.float32)
    _need(weights, "weights", torch.float32)
    _need(inv_perm, "inv_perm", torch.int32)
    T, top = weights.shape
    if tuple(y.shape) != (T * top, stream.shape[1]) or stream.shape[0] != T or inv_perm.numel() != T * top:
        raise RuntimeError("combine_top: shapes do not match")
    with _Span("combine_top"):
        _lib.check(lib.cd_combine_top(y.data_ptr(), inv_perm.data_ptr(), weights.data_ptr(), top, float(scale),
                                      stream.data_ptr(), T, stream.shape[1], fp32, _stream()), "cd_combine_top")
    return stream
