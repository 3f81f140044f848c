"""Pimezen: a decoder whose layers run sliding-window softmax attention and gated linear attention
side by side on the same input, followed by a clamped gated MLP (or none); layer scales on both
branches, tied embeddings, residual stream in fp32.

The mechanisms live in ``core`` (mixers, mlp, normalization, state) with their constants as
parameters; this file holds the configuration, the assembly and the names of the tensors in a
checkpoint.  Storage is bf16 (tensor-core kernels) or fp32 (every operation in 32 bits).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import torch
import torch.nn as nn

from .. import ops
from ..core._cache import DerivedCache
from ..core.mixers import GatedLinearAttention, ParallelMixers, WindowAttention
from ..core.mlp import ClampedGLU
from ..core.normalization import StreamNorm
from ..core.padding import pad_vector
from ..core.state import DecoderState
from .decoder import StreamDecoder


@dataclass
class WindowSpec:
    """Left mixer: sliding-window attention."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int

    @classmethod
    def from_dict(cls, d: dict) -> "WindowSpec":
        return cls(d["heads"], d["kv_heads"], d["dim"], d["vdim"], float(d["scale"]),
                   d["mask"]["size"], d["mask"].get("keep_first", 0))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                "scale": self.scale, "mask": {"size": self.window, "keep_first": self.keep_first}}


@dataclass
class LinearSpec:
    """Right mixer: gated linear attention."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16             # inner width of the decay projection (a checkpoint's tensors decide)

    @classmethod
    def from_dict(cls, d: dict) -> "LinearSpec":
        return cls(d["heads"], d["dim"], d["vdim"], float(d["tau"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}


@dataclass
class LayerSpec:
    left: WindowSpec
    right: LinearSpec
    left_scale: float
    right_scale: float
    ff: Optional[int]          # None: no feed-forward
    limit: float = 0.0

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d["type"] != "parallel":
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mix, mlp = d["mixer"], d.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        return cls(WindowSpec.from_dict(mix["left"]), LinearSpec.from_dict(mix["right"]),
                   float(mix["left_scale"]), float(mix["right_scale"]),
                   None if mlp is None else mlp["ff"], 0.0 if mlp is None else float(mlp["limit"]))

    def to_dict(self) -> dict:
        return {"type": "parallel",
                "mixer": {"left": self.left.to_dict(), "right": self.right.to_dict(),
                          "left_scale": self.left_scale, "right_scale": self.right_scale},
                "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff, "limit": self.limit}}


@dataclass
class PimezenConfig:
    vocab: int
    width: int
    eps: float
    layers: List[LayerSpec]

    architecture = "Pimezen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PimezenConfig":
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]),
                   [LayerSpec.from_dict(x) for x in d["layers"]])

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps}, "layers": [x.to_dict() for x in self.layers]}


class PimezenLayer(nn.Module):
    """x += ls1 * mixers(norm1(x)); x += ls2 * mlp(norm2(x)), in place on the fp32 stream."""

    def __init__(self, width: int, spec: LayerSpec, eps: float) -> None:
        super().__init__()
        L, R = spec.left, spec.right
        self.norm1 = StreamNorm(width, eps, offset=1.0)
        self.mixers = ParallelMixers(
            {"left": WindowAttention(width, L.heads, L.kv_heads, L.dim, L.vdim, L.window, L.keep_first,
                                     L.scale, eps),
             "right": GatedLinearAttention(width, R.heads, R.dim, R.vdim, R.rank, R.tau, eps)},
            {"left": spec.left_scale, "right": spec.right_scale})
        self.ls1 = nn.Parameter(torch.ones(width))
        self.mlp = None
        if spec.ff is not None:
            self.norm2 = StreamNorm(width, eps, offset=1.0)
            self.mlp = ClampedGLU(width, spec.ff, spec.limit)
            self.ls2 = nn.Parameter(torch.ones(width))
        self._derived = DerivedCache()

    def _scale(self, name: str, ldx: int) -> torch.Tensor:
        p = getattr(self, name)
        return self._derived.get(name, (p,), lambda: pad_vector(p.detach(), ldx))

    def forward(self, x: torch.Tensor, parts, state: DecoderState, batch: int, seq_len: int):
        x = self.mixers.run(self.norm1(x), x, self._scale("ls1", x.shape[1]), parts, state, batch, seq_len)
        if self.mlp is not None:
            x = self.mlp.run(self.norm2(x), x, self._scale("ls2", x.shape[1]))
        return x


class PimezenModel(StreamDecoder):
    config_class = PimezenConfig

    def __init__(self, config: PimezenConfig) -> None:
        super().__init__(config)
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.layers = nn.ModuleList(PimezenLayer(config.width, s, config.eps) for s in config.layers)
        self.norm = StreamNorm(config.width, config.eps, offset=1.0)
        for m in self.modules():
            if isinstance(m, (nn.Linear, nn.Embedding)):
                nn.init.normal_(m.weight, std=0.02)

    # ------------------------------------------------------------------ forward
    def embed(self, input_ids: torch.Tensor, state: DecoderState) -> torch.Tensor:
        table = self.padded_rows("table", self.embed_tokens.weight)
        return ops.embed_rows(input_ids, table, self.config.width, table.shape[1])

    def logits(self, x: torch.Tensor) -> torch.Tensor:
        table = self.padded_rows("table", self.embed_tokens.weight)
        return ops.linear_to_f32(self.norm(x), table, tag="linear_lm_head")[:, : self.config.vocab]

    # ------------------------------------------------------------------ checkpoints
    def checkpoint_names(self) -> Dict[str, str]:
        """Parameter name -> tensor name in a checkpoint."""
        names = {"embed_tokens.weight": "embed", "norm.weight": "final.norm"}
        left = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
                "q_norm": "q.norm", "k_norm": "k.norm", "r1": "r1", "r2": "r2", "talk": "talk"}
        right = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "g_proj.weight": "g",
                 "o_proj.weight": "o", "norm": "norm", "a1_proj.weight": "a1", "a2_proj.weight": "a2",
                 "a2_proj.bias": "a2.b"}
        mlp = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}
        for i, layer in enumerate(self.layers):
            a, b = f"layers.{i}.", f"l{i}."
            names[a + "norm1.weight"], names[a + "ls1"] = b + "norm1", b + "ls1"
            for branch, table in (("left", left), ("right", right)):
                for k, v in table.items():
                    names[f"{a}mixers.branches.{branch}.{k}"] = f"{b}mix.{branch}.{v}"
            if layer.mlp is not None:
                names[a + "norm2.weight"], names[a + "ls2"] = b + "norm2", b + "ls2"
                for k, v in mlp.items():
                    names[f"{a}mlp.{k}"] = f"{b}mlp.{v}"
        return names

    @classmethod
    def sizes_from_tensors(cls, config: PimezenConfig, tensors: Dict[str, torch.Tensor]) -> None:
        for i, layer in enumerate(config.layers):
            a1 = tensors.get(f"l{i}.mix.right.a1")
            if a1 is not None:                       # a missing tensor is reported by the loader
                layer.right.rank = a1.shape[0]
