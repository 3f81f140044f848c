"""Rugedra: a pre-norm decoder whose layers are latent attention or the gated delta rule with per-channel
decay, each followed by a squared-relu MLP, a mixture of clamped gated experts, or nothing.  Learned
position vectors, layer norms without a bias, one residual multiplier, an untied and scaled output
projection, residual stream in fp32.

The mechanisms live in ``core`` (mixers, mlp, routed_experts, normalization, state) with their constants
as parameters; this file holds the configuration, the assembly and the names of the tensors in a
checkpoint.  Storage is bf16 (tensor-core kernels) or fp32 (every operation in 32 bits).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Union

import torch
import torch.nn as nn

from .. import ops
from ..core.mixers import DeltaRule, LatentAttention, ParallelMixers
from ..core.mlp import SquaredReLU
from ..core.normalization import StreamNorm
from ..core.routed_experts import RoutedExperts
from ..core.state import DecoderState
from .decoder import StreamDecoder


@dataclass
class LatentSpec:
    """Latent attention."""
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    scale: float
    rot_dims: int
    rot_base: float

    kind = "latent_attention"

    @classmethod
    def from_dict(cls, d: dict) -> "LatentSpec":
        return cls(d["heads"], d["dim"], d["rot_dim"], d["vdim"], d["kv_rank"], float(d["scale"]), d["rot"]["dims"],
                   float(d["rot"]["base"]))

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot, "vdim": self.vdim, "kv_rank": self.rank,
                "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dims}}

    def build(self, width: int, positions: int, eps: float) -> LatentAttention:
        return LatentAttention(width, self.heads, self.dim, self.rot, self.vdim, self.rank, self.scale, self.rot_dims,
                               self.rot_base, positions, eps)

    tensors = {"q_proj.weight": "q", "kv_proj.weight": "dkv", "kv_norm": "dkv.norm", "uk_proj.weight": "uk",
               "uv_proj.weight": "uv", "g_proj.weight": "g", "o_proj.weight": "o"}


@dataclass
class DeltaSpec:
    """Gated delta rule with a decay per key channel."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    rank: int = 16             # inner widths of the decay and gate projections (a checkpoint's tensors
    gate_rank: int = 16        # decide)

    kind = "channel_delta"

    @classmethod
    def from_dict(cls, d: dict) -> "DeltaSpec":
        return cls(d["heads"], d["kv_heads"], d["dim"], d["vdim"], d["conv"])

    def to_dict(self) -> dict:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.taps}

    def build(self, width: int, positions: int, eps: float) -> DeltaRule:
        return DeltaRule(width, self.heads, self.kv_heads, self.dim, self.vdim, self.taps, self.rank, self.gate_rank, eps)

    tensors = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "q_conv": "q.conv",
               "k_conv": "k.conv", "v_conv": "v.conv", "b_proj.weight": "b", "a1_proj.weight": "a1",
               "a2_proj.weight": "a2", "A_log": "A_log", "dt_bias": "dt_bias", "g1_proj.weight": "g1",
               "g2_proj.weight": "g2", "norm": "norm", "o_proj.weight": "o"}


@dataclass
class DenseSpec:
    """Squared-relu MLP."""
    ff: int

    @classmethod
    def from_dict(cls, d: dict) -> "DenseSpec":
        return cls(d["ff"])

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}

    def build(self, width: int) -> SquaredReLU:
        return SquaredReLU(width, self.ff)

    def tensors(self) -> Dict[str, Union[str, List[str]]]:
        return {"up_proj.weight": "up", "down_proj.weight": "down"}


@dataclass
class ExpertsSpec:
    """Mixture of clamped gated experts."""
    ff: int
    limit: float
    experts: int
    top: int
    groups: Optional[int] = None     # None: no groups in the config
    keep: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "ExpertsSpec":
        r = d["router"]
        g = r.get("groups") or {}
        return cls(d["expert"]["ff"], float(d["expert"]["limit"]), r["experts"], r["top"], g.get("count"), g.get("keep"))

    def to_dict(self) -> dict:
        router = {"experts": self.experts, "top": self.top}
        if self.groups is not None:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": router}

    def build(self, width: int) -> RoutedExperts:
        return RoutedExperts(width, self.ff, self.experts, self.top, self.limit, self.groups or 1, self.keep or 1)

    def tensors(self) -> Dict[str, Union[str, List[str]]]:
        names = {"router.weight": "router"}
        for n in ("gate", "up", "down"):
            names[n + "_proj"] = [f"e{e}.{n}" for e in range(self.experts)]
        return names


MIXERS = {c.kind: c for c in (LatentSpec, DeltaSpec)}
MLPS = {"dense": DenseSpec, "moe": ExpertsSpec}


@dataclass
class LayerSpec:
    mixer: Union[LatentSpec, DeltaSpec]
    mlp: Union[DenseSpec, ExpertsSpec, None]

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp is not None and mlp["kind"] not in MLPS:
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        return cls(MIXERS[d["type"]].from_dict(d["mixer"]), None if mlp is None else MLPS[mlp["kind"]].from_dict(mlp))

    def to_dict(self) -> dict:
        return {"type": self.mixer.kind, "mixer": self.mixer.to_dict(),
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass
class RugedraConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    residual_mult: float
    logit_scale: float
    layers: List[LayerSpec]

    architecture = "Rugedra"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "RugedraConfig":
        return cls(d["vocab"], d["width"], d["max_positions"], float(d["norm"]["eps"]), float(d["residual_mult"]),
                   float(d["logit_scale"]), [LayerSpec.from_dict(x) for x in d["layers"]])

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "max_positions": self.max_positions, "norm": {"eps": self.eps}, "residual_mult": self.residual_mult,
                "logit_scale": self.logit_scale, "layers": [x.to_dict() for x in self.layers]}


class RugedraLayer(nn.Module):
    """x += m * mixer(norm1(x)); x += m * mlp(norm2(x)), in place on the fp32 stream."""

    def __init__(self, spec: LayerSpec, config: RugedraConfig) -> None:
        super().__init__()
        self.mult = config.residual_mult
        self.norm1 = StreamNorm(config.width, config.eps, centred=True)
        self.mixers = ParallelMixers({"mix": spec.mixer.build(config.width, config.max_positions, config.eps)},
                                     {"mix": 1.0})
        self.mlp = None
        if spec.mlp is not None:
            self.norm2 = StreamNorm(config.width, config.eps, centred=True)
            self.mlp = spec.mlp.build(config.width)

    def forward(self, x: torch.Tensor, parts, state: DecoderState, batch: int, seq_len: int):
        x = self.mixers.run(self.norm1(x), x, None, parts, state, batch, seq_len, scale=self.mult)
        if self.mlp is not None:
            x = self.mlp.run(self.norm2(x), x, scale=self.mult)
        return x


class RugedraModel(StreamDecoder):
    config_class = RugedraConfig

    def __init__(self, config: RugedraConfig) -> None:
        super().__init__(config)
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.embed_positions = nn.Embedding(config.max_positions, config.width)
        self.layers = nn.ModuleList(RugedraLayer(s, config) for s in config.layers)
        self.norm = StreamNorm(config.width, config.eps, centred=True)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
        for m in self.modules():
            if isinstance(m, (nn.Linear, nn.Embedding)):
                nn.init.normal_(m.weight, std=0.02)

    def new_state(self, batch: int, capacity: Optional[int] = None) -> DecoderState:
        if capacity is not None and capacity > self.config.max_positions:
            raise ValueError(f"a capacity of {capacity} tokens, but the model has {self.config.max_positions} positions")
        return super().new_state(batch, capacity)

    # ------------------------------------------------------------------ forward
    def embed(self, input_ids: torch.Tensor, state: DecoderState) -> torch.Tensor:
        table = self.padded_rows("table", self.embed_tokens.weight)
        positions = self.padded_rows("positions", self.embed_positions.weight)
        if state.length + input_ids.shape[1] > self.config.max_positions:
            raise RuntimeError(f"the model has {self.config.max_positions} positions")
        return ops.embed_positions(input_ids, table, positions, self.config.width, table.shape[1], input_ids.shape[1],
                                   0 if state.device_position else state.length,
                                   state.position if state.device_position else None)

    def logits(self, x: torch.Tensor) -> torch.Tensor:
        head = self.padded_rows("head", self.lm_head.weight)
        return ops.linear_to_f32(self.norm(x), head, tag="linear_lm_head",
                                 scale=self.config.logit_scale)[:, : self.config.vocab]

    # ------------------------------------------------------------------ checkpoints
    def checkpoint_names(self):
        names = {"embed_tokens.weight": "embed", "embed_positions.weight": "pos", "norm.weight": "final.norm",
                 "lm_head.weight": "head"}
        for i, spec in enumerate(self.config.layers):
            a, b = f"layers.{i}.", f"l{i}."
            names[a + "norm1.weight"] = b + "norm1"
            for k, v in spec.mixer.tensors.items():
                names[f"{a}mixers.branches.mix.{k}"] = f"{b}mix.{v}"
            if spec.mlp is not None:
                names[a + "norm2.weight"] = b + "norm2"
                for k, v in spec.mlp.tensors().items():
                    names[f"{a}mlp.{k}"] = f"{b}mlp.{v}" if isinstance(v, str) else [f"{b}mlp.{n}" for n in v]
        return names

    @classmethod
    def sizes_from_tensors(cls, config: RugedraConfig, tensors: Dict[str, torch.Tensor]) -> None:
        for i, layer in enumerate(config.layers):
            for name, field in (("a1", "rank"), ("g1", "gate_rank")):
                t = tensors.get(f"l{i}.mix.{name}")
                if isinstance(layer.mixer, DeltaSpec) and t is not None:   # a missing tensor is reported by the loader
                    setattr(layer.mixer, field, t.shape[0])
