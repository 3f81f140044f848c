"""Which model class serves which checkpoint: the ``architecture`` entry of config.json (absent in
checkpoints of the reference, which hold a ComplexityModel)."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Optional, Type

import torch

from .modeling import ComplexityModel
from .pimezen import PimezenModel
from .rugedra import RugedraModel

DEFAULT_ARCHITECTURE = "Complexity"
MODELS: Dict[str, Type[torch.nn.Module]] = {
    DEFAULT_ARCHITECTURE: ComplexityModel,
    "Pimezen": PimezenModel,
    "Rugedra": RugedraModel,
}


def model_class(config: dict) -> Type[torch.nn.Module]:
    name = config.get("architecture", DEFAULT_ARCHITECTURE)
    if name not in MODELS:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(MODELS)}")
    return MODELS[name]


def load_model(path: str, device: str = "cuda", dtype: Optional[torch.dtype] = None) -> torch.nn.Module:
    """Loads the checkpoint folder `path` with the class that its config.json names."""
    cls = model_class(json.loads((Path(path) / "config.json").read_text()))
    if cls is ComplexityModel:
        model = cls.from_pretrained(path, device=device)
        return model.to(dtype or torch.bfloat16).eval()
    return cls.from_pretrained(path, device=device, dtype=dtype)
