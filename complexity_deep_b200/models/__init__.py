"""Model classes with the reference's names (complexity_deep/models/__init__.py:5-16)."""
from .config import ComplexityConfig
from .modeling import ComplexityModel, CausalLMOutput, ModelOutput
from .pimezen import PimezenConfig, PimezenModel
from .rugedra import RugedraConfig, RugedraModel
from .registry import load_model, model_class
from .utils import DecodeGraph, PrefillGraph, create_complexity_model, count_parameters

__all__ = ["ComplexityConfig", "ComplexityModel", "CausalLMOutput", "ModelOutput",
           "create_complexity_model", "count_parameters", "PrefillGraph", "DecodeGraph",
           "PimezenConfig", "PimezenModel", "RugedraConfig", "RugedraModel", "load_model", "model_class"]
