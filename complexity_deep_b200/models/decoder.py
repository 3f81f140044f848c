"""What the decoders with an fp32 residual stream and a carried ``DecoderState`` share: the step
function, states and their pool, and checkpoints in safetensors files."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, List, Optional, Union

import torch
import torch.nn as nn

from ..core._cache import DerivedCache
from ..core.padding import ROW_ALIGN, pad_rows, round_up
from ..core.state import DecoderState, StatePool
from .generation import GenerationMixin
from .modeling import CausalLMOutput
from .weights import read_safetensors, write_safetensors


class StreamDecoder(nn.Module, GenerationMixin):
    """A subclass sets ``config_class``, builds ``embed_tokens`` and ``layers`` (each with ``mixers`` and a
    ``forward(x, parts, state, batch, seq_len)`` that updates the stream in place) and implements the
    hooks below."""
    config_class = None

    def __init__(self, config) -> None:
        super().__init__()
        self.config = config
        self._derived = DerivedCache()

    # ------------------------------------------------------------------ hooks
    def embed(self, input_ids: torch.Tensor, state: DecoderState) -> torch.Tensor:
        """The fp32 stream [B * S, width padded] of the next tokens."""
        raise NotImplementedError

    def logits(self, x: torch.Tensor) -> torch.Tensor:
        """fp32 [rows, vocab] from the stream after the last layer."""
        raise NotImplementedError

    def checkpoint_names(self) -> Dict[str, Union[str, List[str]]]:
        """Parameter name -> tensor name in a checkpoint, or the names of its slices along dimension 0."""
        raise NotImplementedError

    @classmethod
    def sizes_from_tensors(cls, config, tensors: Dict[str, torch.Tensor]) -> None:
        """Fills in sizes that only the tensors' shapes give."""

    # ------------------------------------------------------------------ state
    def new_state(self, batch: int, capacity: Optional[int] = None) -> DecoderState:
        w = self.embed_tokens.weight
        return DecoderState([layer.mixers.new_state(batch, w.device, w.dtype, capacity) for layer in self.layers],
                            batch, w.device, capacity)

    def make_decode_cache(self, batch: int, capacity: int) -> DecoderState:
        """State for captured decode steps: the position is read on the device."""
        state = self.new_state(batch, capacity)
        state.device_position = True
        return state

    def state_pool(self, batch: int = 1) -> StatePool:
        return StatePool(lambda: self.new_state(batch))

    # ------------------------------------------------------------------ forward
    def padded_rows(self, name: str, w: torch.Tensor) -> torch.Tensor:
        """A [rows, width] weight padded to the stream's width."""
        return self._derived.get(name, (w,), lambda: pad_rows(
            w.detach(), round_up(w.shape[0], ROW_ALIGN), round_up(w.shape[1], ROW_ALIGN)))

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor, past_key_values: Optional[DecoderState] = None,
                use_cache: bool = False, logit_rows: Optional[torch.Tensor] = None) -> CausalLMOutput:
        """input_ids [B, S]: the next S tokens of B sequences.  ``past_key_values``: the state
        returned by an earlier call, which is carried on IN PLACE; None starts new sequences.
        ``logit_rows`` (indices into the B * S tokens) restricts the logits to those tokens, which
        then come back as [rows, vocab]."""
        B, S = input_ids.shape
        state = past_key_values if past_key_values is not None else self.new_state(B)
        if state.batch != B:
            raise ValueError(f"the state holds {state.batch} sequences, the call has {B}")
        if state.device_position and S != 1:
            raise RuntimeError("a device-side position takes one new token per sequence")
        x = self.embed(input_ids, state)
        for layer, parts in zip(self.layers, state.layers):
            x = layer(x, parts, state, B, S)
        state.advance(S)
        if logit_rows is not None:
            x = x[logit_rows].contiguous()
        if x.shape[0] == 0:
            return CausalLMOutput(logits=x.new_empty(0, self.config.vocab),
                                  past_key_values=state if use_cache else None)
        logits = self.logits(x)
        if logit_rows is None:
            logits = logits.unflatten(0, (B, S))
        return CausalLMOutput(logits=logits, past_key_values=state if use_cache else None)

    # ------------------------------------------------------------------ checkpoints
    @classmethod
    def from_pretrained(cls, path: str, device: str = "cpu", dtype: Optional[torch.dtype] = None) -> "StreamDecoder":
        """Loads config.json and model.safetensors; dtype None keeps bfloat16."""
        source = Path(path)
        config = cls.config_class.from_dict(json.loads((source / "config.json").read_text()))
        tensors = read_safetensors(source / "model.safetensors")
        cls.sizes_from_tensors(config, tensors)
        with torch.device("meta"):
            model = cls(config)
        dtype = dtype or torch.bfloat16
        names = model.checkpoint_names()
        params = dict(model.named_parameters())
        wanted = [n for v in names.values() for n in ([v] if isinstance(v, str) else v)]
        missing = [n for n in wanted if n not in tensors]
        extra = sorted(set(tensors) - set(wanted))
        if missing or extra:
            raise ValueError(f"checkpoint does not fit the config: missing {missing}, unexpected {extra}")
        state = {}
        for k, v in names.items():
            parts = [v] if isinstance(v, str) else v
            shape = params[k].shape if isinstance(v, str) else params[k].shape[1:]
            for n in parts:
                if tensors[n].shape != shape:
                    raise ValueError(f"{n}: shape {tuple(tensors[n].shape)}, the config implies {tuple(shape)}")
            whole = tensors[v] if isinstance(v, str) else torch.stack([tensors[n] for n in parts])
            state[k] = whole.to(device=device, dtype=dtype, copy=True)
        model.load_state_dict(state, strict=True, assign=True)
        return model.requires_grad_(False).eval()

    def save_pretrained(self, path: str) -> None:
        target = Path(path)
        target.mkdir(parents=True, exist_ok=True)
        (target / "config.json").write_text(json.dumps(self.config.to_dict(), indent=1))
        params = dict(self.named_parameters())
        tensors = {}
        for k, v in self.checkpoint_names().items():
            if isinstance(v, str):
                tensors[v] = params[k]
            else:
                tensors.update(zip(v, params[k]))
        write_safetensors(target / "model.safetensors", tensors)

    def num_parameters(self, trainable_only: bool = True) -> int:
        return sum(p.numel() for p in self.parameters() if p.requires_grad or not trainable_only)
