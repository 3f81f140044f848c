"""Per-sequence state of decoders that mix several kinds of layer: rings of keys and values for window
attention, fp32 matrices for recurrences, rings of inputs for short convolutions, and latent rows that
grow with the sequence.

``StaticKVCache`` (core.attention) keeps every cached token; here each mixer of a layer declares
what it carries from call to call (``new_state``), ``DecoderState`` holds one such state per mixer
and layer together with the position, and ``StatePool`` hands the states out to requests and takes
them back."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


class WindowState:
    """Keys and values of the window and of the kept first tokens: ``keep + window`` slots per
    sequence.  Position j < keep stays in slot j, any other position sits in slot
    ``keep + (j - keep) % window`` until position j + window replaces it.  What a slot held before a
    reset is never read: visibility follows from the position alone."""

    def __init__(self, batch: int, window: int, keep: int, kv_heads: int, key_width: int,
                 value_width: int, device, dtype) -> None:
        slots = keep + window
        self.k = torch.zeros(batch, slots, kv_heads, key_width, dtype=dtype, device=device)
        self.v = torch.zeros(batch, slots, kv_heads, value_width, dtype=dtype, device=device)

    def reset(self) -> None:
        pass

    def copy_(self, other: "WindowState") -> None:
        self.k.copy_(other.k)
        self.v.copy_(other.v)


class RecurrentState:
    """fp32 matrices [batch, heads, rows, columns], zero at the start of a sequence."""

    def __init__(self, batch: int, heads: int, rows: int, cols: int, device) -> None:
        self.s = torch.zeros(batch, heads, rows, cols, dtype=torch.float32, device=device)

    def reset(self) -> None:
        self.s.zero_()

    def copy_(self, other: "RecurrentState") -> None:
        self.s.copy_(other.s)


class DeltaState(RecurrentState):
    """A recurrence's matrices together with the last inputs of the short convolution ahead of it:
    position p in slot ``p % taps``.  Slots of positions before 0 are never read."""

    def __init__(self, batch: int, heads: int, rows: int, cols: int, taps: int, channels: int, device,
                 dtype) -> None:
        super().__init__(batch, heads, rows, cols, device)
        self.ring = torch.zeros(batch, taps, channels, dtype=dtype, device=device)

    def copy_(self, other: "DeltaState") -> None:
        super().copy_(other)
        self.ring.copy_(other.ring)


class LatentState:
    """One row per cached token, shared by all heads: [batch, capacity, width].  The buffer grows by
    doubling up to `limit` rows; with a given capacity it is fixed (captured steps keep its address).
    Rows beyond the sequence's length are never read."""

    def __init__(self, batch: int, width: int, limit: int, device, dtype, capacity: Optional[int] = None) -> None:
        self.limit, self.fixed = limit, capacity is not None
        self.rows = torch.zeros(batch, min(capacity or 256, limit), width, dtype=dtype, device=device)

    def reserve(self, tokens: int) -> torch.Tensor:
        """The buffer, with room for `tokens` rows per sequence."""
        have = self.rows.shape[1]
        if tokens > have:
            if self.fixed or tokens > self.limit:
                raise RuntimeError(f"{tokens} tokens do not fit a cache of {have if self.fixed else self.limit}")
            grown = self.rows.new_zeros(self.rows.shape[0], min(max(tokens, 2 * have), self.limit), self.rows.shape[2])
            grown[:, :have] = self.rows
            self.rows = grown
        return self.rows

    def reset(self) -> None:
        pass

    def copy_(self, other: "LatentState") -> None:
        n = other.rows.shape[1]
        if not self.fixed:
            self.reserve(n)
        n = min(n, self.rows.shape[1])
        self.rows[:, :n] = other.rows[:, :n]


class DecoderState:
    """State of a batch of sequences of equal length: ``layers[i][name]`` is what mixer `name` of
    layer i carries.  ``length`` tokens have been seen; ``position`` mirrors it on the device so
    that a captured decode step can be replayed at any length (``device_position``)."""

    def __init__(self, layers: List[Dict[str, object]], batch: int, device,
                 capacity: Optional[int] = None) -> None:
        self.layers = layers
        self.batch = batch
        self.capacity = capacity          # None: unlimited
        self.length = 0
        self.position = torch.zeros(1, dtype=torch.int32, device=device)
        self.device_position = False

    def as_past(self) -> "DecoderState":
        return self

    def advance(self, tokens: int) -> None:
        """`tokens` more tokens per sequence have been processed (a captured step moves the
        device-side position instead, see ``advance_device``)."""
        if not self.device_position:
            self.length += tokens

    def advance_device(self) -> None:
        """Moves the device-side position by one token (stream ordered, capturable)."""
        self.position.add_(1)

    def reset(self) -> None:
        self.length = 0
        self.position.zero_()
        for layer in self.layers:
            for part in layer.values():
                part.reset()

    def set_length(self, length: int) -> None:
        """Only a restart is possible: a recurrence cannot be cut back."""
        if length != 0:
            raise ValueError("a DecoderState can only be set back to length 0")
        self.reset()

    def load(self, other: "DecoderState") -> None:
        """Takes over the contents of another state of the same batch."""
        if other.batch != self.batch or len(other.layers) != len(self.layers):
            raise ValueError("states of different shape")
        if self.capacity is not None and other.length > self.capacity:
            raise ValueError(f"{other.length} cached tokens do not fit a capacity of {self.capacity}")
        for mine, theirs in zip(self.layers, other.layers):
            for name, part in mine.items():
                part.copy_(theirs[name])
        self.length = other.length
        self.position.fill_(other.length)


class StatePool:
    """Hands out states to requests by id and takes them back; a returned state is reset and given
    to the next request."""

    def __init__(self, make) -> None:
        self._make = make
        self._free: List[DecoderState] = []
        self._live: Dict[str, DecoderState] = {}

    def get(self, request_id: str) -> DecoderState:
        state = self._live.get(request_id)
        if state is None:
            state = self._free.pop() if self._free else self._make()
            state.reset()
            self._live[request_id] = state
        return state

    def release(self, request_id: str) -> None:
        state = self._live.pop(request_id, None)
        if state is not None:
            self._free.append(state)

    def __len__(self) -> int:
        return len(self._live)
