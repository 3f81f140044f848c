"""Autoregressive generation shared by the model classes: sampling rules and the decode loop."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F


def sample_next(logits: torch.Tensor, temperature: float = 1.0, top_k: int = 50, top_p: float = 0.9,
                do_sample: bool = True) -> torch.Tensor:
    """Next token [B, 1] from the logits [B, V] of the last position; same filtering rules as the
    reference (complexity_deep/models/modeling.py:256-296): temperature, then top-k, then nucleus
    top-p that always keeps the best token."""
    scores = logits.float() / temperature
    if top_k > 0:
        kth = torch.topk(scores, min(top_k, scores.shape[-1])).values[..., -1:]
        scores = scores.masked_fill(scores < kth, float("-inf"))
    if top_p < 1.0:
        ordered, order = torch.sort(scores, descending=True)
        mass = torch.cumsum(F.softmax(ordered, dim=-1), dim=-1)
        drop = mass > top_p
        drop = torch.cat([torch.zeros_like(drop[..., :1]), drop[..., :-1]], dim=-1)
        scores = scores.masked_fill(drop.scatter(1, order, drop), float("-inf"))
    if do_sample:
        return torch.multinomial(F.softmax(scores, dim=-1), num_samples=1)
    return scores.argmax(dim=-1, keepdim=True)


class GenerationMixin:
    """``generate`` for a model whose forward takes ``past_key_values`` / ``use_cache`` and returns
    the logits together with the cache of all tokens seen so far."""

    @torch.no_grad()
    def generate(
        self,
        input_ids: torch.Tensor,
        max_new_tokens: int = 100,
        temperature: float = 1.0,
        top_k: int = 50,
        top_p: float = 0.9,
        do_sample: bool = True,
        eos_token_id: Optional[int] = None,
    ) -> torch.Tensor:
        """Autoregressive sampling with a cache; stops when every sequence of the batch has just
        produced the end token (the config's, unless given here; none if neither has one)."""
        eos = getattr(self.config, "eos_token_id", None) if eos_token_id is None else eos_token_id
        cache = None
        for _ in range(max_new_tokens):
            step_ids = input_ids if cache is None else input_ids[:, -1:]
            out = self.forward(step_ids, past_key_values=cache, use_cache=True)
            cache = out.past_key_values
            nxt = sample_next(out.logits[:, -1, :], temperature, top_k, top_p, do_sample)
            input_ids = torch.cat([input_ids, nxt], dim=-1)
            if eos is not None and bool((nxt == eos).all()):
                break
        return input_ids
