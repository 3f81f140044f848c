"""Small Pimezen configurations and random checkpoints for the tests."""
import json

import numpy as np
import torch

from oracle import pimezen_oracle as po


def layer(heads, kv_heads, dim, vdim, size, keep, scale, r_heads, r_dim, r_vdim, tau, ls, rs, ff=None, limit=1.0):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                               "mask": {"size": size, "keep_first": keep}},
                      "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "tau": tau},
                      "left_scale": ls, "right_scale": rs},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(vocab, width, eps, layers):
    return {"architecture": "Pimezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # sizes that no power of two divides, a layer without feed-forward, layers that differ
    "odd": (config(101, 72, 1e-5, [
        layer(6, 2, 24, 40, 19, 3, 0.3, 3, 20, 24, 3.0, 0.7, 1.3, ff=100, limit=0.8),
        layer(3, 3, 12, 8, 7, 0, 0.25, 2, 36, 52, 16.0, 1.0, 0.5),
        layer(4, 1, 40, 16, 33, 5, 0.2, 5, 8, 16, 0.5, -0.4, 0.9, ff=52, limit=2.5)]), 5),
    # neither the width nor the vocabulary nor the feed-forward a multiple of 8
    "ragged": (config(67, 43, 1e-3, [
        layer(2, 1, 10, 6, 5, 1, 0.4, 1, 7, 9, 2.0, 1.1, 0.6, ff=29, limit=1.7),
        layer(2, 2, 6, 10, 11, 2, 0.4, 3, 5, 3, 8.0, 0.6, 1.0, ff=31, limit=0.6)]), 3),
    # wide heads, a window longer than most prompts, keep_first longer than the window
    "wide": (config(256, 256, 1e-6, [
        layer(4, 2, 128, 128, 300, 4, 0.09, 2, 128, 128, 16.0, 0.8, 0.8, ff=512, limit=4.0),
        layer(16, 4, 64, 64, 10, 24, 0.125, 4, 64, 64, 16.0, 1.0, 1.0, ff=320, limit=7.0)]), 16),
}


def bf16_weights(cfg, rank, seed=0):
    """Random weights rounded to bf16, as float64."""
    return {k: torch.tensor(v).to(torch.bfloat16).double().numpy()
            for k, v in po.random_weights(cfg, rank, seed).items()}


def write_checkpoint(path, cfg, weights):
    from complexity_deep_b200.models.weights import write_safetensors
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", {k: torch.tensor(v).to(torch.bfloat16) for k, v in weights.items()})
    return str(path)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)
