"""Small Rugedra configurations and random checkpoints for the tests."""
import json

import numpy as np
import torch

from oracle import rugedra_oracle as ro


def latent(heads, dim, rot, vdim, rank, scale, base, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "rot": {"base": base, "dims": rot}}}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}


def config(vocab, width, eps, mult, logit_scale, positions, layers):
    return {"architecture": "Rugedra", "vocab": vocab, "width": width, "max_positions": positions,
            "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale, "layers": layers}


CASES = {
    # sizes that no power of two divides, a layer without feed-forward, both kinds of layer in turn
    "odd": (config(101, 72, 1e-4, 0.6, 0.37, 400, [
        delta(4, 2, 24, 36, 3, moe(6, 3, 20, 0.8, (3, 2))),
        latent(3, 24, 12, 20, 40, 0.2, 500.0, dense(52)),
        latent(5, 8, 20, 24, 56, 0.25, 1e4),
        delta(3, 3, 40, 16, 4, dense(100)),
        latent(2, 40, 8, 48, 24, 0.15, 100.0, moe(10, 2, 36, 2.5, (5, 1)))]), 13),
    # neither the width nor the vocabulary nor any feed-forward a multiple of 8; one tap; no groups
    "ragged": (config(67, 43, 1e-3, 1.3, 1.7, 331, [
        latent(2, 10, 6, 9, 21, 0.3, 1000.0, moe(5, 1, 29, 0.6)),
        delta(3, 1, 7, 9, 1, dense(31)),
        delta(2, 2, 18, 5, 6, moe(9, 4, 13, 1.5, (3, 3)))]), 3),
    # heads of the sizes that the tensor-core forms are made for
    "wide": (config(256, 256, 1e-6, 0.8, 0.5, 512, [
        latent(6, 128, 64, 128, 256, 0.09, 1e5, moe(16, 4, 64, 3.0, (4, 2))),
        delta(4, 2, 128, 128, 4, dense(512)),
        latent(4, 64, 32, 96, 160, 0.11, 1e4, dense(320)),
        delta(3, 3, 64, 80, 2, moe(24, 6, 40, 1.2))]), 32),
}


def bf16_weights(cfg, rank, seed=0):
    """Random weights rounded to bf16, as float64."""
    return {k: torch.tensor(v).to(torch.bfloat16).double().numpy()
            for k, v in ro.random_weights(cfg, rank, seed).items()}


def write_checkpoint(path, cfg, weights):
    from complexity_deep_b200.models.weights import write_safetensors
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", {k: torch.tensor(v).to(torch.bfloat16) for k, v in weights.items()})
    return str(path)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)
