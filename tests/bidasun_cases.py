"""Small random Bidasun models for the tests, and checkpoints of them."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

from tensorwarp_b200 import checkpoint
from tensorwarp_b200.models import bidasun


def attention(heads, kv_heads, dim, vdim, size=None, keep_first=0, scale=0.2):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep_first}
    return m


def layer(mixer, ff):
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, max_positions=320, eps=1e-5):
    return {"architecture": "Bidasun", "width": width, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": eps},
            "layers": layers}


# no two sizes alike, nothing a multiple of what the kernels like, a layer without a feed-forward, one without a window
UNEVEN = config(52, 131, [
    layer(attention(4, 2, 24, 40, 9, 3, 0.3), 72),
    layer(attention(3, 1, 32, 12, 20, 0, 0.15), None),
    layer(attention(2, 2, 76, 144, 1, 5, 0.1), 50),
    layer(attention(6, 3, 10, 7), 33),
], eps=3e-4)
# windows and kept keys around the 64-key tiles
TILES = config(160, 300, [
    layer(attention(4, 2, 64, 64, 64, 1, 0.15), 192),
    layer(attention(4, 1, 128, 128, 65, 64, 0.1), 160),
    layer(attention(2, 2, 64, 96, 130, 70, 0.15), None),
    layer(attention(3, 3, 96, 64, 63, 65, 0.12), 128),
], max_positions=512)
# many query heads on one key/value head, heads wider than a tile's columns
WIDE = config(96, 77, [
    layer(attention(16, 1, 48, 32, 33, 2, 0.2), 64),
    layer(attention(10, 2, 160, 272, 50, 4, 0.08), 80),
], max_positions=256)
CASES = {"uneven": UNEVEN, "tiles": TILES, "wide": WIDE}


def weights(cfg, seed):
    """Random tensors by name, bfloat16.  Score spreads of a few units, distance biases that differ by head, sharp shifts:
    a lost key, a wrong distance or a lost state shows in the logits."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in bidasun.tensor_shapes(bidasun.parse_config(cfg)).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = rng.uniform(0.5, 1.5, shape)
        elif leaf == "shift":
            t = rng.uniform(-0.3, 1.0, shape)
        elif leaf == "r1":
            t = rng.uniform(0.05, 1.5, shape)
        elif leaf == "r2":
            t = rng.uniform(0.02, 0.5, shape)
        elif leaf == "pb":
            t = rng.uniform(-4.0, -1.0, shape)
        elif name in ("embed", "pos"):
            t = rng.standard_normal(shape)
        else:
            t = rng.standard_normal(shape) / np.sqrt(shape[-1]) * 1.3
        out[name] = torch.from_numpy(np.asarray(t, np.float32)).to(torch.bfloat16)
    return out


def save(folder, cfg, tensors):
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    checkpoint.write_safetensors(os.path.join(folder, "model.safetensors"), tensors)


def as_float64(tensors):
    return {k: v.double().numpy() for k, v in tensors.items()}


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def error(got, want):
    """Root mean square of the difference per row, in units of the expected logits' spread."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()
