"""Small random Zukotar models for the tests, and checkpoints of them."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

from tensorwarp_b200 import checkpoint, dense
from tensorwarp_b200.models import zukotar


def latent(heads, dim, rot, vdim, rank, size=None, scale=0.2, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if size is not None:
        m["mask"] = {"size": size}
    return "latent_attention", m


def linear(heads, dim, vdim, tau=4.0):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def experts(n, top, ff, groups=None):
    router = {"experts": n, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(mixer, mlp):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(width, vocab, layers, loop=None, eps=1e-5, embed=1.0):
    out = {"architecture": "Zukotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed}, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


# no two sizes alike, nothing a multiple of what the kernels like, a layer without a feed-forward, one without a window,
# routers with several kept groups, one kept group and none; the loop starts at the first layer
UNEVEN = config(52, 131, [
    layer(linear(3, 20, 36, 4.0), experts(10, 4, 24, (5, 3))),
    layer(latent(5, 24, 6, 40, 37, 9, 0.3), experts(6, 2, 40, (3, 1))),
    layer(linear(2, 12, 7, 1.0), None),
    layer(latent(2, 33, 20, 12, 18, None, 0.15, 500.0), experts(7, 3, 9)),
], loop=(0, 2, 2), eps=3e-4, embed=3.0)
# windows around the 64-key tiles, heads and chunks of the tensor-core kernels' sizes; all experts are used, so that
# no choice can tip over between two precisions; the loop ends with the last layer
TILES = config(160, 300, [
    layer(latent(3, 64, 16, 64, 48, 64, 0.12), experts(3, 3, 48)),
    layer(linear(2, 64, 64, 16.0), experts(2, 2, 80)),
    layer(latent(2, 128, 64, 128, 96, 65, 0.08, 1e5), None),
    layer(linear(2, 128, 128, 8.0), experts(3, 3, 32)),
    layer(latent(4, 48, 32, 80, 64, 130, 0.1), experts(4, 4, 16)),
], loop=(3, 5, 2), embed=0.5)
# wider than the tensor-core kernels take, one head, more value than key columns
WIDE = config(96, 77, [
    layer(linear(1, 144, 160, 2.0), experts(5, 1, 64, (5, 1))),
    layer(latent(2, 160, 100, 272, 150, 33, 0.06), experts(4, 4, 20, (2, 2))),
    layer(linear(5, 16, 48, 32.0), experts(3, 3, 130)),
], loop=(1, 2, 3), embed=8.0)
CASES = {"uneven": UNEVEN, "tiles": TILES, "wide": WIDE}
RANKS = {"uneven": 5, "tiles": 16, "wide": 40}          # of the gated linear layers' low-rank projection


def spec(cfg, rank):
    return zukotar.parse_config(cfg, lambda name: (rank, cfg["width"]))


def weights(cfg, seed, rank):
    """Random tensors by name, bfloat16.  Score spreads of a few units, decays from slow to fast, routers that decide
    clearly: a lost key, a lost state or a wrong expert shows in the logits."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in zukotar.tensor_shapes(spec(cfg, rank)).items():
        leaf = name.split(".")[-1]
        if "norm" in leaf:
            t = rng.uniform(0.5, 1.5, shape)
        elif name.endswith("a2.b"):
            t = rng.uniform(-1.0, 6.0, shape)
        elif name in ("embed", "loop.step"):
            t = rng.standard_normal(shape)
        elif leaf == "router":
            t = rng.standard_normal(shape) / np.sqrt(shape[-1]) * 3.0
        else:
            t = rng.standard_normal(shape) / np.sqrt(shape[-1]) * 1.3
        out[name] = torch.from_numpy(np.asarray(t, np.float32)).to(torch.bfloat16)
    return out


def model(cfg, tensors, rank, dtype, device="cuda"):
    s = spec(cfg, rank)
    return dense.DenseModel(s, zukotar.model_tensors(s, lambda n, shape: tensors[n]), dtype, device)


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
