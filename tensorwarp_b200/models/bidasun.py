"""Bidasun: learned positions, token shift, windowed sigmoid attention with kept first keys and a
logarithmic distance bias, output gate, tanh-GELU gated feed-forward, RMS norms on sublayer outputs only."""
from __future__ import annotations

from typing import Callable, Dict, Tuple

import torch

from .. import dense
from ..checkpoint import CheckpointError
from ..engine import DenseEngine
from ..registry import register


def _only(where: str, d: dict, known) -> None:
    extra = sorted(set(d) - set(known))
    if extra:
        raise CheckpointError(f"{where}: unknown keys {', '.join(extra)}")


def parse_config(config: dict) -> dense.DecoderSpec:
    layers = []
    for i, entry in enumerate(config["layers"]):
        if entry["type"] != "attention":
            raise CheckpointError(f"layer {i}: unknown mixer type {entry['type']!r}")
        mx = entry["mixer"]
        _only(f"layer {i}: mixer", mx, ("heads", "kv_heads", "dim", "vdim", "scale", "mask"))
        mask = mx.get("mask") or {}
        _only(f"layer {i}: mask", mask, ("size", "keep_first"))
        if mx["kv_heads"] < 1 or mx["heads"] % mx["kv_heads"]:
            raise CheckpointError(f"layer {i}: {mx['heads']} query heads over {mx['kv_heads']} key/value heads")
        mlp = entry.get("mlp")
        if mlp is not None:
            _only(f"layer {i}: mlp", mlp, ("kind", "ff"))
            if mlp.get("kind", "dense") != "dense":
                raise CheckpointError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        mixer = dense.AttentionSpec(heads=int(mx["heads"]), kv_heads=int(mx["kv_heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]),
                                    scale=float(mx["scale"]), window=int(mask.get("size", dense.UNBOUNDED_WINDOW)),
                                    keep_first=int(mask.get("keep_first", 0)))
        layers.append(dense.LayerSpec(mixer=mixer, ff=int(mlp["ff"]) if mlp is not None else None))
    return dense.DecoderSpec(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]),
                             max_positions=int(config["max_positions"]), layers=layers)


def tensor_shapes(spec: dense.DecoderSpec) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape."""
    w = spec.width
    out = {"embed": (spec.vocab, w), "pos": (spec.max_positions, w), "final.norm": (w,), "head": (spec.vocab, w)}
    for i, layer in enumerate(spec.layers):
        m, p = layer.mixer, f"l{i}."
        qn, kn, vn, on = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim, m.heads * m.vdim
        out.update({p + "norm1": (w,), p + "shift": (w,), p + "mix.q": (qn, w), p + "mix.k": (kn, w), p + "mix.v": (vn, w),
                    p + "mix.g": (on, w), p + "mix.o": (w, on), p + "mix.q.norm": (qn,), p + "mix.k.norm": (kn,),
                    p + "mix.r1": (m.heads,), p + "mix.r2": (m.heads,), p + "mix.pb": (m.heads,)})
        if layer.ff is not None:
            out.update({p + "norm2": (w,), p + "mlp.gate": (layer.ff, w), p + "mlp.up": (layer.ff, w), p + "mlp.down": (w, layer.ff)})
    return out


def model_tensors(spec: dense.DecoderSpec, get: Callable[[str, Tuple[int, ...]], torch.Tensor]) -> dense.ModelTensors:
    shapes = tensor_shapes(spec)

    def t(name):
        return get(name, shapes[name])

    def layer(i):
        p, ff = f"l{i}.", spec.layers[i].ff is not None
        return dense.LayerTensors(
            q=t(p + "mix.q"), k=t(p + "mix.k"), v=t(p + "mix.v"), gate=t(p + "mix.g"), o=t(p + "mix.o"),
            q_norm=t(p + "mix.q.norm"), k_norm=t(p + "mix.k.norm"), r1=t(p + "mix.r1"), r2=t(p + "mix.r2"), pb=t(p + "mix.pb"),
            shift=t(p + "shift"), norm1=t(p + "norm1"), norm2=t(p + "norm2") if ff else None,
            mlp_gate=t(p + "mlp.gate") if ff else None, mlp_up=t(p + "mlp.up") if ff else None,
            mlp_down=t(p + "mlp.down") if ff else None)

    return dense.ModelTensors(embed=t("embed"), pos=t("pos"), final_norm=t("final.norm"), head=t("head"), layer=layer)


@register("Bidasun")
def build(config: dict, weights, dtype: torch.dtype = torch.bfloat16, device="cuda", **engine_options) -> DenseEngine:
    if weights is None:
        raise CheckpointError("Bidasun needs model.safetensors beside config.json")
    spec = parse_config(config)
    return DenseEngine(dense.DenseModel(spec, model_tensors(spec, weights.get), dtype, device), **engine_options)
