"""Zukotar: windowed latent attention and gated linear attention layers in any order, a stretch of layers that runs
several times, norms before and after each sublayer, grouped experts with squared-relu, tied output."""
from __future__ import annotations

from typing import Callable, Dict, Optional, Tuple

import torch

from .. import dense
from ..checkpoint import CheckpointError
from ..engine import DenseEngine
from ..registry import register
from .bidasun import _only


def _sizes(where: str, d: dict, *names):
    for n in names:
        if int(d[n]) < 1:
            raise CheckpointError(f"{where}: {n} = {d[n]}")
    return [int(d[n]) for n in names]


def _mixer(where: str, entry: dict, rank: Callable[[], int]):
    mx, kind = entry["mixer"], entry["type"]
    if kind == "latent_attention":
        _only(f"{where}: mixer", mx, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot", "mask"))
        mask, rot = mx.get("mask") or {}, mx["rot"]
        _only(f"{where}: mask", mask, ("size",))
        _only(f"{where}: rot", rot, ("base", "dims"))
        heads, dim, rot_dim, vdim, kv_rank = _sizes(where, mx, "heads", "dim", "rot_dim", "vdim", "kv_rank")
        if rot_dim % 2 or int(rot.get("dims", rot_dim)) != rot_dim:
            raise CheckpointError(f"{where}: {rot.get('dims')} of {rot_dim} rotated dimensions")
        window = int(mask["size"]) if mask.get("size") is not None else dense.UNBOUNDED_WINDOW
        if window < 1:
            raise CheckpointError(f"{where}: a window of {window}")
        return dense.LatentAttentionSpec(heads=heads, dim=dim, rot_dim=rot_dim, rot_base=float(rot["base"]), vdim=vdim, rank=kv_rank,
                                         scale=float(mx["scale"]), window=window)
    if kind == "gla":
        _only(f"{where}: mixer", mx, ("heads", "dim", "vdim", "tau"))
        heads, dim, vdim = _sizes(where, mx, "heads", "dim", "vdim")
        return dense.GatedLinearSpec(heads=heads, dim=dim, vdim=vdim, tau=float(mx["tau"]), rank=rank())
    raise CheckpointError(f"{where}: unknown mixer type {kind!r}")


def _feed_forward(where: str, mlp: Optional[dict]) -> Optional[dense.RoutedSpec]:
    if mlp is None:
        return None
    _only(f"{where}: mlp", mlp, ("kind", "expert", "router"))
    if mlp.get("kind", "moe") != "moe":
        raise CheckpointError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
    router, expert = mlp["router"], mlp["expert"]
    _only(f"{where}: router", router, ("experts", "top", "groups"))
    _only(f"{where}: expert", expert, ("ff",))
    groups = router.get("groups") or {"count": 1, "keep": 1}
    _only(f"{where}: groups", groups, ("count", "keep"))
    experts, top = _sizes(where, router, "experts", "top")
    count, keep = _sizes(where, groups, "count", "keep")
    if experts % count or keep > count or top > keep * (experts // count):
        raise CheckpointError(f"{where}: {top} of {experts} experts in {keep} of {count} groups")
    return dense.RoutedSpec(experts=experts, top=top, ff=_sizes(where, expert, "ff")[0], groups=count, keep=keep)


def parse_config(config: dict, shape: Callable[[str], Tuple[int, ...]]) -> dense.DecoderSpec:
    """shape: a tensor's shape by name; the low-rank size of a gated linear layer is only to be found there."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        where = f"layer {i}"
        mixer = _mixer(where, entry, lambda: int(shape(f"l{i}.mix.a1")[0]))
        layers.append(dense.LayerSpec(mixer=mixer, ff=_feed_forward(where, entry.get("mlp"))))
    loop = config.get("loop")
    if loop is not None:
        _only("loop", loop, ("start", "stop", "times"))
        loop = dense.LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
            raise CheckpointError(f"loop {loop.start} .. {loop.stop}, {loop.times} times over {len(layers)} layers")
    return dense.DecoderSpec(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]), layers=layers,
                             embed_scale=float((config.get("embedding") or {}).get("scale", 1.0)), loop=loop)


def tensor_shapes(spec: dense.DecoderSpec) -> Dict[str, Tuple[int, ...]]:
    """Every tensor of a checkpoint and its shape."""
    w = spec.width
    out = {"embed": (spec.vocab, w), "final.norm": (w,)}
    if spec.loop is not None:
        out["loop.step"] = (spec.loop.times, w)
    for i, layer in enumerate(spec.layers):
        m, p = layer.mixer, f"l{i}."
        x = p + "mix."
        vn = m.heads * m.vdim
        out.update({p + "norm1": (w,), p + "norm1b": (w,), x + "o": (w, vn)})
        if isinstance(m, dense.LatentAttentionSpec):
            out.update({x + "q": (m.heads * (m.dim + m.rot_dim), w), x + "dkv": (m.rank + m.rot_dim, w), x + "dkv.norm": (m.rank,),
                        x + "uk": (m.heads * m.dim, m.rank), x + "uv": (vn, m.rank), x + "g": (m.heads, w)})
        else:
            kn = m.heads * m.dim
            out.update({x + "q": (kn, w), x + "k": (kn, w), x + "v": (vn, w), x + "g": (vn, w), x + "norm": (m.vdim,),
                        x + "a1": (m.rank, w), x + "a2": (kn, m.rank), x + "a2.b": (kn,)})
        if layer.ff is not None:
            y = p + "mlp."
            out.update({p + "norm2": (w,), p + "norm2b": (w,), y + "router": (layer.ff.experts, w)})
            for e in range(layer.ff.experts):
                out.update({f"{y}e{e}.up": (layer.ff.ff, w), f"{y}e{e}.down": (w, layer.ff.ff)})
    return out


def model_tensors(spec: dense.DecoderSpec, get: Callable[[str, Tuple[int, ...]], torch.Tensor]) -> dense.ModelTensors:
    shapes = tensor_shapes(spec)

    def t(name):
        return get(name, shapes[name])

    def layer(i):
        p, m = f"l{i}.", spec.layers[i].mixer
        x = p + "mix."
        out = dense.LayerTensors(q=t(x + "q"), o=t(x + "o"), gate=t(x + "g"), pre1=t(p + "norm1"), norm1=t(p + "norm1b"))
        if isinstance(m, dense.LatentAttentionSpec):
            out.latent, out.latent_norm = t(x + "dkv"), t(x + "dkv.norm")
            out.expand_k, out.expand_v = t(x + "uk"), t(x + "uv")
        else:
            out.k, out.v, out.head_norm = t(x + "k"), t(x + "v"), t(x + "norm")
            out.low, out.decay, out.decay_bias = t(x + "a1"), t(x + "a2"), t(x + "a2.b")
        if spec.layers[i].ff is not None:
            out.pre2, out.norm2, out.router = t(p + "norm2"), t(p + "norm2b"), t(p + "mlp.router")
            out.expert = lambda e: (t(f"{p}mlp.e{e}.up"), t(f"{p}mlp.e{e}.down"))
        return out

    return dense.ModelTensors(embed=t("embed"), pos=None, final_norm=t("final.norm"), head=None, layer=layer,
                              step=t("loop.step") if spec.loop is not None else None)


@register("Zukotar")
def build(config: dict, weights, dtype: torch.dtype = torch.bfloat16, device="cuda", **engine_options) -> DenseEngine:
    if weights is None:
        raise CheckpointError("Zukotar needs model.safetensors beside config.json")
    spec = parse_config(config, weights.shape)
    return DenseEngine(dense.DenseModel(spec, model_tensors(spec, weights.get), dtype, device), **engine_options)
