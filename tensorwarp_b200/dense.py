"""Decoder models with dense 16-bit or 32-bit weights: what a model is made of, and its weights on the device.

A model file in ``models/`` describes its design as a ``DecoderSpec``, whose mechanisms are
parameters (a None leaves one out), and names its tensors; everything else (padding, fusion, the cache,
the step) is shared.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Tuple, Union

import torch

from . import _dense

UNBOUNDED_WINDOW = 1 << 30


# ------------------------------------------------------------------- designs --
@dataclass
class AttentionSpec:
    """Sigmoid attention.  Weight of key j for query i: sigmoid(scale * q.k - r1 * ln(1 + r2 * (i - j)) + pb), not
    normalised; visible when j <= i and (i - j < window or j < keep_first)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = UNBOUNDED_WINDOW
    keep_first: int = 0


@dataclass
class LatentAttentionSpec:
    """Softmax attention over keys and values that every head maps from one normed latent of `rank` numbers per token,
    plus `rot_dim` rotated dimensions whose key part all heads share; one sigmoid gate per head."""
    heads: int
    dim: int
    rot_dim: int
    rot_base: float
    vdim: int
    rank: int
    scale: float
    window: int = UNBOUNDED_WINDOW


@dataclass
class GatedLinearSpec:
    """Gated linear attention: S_t = diag(alpha_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t with
    alpha = sigmoid(low-rank projection)^(1/tau); o normed per head, times silu(gate)."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int                           # of the low-rank projection


@dataclass
class RoutedSpec:
    """`top` of `experts` small feed-forwards W_down relu(W_up h)^2 per token, weighted by their softmax scores; chosen among
    the experts of the `keep` best of `groups` groups of neighbours."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1


@dataclass
class LayerSpec:
    mixer: Union[AttentionSpec, LatentAttentionSpec, GatedLinearSpec]
    ff: Union[None, int, RoutedSpec]                # width of a gated feed-forward, or experts; None = the layer has none


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row; every pass has a cache or state of its own and a vector
    that joins the residual stream ahead of it."""
    start: int
    stop: int
    times: int


@dataclass
class DecoderSpec:
    vocab: int
    width: int
    eps: float
    layers: List[LayerSpec]
    max_positions: Optional[int] = None             # None = any position
    embed_scale: float = 1.0
    loop: Optional[LoopSpec] = None

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layer runs in order: (layer, pass whose vector joins ahead of it or None)."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, None) for i in range(n)]
        inner = [(i, t if i == loop.start else None) for t in range(loop.times) for i in range(loop.start, loop.stop)]
        return [(i, None) for i in range(loop.start)] + inner + [(i, None) for i in range(loop.stop, n)]


@dataclass
class LayerTensors:
    """One layer's weights by role.  Matrices are [out, in]; what the design does not have stays None."""
    q: torch.Tensor
    o: torch.Tensor
    gate: torch.Tensor                              # output gate of the mixer
    norm1: torch.Tensor                             # on the mixer's output
    k: Optional[torch.Tensor] = None
    v: Optional[torch.Tensor] = None
    pre1: Optional[torch.Tensor] = None             # on the mixer's input
    pre2: Optional[torch.Tensor] = None             # on the feed-forward's input
    norm2: Optional[torch.Tensor] = None            # on the feed-forward's output
    # sigmoid attention
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    r1: Optional[torch.Tensor] = None
    r2: Optional[torch.Tensor] = None
    pb: Optional[torch.Tensor] = None
    shift: Optional[torch.Tensor] = None
    # latent attention
    latent: Optional[torch.Tensor] = None           # rows: latent, then the shared key part
    latent_norm: Optional[torch.Tensor] = None
    expand_k: Optional[torch.Tensor] = None
    expand_v: Optional[torch.Tensor] = None
    # gated linear attention
    low: Optional[torch.Tensor] = None
    decay: Optional[torch.Tensor] = None
    decay_bias: Optional[torch.Tensor] = None
    head_norm: Optional[torch.Tensor] = None
    # gated feed-forward
    mlp_gate: Optional[torch.Tensor] = None
    mlp_up: Optional[torch.Tensor] = None
    mlp_down: Optional[torch.Tensor] = None
    # routed feed-forward: expert -> (up, down)
    router: Optional[torch.Tensor] = None
    expert: Optional[Callable[[int], Tuple[torch.Tensor, torch.Tensor]]] = None


@dataclass
class ModelTensors:
    embed: torch.Tensor
    pos: Optional[torch.Tensor]
    final_norm: torch.Tensor
    head: Optional[torch.Tensor]                    # None = the embedding table
    layer: Callable[[int], LayerTensors]            # called once per layer, in order
    step: Optional[torch.Tensor] = None             # [passes, width]


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def distance_table(r1: torch.Tensor, r2: torch.Tensor, pb: torch.Tensor, length: int) -> torch.Tensor:
    """[heads, length]: what is added to the scaled score at each distance, pb - r1 * ln(1 + r2 * d)."""
    d = torch.arange(length, dtype=torch.float64, device=r1.device)
    r1, r2, pb = r1.double(), r2.double(), pb.double()
    return (pb[:, None] - r1[:, None] * torch.log1p(r2[:, None] * d)).float()


def rotation_table(base: float, dims: int, positions: int, device) -> torch.Tensor:
    """[positions, pad16(dims) / 2, 2]: cosine and sine of position * base^(-2i / dims), made in FP64; the padding stays as it is."""
    i = torch.arange(dims // 2, dtype=torch.float64, device=device)
    angle = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * torch.pow(base, -2.0 * i / dims)
    out = torch.zeros((positions, pad16(dims) // 2, 2), dtype=torch.float32, device=device)
    out[:, :, 0] = 1.0
    out[:, :dims // 2, 0], out[:, :dims // 2, 1] = torch.cos(angle).float(), torch.sin(angle).float()
    return out


class DenseModel:
    """Weights on the device, padded and fused for the kernels of ``include/twm_dense.h``."""

    def __init__(self, spec: DecoderSpec, tensors: ModelTensors, dtype: torch.dtype = torch.bfloat16, device="cuda"):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: the dense kernels take bfloat16 and float32")
        self.spec, self.dtype, self.device = spec, dtype, torch.device(device)
        self.runs = spec.runs()
        self.width_pad = pad16(spec.width)
        self.embed = self._rows(tensors.embed)
        self.pos = self._rows(tensors.pos) if tensors.pos is not None else None
        self.head = self._rows(tensors.head) if tensors.head is not None else self.embed
        self.final_norm = self._vector(tensors.final_norm, self.width_pad)
        self.step = [self._vector(t, self.width_pad) for t in tensors.step] if tensors.step is not None else []
        self.layers: List[Dict[str, Optional[torch.Tensor]]] = []
        for i, layer in enumerate(spec.layers):
            self.layers.append(self._layer(layer, tensors.layer(i)))

    # --------------------------------------------------------------- padding --
    def _rows(self, t: torch.Tensor, cols: Optional[int] = None) -> torch.Tensor:
        """[n, cols] with its rows zero-padded to a multiple of 16 elements."""
        n, c = t.shape
        out = torch.zeros((n, pad16(cols or c)), dtype=self.dtype, device=self.device)
        out[:, :c] = t.to(self.device, self.dtype)
        return out

    def _block(self, t: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
        """[rows, cols] with t in its corner and zeros around it."""
        out = torch.zeros((rows, cols), dtype=self.dtype, device=self.device)
        out[:t.shape[0], :t.shape[1]] = t.to(self.device, self.dtype)
        return out

    def _vector(self, t: torch.Tensor, size: int) -> torch.Tensor:
        out = torch.zeros(size, dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.to(self.device, torch.float32)
        return out

    def _head_rows(self, t: torch.Tensor, heads: int, dim: int, cols: Optional[int] = None) -> torch.Tensor:
        """[heads * dim, in] -> [heads * dim_pad, in_pad]: every head's rows padded with zero rows."""
        cols = cols or self.width_pad
        out = torch.zeros((heads, pad16(dim), cols), dtype=self.dtype, device=self.device)
        out[:, :dim, :t.shape[1]] = t.to(self.device, self.dtype).reshape(heads, dim, -1)
        return out.reshape(heads * pad16(dim), cols)

    def _head_vector(self, t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
        out = torch.zeros((heads, pad16(dim)), dtype=torch.float32, device=self.device)
        out[:, :dim] = t.to(self.device, torch.float32).reshape(heads, dim)
        return out.reshape(-1)

    def _layer(self, spec: LayerSpec, t: LayerTensors) -> Dict[str, Optional[torch.Tensor]]:
        m, w = spec.mixer, {}
        {AttentionSpec: self._sigmoid, LatentAttentionSpec: self._latent, GatedLinearSpec: self._linear}[type(m)](m, t, w)
        out = torch.zeros((self.spec.width, m.heads, pad16(m.vdim)), dtype=self.dtype, device=self.device)
        out[:, :, :m.vdim] = t.o.to(self.device, self.dtype).reshape(self.spec.width, m.heads, m.vdim)
        w["w_out"] = out.reshape(self.spec.width, -1)
        for name in ("norm1", "norm2", "pre1", "pre2"):
            v = getattr(t, name)
            w[name] = self._vector(v, self.width_pad) if v is not None else None
        if isinstance(spec.ff, RoutedSpec):
            self._routed(spec.ff, t, w)
        elif spec.ff is not None:
            ff, fp = spec.ff, pad16(spec.ff)
            w["w_gate_up"] = torch.cat([self._block(t.mlp_gate, fp, self.width_pad), self._block(t.mlp_up, fp, self.width_pad)])
            w["w_down"] = self._rows(t.mlp_down, ff)
        return w

    def _sigmoid(self, m: AttentionSpec, t: LayerTensors, w: dict) -> None:
        w["w_in"] = torch.cat([self._head_rows(t.q, m.heads, m.dim), self._head_rows(t.k, m.kv_heads, m.dim),
                               self._head_rows(t.v, m.kv_heads, m.vdim), self._head_rows(t.gate, m.heads, m.vdim)])
        w["q_norm"] = self._head_vector(t.q_norm, m.heads, m.dim)
        w["k_norm"] = self._head_vector(t.k_norm, m.kv_heads, m.dim)
        w["bias_table"] = distance_table(t.r1.to(self.device), t.r2.to(self.device), t.pb.to(self.device), self.spec.max_positions)
        w["shift"] = self._vector(t.shift, self.width_pad) if t.shift is not None else None

    def _latent(self, m: LatentAttentionSpec, t: LayerTensors, w: dict) -> None:
        dp, rp, kp, wp = pad16(m.dim), pad16(m.rot_dim), pad16(m.rank), self.width_pad
        q = torch.zeros((m.heads, dp + rp, wp), dtype=self.dtype, device=self.device)
        src = t.q.to(self.device, self.dtype).reshape(m.heads, m.dim + m.rot_dim, -1)
        q[:, :m.dim, :src.shape[2]] = src[:, :m.dim]
        q[:, dp:dp + m.rot_dim, :src.shape[2]] = src[:, m.dim:]
        w["w_in"] = torch.cat([q.reshape(-1, wp), self._block(t.latent[:m.rank], kp, wp), self._block(t.latent[m.rank:], rp, wp),
                               self._block(t.gate, pad16(m.heads), wp)])
        w["w_expand"] = torch.cat([self._head_rows(t.expand_k, m.heads, m.dim, kp), self._head_rows(t.expand_v, m.heads, m.vdim, kp)])
        w["latent_norm"] = self._vector(t.latent_norm, kp)

    def _linear(self, m: GatedLinearSpec, t: LayerTensors, w: dict) -> None:
        rp, wp = pad16(m.rank), self.width_pad
        w["w_in"] = torch.cat([self._head_rows(t.q, m.heads, m.dim), self._head_rows(t.k, m.heads, m.dim),
                               self._head_rows(t.v, m.heads, m.vdim), self._head_rows(t.gate, m.heads, m.vdim), self._block(t.low, rp, wp)])
        w["w_decay"] = self._head_rows(t.decay, m.heads, m.dim, rp)
        w["decay_bias"] = self._head_vector(t.decay_bias, m.heads, m.dim)
        w["head_norm"] = self._vector(t.head_norm, pad16(m.vdim))

    def _routed(self, ff: RoutedSpec, t: LayerTensors, w: dict) -> None:
        fp, wp = pad16(ff.ff), self.width_pad
        w["w_router"] = self._rows(t.router)
        w["w_gate_up"] = torch.zeros((ff.experts, fp, wp), dtype=self.dtype, device=self.device)
        w["w_down"] = torch.zeros((ff.experts, self.spec.width, fp), dtype=self.dtype, device=self.device)
        for e in range(ff.experts):
            up, down = t.expert(e)
            w["w_gate_up"][e, :ff.ff, :self.spec.width] = up.to(self.device, self.dtype)
            w["w_down"][e, :, :ff.ff] = down.to(self.device, self.dtype)

    # ------------------------------------------------------------ description --
    def descriptor(self, state) -> _dense.Model:
        """The C view of this model over `state` (state.SequenceState).  Keeps what it points to alive."""
        n = len(self.runs)
        array, tables = (_dense.Layer * max(n, 1))(), {}
        for run, (i, joined) in enumerate(self.runs):
            spec, w, lay = self.spec.layers[i], self.layers[i], array[run]
            m, ff = spec.mixer, spec.ff
            lay.heads, lay.dim, lay.vdim, lay.dim_pad, lay.vdim_pad = m.heads, m.dim, m.vdim, pad16(m.dim), pad16(m.vdim)
            if isinstance(m, AttentionSpec):
                lay.mixer, lay.kv_heads, lay.scale = _dense.MIX_SIGMOID, m.kv_heads, m.scale
                lay.window, lay.keep_first = min(m.window, UNBOUNDED_WINDOW), m.keep_first
            elif isinstance(m, LatentAttentionSpec):
                lay.mixer, lay.scale, lay.window = _dense.MIX_LATENT, m.scale, min(m.window, UNBOUNDED_WINDOW)
                lay.rank, lay.rank_pad, lay.rot_pad = m.rank, pad16(m.rank), pad16(m.rot_dim)
                key = (m.rot_base, m.rot_dim)
                if key not in tables:
                    tables[key] = rotation_table(m.rot_base, m.rot_dim, state.capacity, self.device)
                lay.rot_table = tables[key].data_ptr()
            else:
                lay.mixer, lay.scale, lay.inv_tau = _dense.MIX_GLA, m.dim ** -0.5, 1.0 / m.tau
                lay.rank, lay.rank_pad = m.rank, pad16(m.rank)
            lay.ff_pad = 0 if ff is None else pad16(ff.ff if isinstance(ff, RoutedSpec) else ff)
            if isinstance(ff, RoutedSpec):
                lay.experts, lay.top, lay.groups, lay.keep = ff.experts, ff.top, ff.groups, ff.keep
            for name in ("w_in", "w_out", "w_gate_up", "w_down", "q_norm", "k_norm", "bias_table", "shift", "norm1", "norm2", "pre1", "pre2",
                         "w_expand", "latent_norm", "w_decay", "decay_bias", "head_norm", "w_router"):
                t = w.get(name)
                setattr(lay, name, t.data_ptr() if t is not None else None)
            lay.step = self.step[joined].data_ptr() if joined is not None else None
            for name, t in state.runs[run].items():
                setattr(lay, name, t.data_ptr())
        d = _dense.Model()
        d.dtype = _dense.TWM_DENSE_F32 if self.dtype == torch.float32 else _dense.TWM_DENSE_BF16
        d.width, d.width_pad, d.vocab, d.n_layers = self.spec.width, self.width_pad, self.spec.vocab, n
        d.bias_len, d.capacity, d.slots, d.eps = self.spec.max_positions or 0, state.capacity, state.slots, self.spec.eps
        d.embed_scale = self.spec.embed_scale
        d.embed, d.head, d.final_norm = self.embed.data_ptr(), self.head.data_ptr(), self.final_norm.data_ptr()
        d.pos_embed = self.pos.data_ptr() if self.pos is not None else None
        d.layers = array
        d._keep = (array, state, tables)
        return d
