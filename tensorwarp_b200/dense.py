"""Decoder models with dense 16-bit or 32-bit weights: what a model is made of, and its weights on the device.

A model file in ``models/`` describes its design as a ``DecoderSpec``, whose mechanisms are
parameters (a None leaves one out), and names its tensors; everything else (padding, fusion, the cache,
the step) is shared.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Callable, Dict, List, Optional

import torch

from . import _dense

UNBOUNDED_WINDOW = 1 << 30


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
class LayerSpec:
    mixer: AttentionSpec
    ff: Optional[int]                   # width of the gated feed-forward, None = the layer has none


@dataclass
class DecoderSpec:
    vocab: int
    width: int
    eps: float
    max_positions: int
    layers: List[LayerSpec]


@dataclass
class LayerTensors:
    """One layer's weights by role.  Matrices are [out, in]."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    gate: torch.Tensor                  # output gate of the mixer
    o: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    r1: torch.Tensor
    r2: torch.Tensor
    pb: torch.Tensor
    shift: Optional[torch.Tensor]
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor]
    mlp_gate: Optional[torch.Tensor]
    mlp_up: Optional[torch.Tensor]
    mlp_down: Optional[torch.Tensor]


@dataclass
class ModelTensors:
    embed: torch.Tensor
    pos: Optional[torch.Tensor]
    final_norm: torch.Tensor
    head: torch.Tensor
    layer: Callable[[int], LayerTensors]        # called once per layer, in order


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def distance_table(r1: torch.Tensor, r2: torch.Tensor, pb: torch.Tensor, length: int) -> torch.Tensor:
    """[heads, length]: what is added to the scaled score at each distance, pb - r1 * ln(1 + r2 * d)."""
    d = torch.arange(length, dtype=torch.float64, device=r1.device)
    r1, r2, pb = r1.double(), r2.double(), pb.double()
    return (pb[:, None] - r1[:, None] * torch.log1p(r2[:, None] * d)).float()


class DenseModel:
    """Weights on the device, padded and fused for the kernels of ``include/twm_dense.h``."""

    def __init__(self, spec: DecoderSpec, tensors: ModelTensors, dtype: torch.dtype = torch.bfloat16, device="cuda"):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: the dense kernels take bfloat16 and float32")
        self.spec, self.dtype, self.device = spec, dtype, torch.device(device)
        self.width_pad = pad16(spec.width)
        self.embed = self._rows(tensors.embed)
        self.pos = self._rows(tensors.pos) if tensors.pos is not None else None
        self.head = self._rows(tensors.head)
        self.final_norm = self._vector(tensors.final_norm, self.width_pad)
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

    def _vector(self, t: torch.Tensor, size: int) -> torch.Tensor:
        out = torch.zeros(size, dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.to(self.device, torch.float32)
        return out

    def _head_rows(self, t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
        """[heads * dim, in] -> [heads * dim_pad, in_pad]: every head's rows padded with zero rows."""
        out = torch.zeros((heads, pad16(dim), self.width_pad), dtype=self.dtype, device=self.device)
        out[:, :dim, :t.shape[1]] = t.to(self.device, self.dtype).reshape(heads, dim, -1)
        return out.reshape(heads * pad16(dim), self.width_pad)

    def _head_vector(self, t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
        out = torch.zeros((heads, pad16(dim)), dtype=torch.float32, device=self.device)
        out[:, :dim] = t.to(self.device, torch.float32).reshape(heads, dim)
        return out.reshape(-1)

    def _layer(self, spec: LayerSpec, t: LayerTensors) -> Dict[str, Optional[torch.Tensor]]:
        m, w = spec.mixer, {}
        w["w_in"] = torch.cat([self._head_rows(t.q, m.heads, m.dim), self._head_rows(t.k, m.kv_heads, m.dim),
                               self._head_rows(t.v, m.kv_heads, m.vdim), self._head_rows(t.gate, m.heads, m.vdim)])
        out = torch.zeros((self.spec.width, m.heads, pad16(m.vdim)), dtype=self.dtype, device=self.device)
        out[:, :, :m.vdim] = t.o.to(self.device, self.dtype).reshape(self.spec.width, m.heads, m.vdim)
        w["w_out"] = out.reshape(self.spec.width, -1)
        w["q_norm"] = self._head_vector(t.q_norm, m.heads, m.dim)
        w["k_norm"] = self._head_vector(t.k_norm, m.kv_heads, m.dim)
        w["bias_table"] = distance_table(t.r1.to(self.device), t.r2.to(self.device), t.pb.to(self.device), self.spec.max_positions)
        w["shift"] = self._vector(t.shift, self.width_pad) if t.shift is not None else None
        w["norm1"] = self._vector(t.norm1, self.width_pad)
        if spec.ff is not None:
            fp = pad16(spec.ff)
            gu = torch.zeros((2, fp, self.width_pad), dtype=self.dtype, device=self.device)
            gu[0, :spec.ff, :self.spec.width] = t.mlp_gate.to(self.device, self.dtype)
            gu[1, :spec.ff, :self.spec.width] = t.mlp_up.to(self.device, self.dtype)
            w["w_gate_up"] = gu.reshape(2 * fp, self.width_pad)
            w["w_down"] = self._rows(t.mlp_down)
            w["norm2"] = self._vector(t.norm2, self.width_pad)
        return w

    # ------------------------------------------------------------ description --
    def descriptor(self, state) -> _dense.Model:
        """The C view of this model over `state` (state.SequenceState).  Keeps what it points to alive."""
        n = len(self.spec.layers)
        array = (_dense.Layer * max(n, 1))()
        for i, (spec, w) in enumerate(zip(self.spec.layers, self.layers)):
            m, lay = spec.mixer, array[i]
            lay.heads, lay.kv_heads, lay.dim, lay.vdim = m.heads, m.kv_heads, m.dim, m.vdim
            lay.dim_pad, lay.vdim_pad = pad16(m.dim), pad16(m.vdim)
            lay.window, lay.keep_first, lay.scale = min(m.window, UNBOUNDED_WINDOW), m.keep_first, m.scale
            lay.ff_pad = pad16(spec.ff) if spec.ff is not None else 0
            for name in ("w_in", "w_out", "w_gate_up", "w_down", "q_norm", "k_norm", "bias_table", "shift", "norm1", "norm2"):
                t = w.get(name)
                setattr(lay, name, t.data_ptr() if t is not None else None)
            lay.k_cache, lay.v_cache = state.k[i].data_ptr(), state.v[i].data_ptr()
            lay.shift_state = state.shift[i].data_ptr() if state.shift[i] is not None else None
        d = _dense.Model()
        d.dtype = _dense.TWM_DENSE_F32 if self.dtype == torch.float32 else _dense.TWM_DENSE_BF16
        d.width, d.width_pad, d.vocab, d.n_layers = self.spec.width, self.width_pad, self.spec.vocab, n
        d.bias_len, d.capacity, d.slots, d.eps = self.spec.max_positions, state.capacity, state.slots, self.spec.eps
        d.embed, d.head, d.final_norm = self.embed.data_ptr(), self.head.data_ptr(), self.final_norm.data_ptr()
        d.pos_embed = self.pos.data_ptr() if self.pos is not None else None
        d.layers = array
        d._keep = (array, state)
        return d
