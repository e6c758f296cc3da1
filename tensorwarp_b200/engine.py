"""The step interface every served model has, and the engine of the dense-weight decoders.

An engine keeps the state of several sequences and runs one sequence's step at a time: a portion of
its prompt of any size, or one decoded token.  Prompt portions are enqueued by one native call; a
decoded token replays a captured CUDA graph whose position, slot and token live in device memory,
so one graph serves every sequence.  Sampling stays on the device (greedy).
"""
from __future__ import annotations

import ctypes as C
from typing import Dict, List, Optional, Protocol, Sequence

import torch

from . import _dense
from ._dense import check
from .state import SequenceState


class StepEngine(Protocol):
    vocab: int
    capacity: int                   # tokens per sequence
    max_live: int                   # sequences whose state can be held at once

    def open(self) -> int: ...
    def close(self, seq: int) -> None: ...
    def length(self, seq: int) -> int: ...
    def step(self, seq: int, tokens: Sequence[int], want: Sequence[int] = ()) -> Optional[torch.Tensor]:
        """Run the sequence's next tokens; returns the logits f32 [len(want), vocab] at the wanted places among
        them (valid until the next call), None when nothing is wanted."""
        ...
    def greedy(self, seq: int, tokens: Sequence[int], count: int) -> List[int]:
        """Run the sequence's next tokens, then generate `count` tokens; the last one is not yet run."""
        ...


class DenseEngine:
    LOGITS_BYTES = 256 << 20
    DEFAULT_CAPACITY = 16384            # tokens per sequence of a model without a position limit

    def __init__(self, model, max_tokens: Optional[int] = None, max_live: int = 4, portion: int = 4096, use_pdl: bool = True,
                 use_graphs: bool = True):
        """max_tokens: longest sequence served (a model without a position limit takes any); portion: most tokens of a prompt
        per native call."""
        self.model, self.spec, self.device = model, model.spec, model.device
        self.vocab = self.spec.vocab
        limit = self.spec.max_positions
        capacity = min(limit, max_tokens or limit) if limit is not None else max_tokens or self.DEFAULT_CAPACITY
        self.state = SequenceState(model, max_live, capacity)
        self.capacity, self.max_live = capacity, max_live
        self.flags = _dense.TWM_FLAG_PDL if use_pdl else 0
        self.use_graphs = use_graphs
        self.stream = torch.cuda.Stream(self.device)
        self._desc = model.descriptor(self.state)
        self._allocate(min(capacity, portion))
        self._graphs: Dict[str, torch.cuda.CUDAGraph] = {}
        self.launches_per_step = 0
        torch.cuda.synchronize(self.device)         # weights and state were written on the default stream

    # ---------------------------------------------------------------- buffers --
    def _allocate(self, rows: int) -> None:
        dev, dt, wp = self.device, self.model.dtype, self.model.width_pad
        lays = [self._desc.layers[i] for i in range(self._desc.n_layers)]
        w_in = max([w["w_in"].shape[0] for w in self.model.layers], default=16)
        w_att = max([x.heads * x.vdim_pad for x in lays], default=16)
        w_ff = max([x.ff_pad for x in lays] + [16])
        slots_per_row = max([x.top if x.experts else 1 for x in lays] + [1])
        w_act = max([x.ff_pad * (x.top if x.experts else 1) for x in lays] + [16])
        experts = max([x.experts for x in lays] + [0])
        self.max_rows = rows
        self.max_want = max(1, min(rows, self.LOGITS_BYTES // (4 * self.vocab)))

        def zeros(*shape, dtype):
            return torch.zeros(shape, dtype=dtype, device=dev)

        f32, i32 = torch.float32, torch.int32
        self._buf = dict(meta=zeros(8, dtype=i32), tokens=zeros(rows, dtype=i32), want=zeros(self.max_want, dtype=i32),
                         x0=zeros(rows, wp, dtype=f32), x1=zeros(rows, wp, dtype=f32), y=zeros(rows, wp, dtype=f32),
                         a=zeros(rows, wp, dtype=dt), proj=zeros(rows, w_in, dtype=dt), att=zeros(rows, w_att, dtype=dt),
                         act=zeros(rows * slots_per_row, w_ff, dtype=dt), vec=zeros(w_in + w_att + w_act + wp, dtype=f32),
                         logits=zeros(self.max_want, self.vocab, dtype=f32))
        b = _dense.Buffers(max_rows=rows, max_want=self.max_want)
        latent = [x for x in lays if x.mixer == _dense.MIX_LATENT]
        if latent:
            b.max_keys = min(self.capacity, rows + max(x.window for x in latent) - 1)
            self._buf.update(lat=zeros(b.max_keys, max(x.rank_pad + x.rot_pad for x in latent), dtype=dt),
                             kv=zeros(b.max_keys, max(x.heads * (x.dim_pad + x.vdim_pad) for x in latent), dtype=dt))
        linear = [x for x in lays if x.mixer == _dense.MIX_GLA]
        if linear:
            self._buf.update(decay=zeros(rows, max(x.heads * x.dim_pad for x in linear), dtype=f32),
                             chunk_state=zeros((rows + 63) // 64, max(x.heads * x.dim_pad * x.vdim_pad for x in linear), dtype=f32),
                             mix=zeros(rows, max(x.heads * x.vdim_pad for x in linear), dtype=f32))
        if experts:
            b.max_slots = rows * slots_per_row
            self._buf.update(router_logits=zeros(rows, experts, dtype=f32), route=zeros(3 * b.max_slots + 2 * experts + 1, dtype=i32),
                             route_weight=zeros(b.max_slots, dtype=f32), grouped=zeros(b.max_slots, wp, dtype=dt),
                             expert_out=zeros(b.max_slots, wp, dtype=dt))
        for name, t in self._buf.items():
            setattr(b, name, t.data_ptr())
        self._b = b
        self.history = zeros(max(self.capacity, 1), dtype=i32)
        self._argmax_scratch = zeros(_dense.lib().twm_dense_argmax_scratch_bytes(), dtype=torch.uint8)

    @property
    def logits(self) -> torch.Tensor:
        return self._buf["logits"]

    # --------------------------------------------------------------- sequences --
    def open(self) -> int:
        return self.state.open()

    def close(self, seq: int) -> None:
        self.state.close(seq)

    def length(self, seq: int) -> int:
        return self.state.length(seq)

    def _check_tokens(self, tokens: Sequence[int]) -> None:
        if not tokens:
            raise ValueError("a step brings at least one token")
        if min(tokens) < 0 or max(tokens) >= self.vocab:
            raise ValueError(f"token outside the vocabulary of {self.vocab}")

    # ------------------------------------------------------------------- steps --
    def step(self, seq: int, tokens: Sequence[int], want: Sequence[int] = (), layer_trace: Optional[List[torch.Tensor]] = None):
        """See StepEngine.  layer_trace: a list that receives, per native call, the residual stream after every layer run,
        f32 [layer runs, tokens, width]."""
        tokens, want = list(tokens), list(want)
        self._check_tokens(tokens)
        if any(b <= a for a, b in zip(want, want[1:])) or (want and not 0 <= want[0] <= want[-1] < len(tokens)):
            raise ValueError("wanted places must be increasing and among the step's tokens")
        first = self.state.length(seq)
        self.state.advance(seq, len(tokens))
        if len(tokens) == 1 and layer_trace is None:
            self._set_step(first, seq, tokens[0])
            self._decode("logits" if want else "silent")
            return self._sync(self.logits[:1] if want else None)
        outs, at, w = [], 0, 0
        while at < len(tokens):
            # as many tokens as the buffers take, and no more wanted rows than they take
            end = min(len(tokens), at + self.max_rows)
            if w + self.max_want < len(want):
                end = min(end, want[w + self.max_want])
            here = [p - at for p in want[w:] if p < end]
            trace = self._prefill(seq, first + at, tokens[at:end], here, layer_trace is not None)
            with torch.cuda.stream(self.stream):
                if layer_trace is not None:
                    layer_trace.append(trace[:, :, :self.spec.width].clone())
                if here:
                    rows = self.logits[:len(here)]
                    outs.append(rows if end == len(tokens) else rows.clone())
            w += len(here)
            at = end
        with torch.cuda.stream(self.stream):
            out = (outs[0] if len(outs) == 1 else torch.cat(outs)) if outs else None
        return self._sync(out)

    def _sync(self, out: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        self.stream.synchronize()
        return out

    def _set_step(self, first: int, slot: int, token: int = -1) -> None:
        check(_dense.lib().twm_dense_set_step(C.byref(self._b), first, slot, token, self.stream.cuda_stream), "twm_dense_set_step")

    def _prefill(self, slot: int, first: int, tokens: List[int], want: List[int], trace: bool) -> Optional[torch.Tensor]:
        out = None
        with torch.cuda.stream(self.stream):
            self._buf["tokens"][:len(tokens)].copy_(torch.tensor(tokens, dtype=torch.int32))
            if want:
                self._buf["want"][:len(want)].copy_(torch.tensor(want, dtype=torch.int32))
            self._set_step(first, slot)
            if trace:
                out = torch.empty((len(self.model.runs), len(tokens), self.model.width_pad), dtype=torch.float32, device=self.device)
            self.enqueue_prefill(len(tokens), first, len(want), out)
        return out

    def enqueue_prefill(self, rows: int, first: int, n_want: int, trace: Optional[torch.Tensor] = None) -> None:
        """Enqueue one native prefill call on the engine's stream; tokens, wanted rows and meta are already on the device."""
        check(_dense.lib().twm_dense_prefill(C.byref(self._desc), C.byref(self._b), rows, first, n_want,
                                             trace.data_ptr() if trace is not None else None, self.flags,
                                             self.stream.cuda_stream), "twm_dense_prefill")
        self.launches_per_step = _dense.lib().twm_dense_launches()

    # ------------------------------------------------------------------ decode --
    def _enqueue_decode(self, kind: str) -> None:
        """One decoded token on the engine's stream.  kind: "silent" (state only), "logits", "greedy" (logits, arg-max,
        and position and token advanced on the device)."""
        lib, s = _dense.lib(), self.stream.cuda_stream
        check(lib.twm_dense_decode(C.byref(self._desc), C.byref(self._b), 0 if kind == "silent" else 1, self.flags, s),
              "twm_dense_decode")
        self.launches_per_step = lib.twm_dense_launches()
        if kind == "greedy":
            self._argmax()
            self.launches_per_step = lib.twm_dense_launches()

    def _argmax(self) -> None:
        check(_dense.lib().twm_dense_argmax_advance(C.byref(self._b), self.vocab, 0, self.history.data_ptr(), self.history.numel(),
                                                    self._argmax_scratch.data_ptr(), self._argmax_scratch.numel(), self.flags,
                                                    self.stream.cuda_stream), "twm_dense_argmax_advance")

    def capture_decode(self, kind: str) -> torch.cuda.CUDAGraph:
        graph = self._graphs.get(kind)
        if graph is None:
            graph = torch.cuda.CUDAGraph()
            self.stream.synchronize()
            with torch.cuda.graph(graph, stream=self.stream):       # recorded only: nothing of the state changes
                self._enqueue_decode(kind)
            self._graphs[kind] = graph
        return graph

    def _decode(self, kind: str) -> None:
        with torch.cuda.stream(self.stream):
            if self.use_graphs:
                self.capture_decode(kind).replay()
            else:
                self._enqueue_decode(kind)

    def greedy(self, seq: int, tokens: Sequence[int], count: int) -> List[int]:
        if count < 1:
            return []
        tokens = list(tokens)
        self._check_tokens(tokens)
        first = self.state.length(seq)
        if first + len(tokens) + count - 1 > self.capacity:
            raise ValueError(f"{first} + {len(tokens)} tokens and {count} new ones run past the slot's {self.capacity}")
        replays = count
        with torch.cuda.stream(self.stream):
            self._buf["meta"][3:4].zero_()                          # the step counter indexes the history
            if len(tokens) > 1:
                self.step(seq, tokens, [len(tokens) - 1])
                self._set_step(first + len(tokens) - 1, seq)        # the arg-max advances the position by one
                self._argmax()
                replays -= 1
            else:
                self._set_step(first, seq, tokens[0])
        for _ in range(replays):
            self._decode("greedy")
        if len(tokens) > 1:
            self.state.advance(seq, replays)
        else:
            self.state.advance(seq, count)
        self.stream.synchronize()
        return self.history[:count].tolist()
