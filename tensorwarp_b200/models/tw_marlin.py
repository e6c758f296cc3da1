"""The 4-bit TW-Marlin decoder behind the step interface.

Its engine (``generate.QuantizedGenerationEngine``) has one cache and decodes one token at a time, so a
prompt is run token by token and one sequence is live.  There is no checkpoint format for it here:
weights are seeded synthetic ones of the configured shape.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch

from ..checkpoint import CheckpointError
from ..generate import Q4Model, QuantizedGenerationEngine, TransformerConfig
from ..registry import register
from ..state import StateError


def parse_config(config: dict) -> TransformerConfig:
    fields = {k: v for k, v in config.items() if k not in ("architecture", "seed")}
    try:
        return TransformerConfig(**fields)
    except TypeError as e:
        raise CheckpointError(f"TWMarlinQ4: {e}") from None


class Q4StepEngine:
    max_live = 1

    def __init__(self, engine: QuantizedGenerationEngine):
        self.engine = engine
        self.vocab, self.capacity = engine.cfg.vocab, engine.cfg.max_seq
        self._length: Optional[int] = None

    def open(self) -> int:
        if self._length is not None:
            raise StateError("the engine's one sequence is taken")
        self._length = 0
        return 0

    def close(self, seq: int) -> None:
        self.length(seq)
        self._length = None

    def length(self, seq: int) -> int:
        if seq != 0 or self._length is None:
            raise StateError(f"sequence {seq} is not open")
        return self._length

    def _run(self, token: int) -> None:
        eng = self.engine
        eng.reset_history()
        eng.set_token(token)
        eng.set_position(self._length)          # synchronises
        eng.step_eager()
        torch.cuda.synchronize(eng.model.device)
        self._length += 1

    def _reserve(self, seq: int, tokens: Sequence[int], new: int) -> None:
        if not tokens or min(tokens) < 0 or max(tokens) >= self.vocab:
            raise ValueError("a step brings at least one token of the vocabulary")
        if self.length(seq) + len(tokens) + new > self.capacity:
            raise StateError(f"sequence runs past the cache of {self.capacity} tokens")

    def step(self, seq: int, tokens: Sequence[int], want: Sequence[int] = ()) -> Optional[torch.Tensor]:
        self._reserve(seq, tokens, 0)
        rows, wanted = [], set(want)
        for i, token in enumerate(tokens):
            self._run(token)
            if i in wanted:
                rows.append(self.engine.buf.logits.clone())
        return torch.stack(rows) if rows else None

    def greedy(self, seq: int, tokens: Sequence[int], count: int) -> List[int]:
        self._reserve(seq, tokens, max(count - 1, 0))
        if count < 1:
            return []
        for token in tokens[:-1]:
            self._run(token)
        self.engine.reset_history()
        self.engine.set_position(self._length)
        out = self.engine.generate_tw_marlin_graph(tokens[-1], count)
        self._length += count
        return out


@register("TWMarlinQ4")
def build(config: dict, weights, dtype: torch.dtype = torch.bfloat16, device="cuda", max_tokens: Optional[int] = None,
          **_) -> Q4StepEngine:
    if weights is not None:
        raise CheckpointError("TWMarlinQ4 has no checkpoint format here; remove model.safetensors to run synthetic weights")
    if dtype == torch.float32:
        raise CheckpointError("the 4-bit engine serves 16-bit activations only")
    cfg = parse_config(config)
    if max_tokens:
        cfg.max_seq = min(cfg.max_seq, max_tokens)
    return Q4StepEngine(QuantizedGenerationEngine(Q4Model(cfg, device, seed=int(config.get("seed", 0)))))
