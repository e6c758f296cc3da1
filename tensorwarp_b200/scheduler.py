"""Serves requests on a step engine: first come, first served admission into the engine's free sequences,
prompts in portions, live sequences in turn.

Each turn runs one sequence: the next portion of its prompt, or a burst of greedily decoded tokens
(one host synchronisation a burst).  A sequence's slot goes back to the engine when it has finished.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Deque, Iterator, List, Optional, Sequence


@dataclass
class Request:
    tokens: List[int]
    max_new_tokens: int
    stop_token: Optional[int] = None
    generated: List[int] = field(default_factory=list)
    done: bool = False


@dataclass
class _Live:
    request: Request
    seq: int
    pending: List[int]              # tokens that are not yet run


class Scheduler:
    def __init__(self, engine, portion: int = 2048, burst: int = 16):
        if portion < 1 or burst < 1:
            raise ValueError("portion and burst must be positive")
        self.engine, self.portion, self.burst = engine, portion, burst
        self._waiting: Deque[Request] = deque()
        self._live: Deque[_Live] = deque()

    def submit(self, tokens: Sequence[int], max_new_tokens: int, stop_token: Optional[int] = None) -> Request:
        tokens = list(tokens)
        if not tokens or max_new_tokens < 1:
            raise ValueError("a request has at least one token and asks for at least one")
        if len(tokens) + max_new_tokens - 1 > self.engine.capacity:
            raise ValueError(f"{len(tokens)} tokens and {max_new_tokens} new ones do not fit the {self.engine.capacity} of a sequence")
        if min(tokens) < 0 or max(tokens) >= self.engine.vocab:
            raise ValueError(f"token outside the vocabulary of {self.engine.vocab}")
        request = Request(tokens, max_new_tokens, stop_token)
        self._waiting.append(request)
        return request

    def _admit(self) -> None:
        while self._waiting and len(self._live) < self.engine.max_live:
            request = self._waiting.popleft()
            self._live.append(_Live(request, self.engine.open(), list(request.tokens)))

    def turn(self) -> Optional[Request]:
        """Run one sequence once; returns the request if it has finished with this turn."""
        self._admit()
        if not self._live:
            return None
        live = self._live.popleft()
        request = live.request
        try:
            if len(live.pending) > self.portion:
                self.engine.step(live.seq, live.pending[:self.portion])
                del live.pending[:self.portion]
            else:
                count = min(self.burst, request.max_new_tokens - len(request.generated))
                new = self.engine.greedy(live.seq, live.pending, count)
                if request.stop_token is not None and request.stop_token in new:
                    new = new[:new.index(request.stop_token) + 1]
                    request.done = True
                request.generated += new
                live.pending = request.generated[-1:]
                request.done = request.done or len(request.generated) >= request.max_new_tokens
        except BaseException:
            self.engine.close(live.seq)
            raise
        if request.done:
            self.engine.close(live.seq)
            return request
        self._live.append(live)
        return None

    def run(self) -> Iterator[Request]:
        """Turns until nothing is left, yielding requests as they finish."""
        while self._waiting or self._live:
            request = self.turn()
            if request is not None:
                yield request
