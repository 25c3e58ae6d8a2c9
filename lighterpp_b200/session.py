"""Host-side bookkeeping of the sequence an engine is working on.

The engine computes one sequence at a time: its cache holds the positions 0 .. of that sequence.  A ``Session`` keeps
track of whose sequence that is and how far it has come, cuts work into ``Engine.extend`` / ``Engine.decode`` calls and
gives the cache back when a sequence ends.  Nothing of a finished sequence is read again: attention looks at positions up
to the current one only, and those are rewritten from 0 on.
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import numpy as np

from .engine import Engine


class Session:
    def __init__(self, engine: Engine):
        self.engine = engine
        self.owner: Optional[str] = None
        self.length = 0

    @property
    def capacity(self) -> int:
        return self.engine.cfg.seq_len

    def extend(self, owner: str, tokens: Sequence[int], want: Sequence[int] = ()) -> np.ndarray:
        """The next ``tokens`` of ``owner``'s sequence (a new owner starts at position 0; the previous one must have
        ended); logits of the places ``want`` among them, in the order asked for."""
        if self.owner is None:
            self.owner, self.length = owner, 0
        if owner != self.owner:
            raise RuntimeError(f"sequence {self.owner!r} has not ended: the engine works on one sequence at a time")
        if self.length + len(tokens) > self.capacity:
            raise ValueError(f"{self.length + len(tokens)} positions exceed the cache's {self.capacity}")
        places = sorted(set(int(w) for w in want))
        logits = self.engine.extend(tokens, self.length, places) if len(tokens) else np.empty((0, self.engine.cfg.vocab_size), np.float32)
        self.length += len(tokens)
        return logits[[places.index(int(w)) for w in want]]

    def end(self, owner: str) -> None:
        if owner == self.owner:
            self.owner, self.length = None, 0

    def generate(self, prompt: Sequence[int], n: int, temperature: float = 0.0, penalty: float = 1.0, seed: int = 0,
                 history_window: int = 64) -> List[int]:
        """Samples ``n`` tokens after ``prompt``: the prompt's tokens but the last through the batched path, then the
        device-resident loop of src/main.cpp:163-223."""
        if not len(prompt) or n <= 0:
            raise ValueError("need a prompt and at least one token to sample")
        if len(prompt) - 1 + n > self.capacity:
            raise ValueError(f"{len(prompt) - 1 + n} positions exceed the cache's {self.capacity}")
        me = "generate"
        self.extend(me, list(prompt[:-1]))
        try:
            r = np.random.default_rng(seed).random(n).astype(np.float32)
            out, _ = self.engine.decode(int(prompt[-1]), self.length, n, temperature, penalty, [int(t) for t in prompt][-history_window:],
                                        history_window, r)
        finally:
            self.end(me)
        return [int(t) for t in out]
