"""Batching over one InferenceModel with a paged cache (fp32-stream plans).

`SequenceSlots` names sequences: a request gets a slot of the state at its first tokens and gives slot and pages back at its
end. `BatchScheduler` generates: every step it puts the next token of each running request and portions of waiting prompts
into one batch (InferenceModel.run_batch), up to a budget of rows.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Callable, Deque, Dict, Hashable, List, Optional, Sequence

import numpy as np

from .plan import PAGE_TOKENS


class SequenceSlots:
    def __init__(self, model):
        self.model = model
        self.free: List[int] = list(range(model.batch - 1, -1, -1))   # slot 0 is handed out first
        self.slot: Dict[Hashable, int] = {}

    def of(self, name: Hashable) -> int:
        """The slot of a sequence, taken now if it has none."""
        if name not in self.slot:
            if not self.free:
                raise RuntimeError(f"no free sequence slot for {name!r}: {len(self.slot)} are live")
            self.slot[name] = self.free.pop()
        return self.slot[name]

    def release(self, name: Hashable) -> None:
        slot = self.slot.pop(name, None)
        if slot is not None:
            self.model.reset_sequence(slot)
            self.free.append(slot)

    def run(self, entries, logits: bool = True):
        """[(name, tokens, wanted places), ...] as one batch."""
        return self.model.run_batch([(self.of(name), tokens, want) for name, tokens, want in entries], logits=logits)


@dataclass
class Request:
    name: Hashable
    prompt: Sequence[int]
    max_new_tokens: int
    stop_tokens: Sequence[int] = ()
    generated: List[int] = field(default_factory=list)
    done: bool = False
    _fed: int = 0      # prompt tokens already in the cache


class BatchScheduler:
    """Continuous batching. `sampler` maps a row of logits (fp32) to a token; None = greedy, decided on the device.

    A request is admitted when a slot is free and the pool can hold its prompt and everything it may generate on top of what
    the admitted requests may still need, so a running request never waits for pages."""

    def __init__(self, model, row_budget: int = 2048, sampler: Optional[Callable[[np.ndarray], int]] = None):
        if row_budget < model.batch:
            raise ValueError("the row budget must have room for one token of every sequence")
        self.model, self.slots = model, SequenceSlots(model)
        self.row_budget, self.sampler = row_budget, sampler
        self.pool_pages = model.free_pages
        self.waiting: Deque[Request] = deque()
        self.running: List[Request] = []
        self._promised: Dict[Hashable, int] = {}

    def submit(self, request: Request) -> None:
        total = len(request.prompt) + request.max_new_tokens
        if not request.prompt or request.max_new_tokens < 1:
            raise ValueError("a request needs a prompt and at least one token to generate")
        if total > int(self.model.desc.max_seq) or self._pages(request) > self.pool_pages:
            raise ValueError(f"request {request.name!r}: {total} tokens do not fit the cache")
        if request.name in self._promised or any(r.name == request.name for r in self.waiting):
            raise ValueError(f"request {request.name!r} is already there")
        self.waiting.append(request)

    @staticmethod
    def _pages(request: Request) -> int:
        return -(-(len(request.prompt) + request.max_new_tokens) // PAGE_TOKENS)

    def _admit(self) -> None:
        while self.waiting and self.slots.free and sum(self._promised.values()) + self._pages(self.waiting[0]) <= self.pool_pages:
            request = self.waiting.popleft()
            self._promised[request.name] = self._pages(request)
            self.slots.of(request.name)
            self.running.append(request)

    def step(self) -> List[Request]:
        """One batch; returns the requests that ended with it."""
        self._admit()
        entries, parts = [], []
        room = self.row_budget
        for r in self.running:   # decoding requests first: they always fit
            if r.generated:
                entries.append((r.name, [r.generated[-1]], [0]))
                parts.append(r)
                room -= 1
        for r in self.running:
            left = len(r.prompt) - r._fed
            if r.generated or room <= 0 or left == 0:
                continue
            take = min(left, room)
            entries.append((r.name, list(r.prompt[r._fed:r._fed + take]), [take - 1] if take == left else []))
            parts.append(r)
            r._fed += take
            room -= take
        if not entries:
            return []
        logits, greedy = self.slots.run(entries, logits=self.sampler is not None)
        row, ended = 0, []
        for (_, _, want), r in zip(entries, parts):
            if not want:
                continue
            token = int(greedy[row]) if self.sampler is None else int(self.sampler(logits[row]))
            row += 1
            r.generated.append(token)
            if len(r.generated) >= r.max_new_tokens or token in r.stop_tokens:
                r.done = True
                ended.append(r)
        for r in ended:
            self.running.remove(r)
            self.slots.release(r.name)
            del self._promised[r.name]
        return ended

    def run(self) -> None:
        """Until every submitted request has ended."""
        while self.waiting or self.running:
            self.step()
