"""Requests on a ``StackEngine``: admission, prompt portions, decoding and sampling.

Every step carries one token of each running request and fills the rest of its token budget with portions of waiting
prompts, so long prompts do not hold up decoding.  A request is admitted when a sequence slot is free and the page
pool has room for its prompt and all its new tokens; pages are taken as the sequence grows and returned
when it ends.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field

import torch

from .sampling import sample


@dataclass(eq=False)
class Request:
    prompt: list[int]
    max_new_tokens: int
    stop_token: int | None = None
    tokens: list[int] = field(default_factory=list)      # generated
    slot: int | None = None
    fed: int = 0                                         # prompt tokens in the cache
    done: bool = False

    def total(self) -> int:
        return len(self.prompt) + self.max_new_tokens


class Scheduler:
    def __init__(self, engine, temperature: float = 0.0, top_k: int = 0, top_p: float = 1.0, seed: int = 0, step_tokens: int = 2048):
        self.engine, self.step_tokens = engine, step_tokens
        self.sampling = dict(temperature=temperature, top_k=top_k, top_p=top_p, seed=seed)
        self.waiting: deque[Request] = deque()
        self.running: list[Request] = []
        self.steps = 0

    def add(self, prompt, max_new_tokens: int, stop_token: int | None = None) -> Request:
        r = Request([int(t) for t in prompt], int(max_new_tokens), stop_token)
        if not r.prompt or r.max_new_tokens < 1:
            raise ValueError("a request needs a prompt and at least one new token")
        cache = self.engine.cache
        # one page is the engine's own; a request that can never be admitted must not block the queue
        if r.total() > cache.max_pages * cache.page_size or cache.pages_for(r.total()) > cache.n_pages - 1:
            raise ValueError(f"a request of {r.total()} tokens exceeds the cache")
        self.waiting.append(r)
        return r

    def _promised(self) -> int:
        """Pages that running requests may still take."""
        c = self.engine.cache
        return sum(c.pages_for(r.total()) - c.pages_for(self.engine.cached[r.slot]) for r in self.running)

    def _admit(self):
        c = self.engine.cache
        while self.waiting and self.engine.free_slots():
            r = self.waiting[0]
            if c.pages_for(r.total()) > c.free_pages() - self._promised():
                break
            r.slot = self.engine.open()
            self.running.append(self.waiting.popleft())

    def step(self) -> list[Request]:
        """One engine step; returns the requests that ended in it."""
        self._admit()
        entries, readers, budget = [], [], self.step_tokens
        for r in self.running:
            if r.fed == len(r.prompt):
                entries.append((r.slot, [r.tokens[-1]], [0]))
                readers.append(r)
                budget -= 1
        for r in self.running:
            n = min(len(r.prompt) - r.fed, budget)
            if n > 0:
                part = r.prompt[r.fed:r.fed + n]
                r.fed += n
                budget -= n
                last = r.fed == len(r.prompt)
                entries.append((r.slot, part, [n - 1] if last else []))
                if last:
                    readers.append(r)
        if not entries:
            return []
        logits = self.engine.step(entries)
        self.steps += 1
        ended = []
        if readers:
            for r, tok in zip(readers, sample(logits, step=self.steps, **self.sampling).tolist()):
                r.tokens.append(tok)
                if len(r.tokens) == r.max_new_tokens or tok == r.stop_token:
                    r.done = True
                    ended.append(r)
        for r in ended:
            self.running.remove(r)
            self.engine.close(r.slot)
        return ended

    def run(self) -> None:
        while self.waiting or self.running:
            self.step()


def generate(engine, prompts, max_new_tokens: int, **sampling) -> list[list[int]]:
    """New tokens of every prompt (lists of token ids of any lengths)."""
    s = Scheduler(engine, **sampling)
    reqs = [s.add(p, max_new_tokens) for p in prompts]
    s.run()
    return [r.tokens for r in reqs]
