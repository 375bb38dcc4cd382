"""Serving engine for models that bring their own layer stack (``models.registry.SERVE``).

A step takes the next tokens of any set of sequences - prompts, portions of prompts, single decoded tokens - runs
them as one flat batch against the paged cache and returns the logits asked for.  The model supplies
``stream(batch, cache)``, ``logits(x, rows)``, ``new_cache(...)`` and ``vocab()``; slots, pages, batch layout and decode
graphs live here.

Also usable where a fixed batch advances together (``forward(tokens, commit)``, the interface of
``LlamaInt4Engine``): the speculative decoder runs on it unchanged.
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from types import SimpleNamespace

import torch

from ..ops import _lib


@dataclass(frozen=True)
class Segment:
    """``sequences`` runs of ``count`` consecutive tokens each, from row ``start`` of the batch.  begin: tokens of the
    sequence in ``slot`` that are cached already (several sequences share a segment only with begin == 0)."""
    start: int
    sequences: int
    count: int
    slot: int
    begin: int


@dataclass
class TokenBatch:
    """The flat token batch of a step: ids int64, pos and slot int32, all [N] on the device.  ``prompts`` cover rows
    [0, single_from); the rows after that are handled token by token.  max_len bounds every sequence's length.
    runs [n, 2] int32 on the device: first row and length of every stretch of consecutive tokens of one sequence, the
    prompts' first (None: every row is one).  memo: what layers of one step share."""
    ids: torch.Tensor
    pos: torch.Tensor
    slot: torch.Tensor
    prompts: list[Segment] = field(default_factory=list)
    single_from: int = 0
    max_len: int = 1
    runs: torch.Tensor | None = None
    memo: dict = field(default_factory=dict)


class StackEngine:
    PROMPT_MIN = 32          # shorter portions are handled token by token

    def __init__(self, model, batch: int, max_seq_len: int, page_size: int = 64, pool_tokens: int | None = None, use_graph: bool | None = None):
        """batch: sequences that can be live at once.  pool_tokens: room in the page pool, in tokens (None: every
        sequence owns pages for max_seq_len from the start, as ``forward`` and the speculative decoder need it)."""
        self.model, self.batch, self.max_seq_len = model, batch, max_seq_len
        self.device, self.dtype = model.device, model.dtype
        self.cfg = SimpleNamespace(vocab_size=model.vocab(), model=model.cfg)
        self.pooled = pool_tokens is not None
        kw = {}
        if self.pooled:
            # every live sequence may leave its last page partly empty; one more slot takes the padding rows of graphs
            kw["n_pages"] = (pool_tokens + page_size - 1) // page_size + batch + 1
        self.cache = model.new_cache(batch + (1 if self.pooled else 0), max_seq_len, page_size, **kw)
        # tokens that a caller of ``forward`` may take back after committing them (None: any number)
        self.rollback = self.cache.history - 1 if hasattr(self.cache, "history") else None
        env = os.environ.get("COGITO_SERVE_GRAPH", "1") != "0"
        self.use_graph = (self.device.type == "cuda" and env and self.pooled) if use_graph is None else use_graph
        self._graphs: dict[tuple[int, int], dict] = {}
        self._fresh = True
        if self.pooled:
            self.cached: dict[int, int] = {}                   # slot -> tokens in the cache
            self._pad_slot = self.cache.open()
            self.cache.reserve(self._pad_slot, 1)

    # ------------------------------------------------------------ sequences
    def open(self) -> int:
        slot = self.cache.open()
        self.cached[slot] = 0
        return slot

    def close(self, slot: int):
        del self.cached[slot]
        self.cache.close(slot)

    def free_slots(self) -> int:
        return self.cache.free_slots()

    def room_for(self, length: int) -> bool:
        return self.cache.free_pages() >= self.cache.pages_for(length)

    # ------------------------------------------------------------ one step of any sequences
    @torch.no_grad()
    def step(self, entries: list[tuple[int, list[int], list[int]]], keep=None) -> torch.Tensor:
        """entries: (slot, next tokens, places among them whose logits are wanted).  Returns fp32 logits
        [wanted, vocab] in the order of the entries and places."""
        entries = [(s, t, w) for s, t, w in entries if len(t)]
        if len({s for s, _, _ in entries}) != len(entries):
            raise ValueError("a sequence can only have one entry in a step")
        V = self.cfg.vocab_size
        for s, toks, want in entries:
            if min(toks) < 0 or max(toks) >= V:
                raise ValueError(f"token ids must lie in [0, {V})")
            if any(not 0 <= w < len(toks) for w in want):
                raise ValueError("wanted places must lie among the entry's tokens")
            self.cache.reserve(s, self.cached[s] + len(toks))
        wanted = sum(len(w) for _, _, w in entries)
        if not entries:
            return torch.empty(0, V, device=self.device)
        if self.use_graph and keep is None and all(len(t) == 1 for _, t, _ in entries):
            logits = self._decode_graph(entries)
            rows = [i for i, (_, _, w) in enumerate(entries) for _ in w]
            out = logits[torch.tensor(rows, dtype=torch.int64, device=self.device)] if rows != list(range(len(entries))) else logits.clone()
        else:
            # prompt portions first; the caller's order of the wanted logits is kept by the row list
            order = sorted(range(len(entries)), key=lambda i: len(entries[i][1]) < self.PROMPT_MIN)
            ids, pos, slot, segs, runs, single = [], [], [], [], [], None
            first = {}
            for i in order:
                s, toks, _ = entries[i]
                n, begin = len(toks), self.cached[s]
                first[i] = len(ids)
                if n >= self.PROMPT_MIN:
                    segs.append(Segment(len(ids), 1, n, s, begin))
                elif single is None:
                    single = len(ids)
                runs.append((len(ids), n))
                ids += toks
                pos += range(begin, begin + n)
                slot += [s] * n
            host = torch.tensor([ids, pos, slot], dtype=torch.int64)
            dev = host.to(self.device)
            small = dev[1:].to(torch.int32)
            batch = TokenBatch(dev[0], small[0], small[1], segs, len(ids) if single is None else single, max(pos) + 1,
                               torch.tensor(runs, dtype=torch.int32).to(self.device))
            x = self.model.stream(batch, self.cache, **({} if keep is None else {"keep": keep}))
            rows = [first[i] + w for i, (_, _, want) in enumerate(entries) for w in want]
            out = torch.empty(0, V, device=self.device)
            if rows:
                out = self.model.logits(x, torch.tensor(rows, dtype=torch.int64).to(self.device))
        for s, toks, _ in entries:
            self.cached[s] += len(toks)
        assert out.shape[0] == wanted
        return out

    # ------------------------------------------------------------ decode graphs
    def _decode_graph(self, entries) -> torch.Tensor:
        """One token of each of up to 2^k sequences: the step's ~15 kernels per layer are replayed from a CUDA graph per
        batch size (padded with rows of a scratch sequence) and power-of-two bound of the sequence length."""
        n = len(entries)
        size = 1 << (n - 1).bit_length()
        longest = max(self.cached[s] + 1 for s, _, _ in entries)
        bound = min(max(256, 1 << (longest - 1).bit_length()), self.cache.max_pages * self.cache.page_size)
        g = self._graphs.get((size, bound))
        if g is None:
            g = self._capture(size, bound)
        pad = size - n
        host = torch.tensor([[t[0] for _, t, _ in entries] + [0] * pad, [self.cached[s] for s, _, _ in entries] + [0] * pad,
                             [s for s, _, _ in entries] + [self._pad_slot] * pad], dtype=torch.int64)
        g["in"].copy_(host)
        g["graph"].replay()
        _lib.count_launch(g["launches"])
        return g["logits"][:n]

    def _capture(self, size: int, bound: int) -> dict:
        host = torch.tensor([[0] * size, [0] * size, [self._pad_slot] * size], dtype=torch.int64)
        g = {"in": host.to(self.device)}

        def run():
            small = g["in"][1:].to(torch.int32)
            return self.model.logits(self.model.stream(TokenBatch(g["in"][0], small[0], small[1], [], 0, bound), self.cache))
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):                        # lazily created state (counters, function attributes) comes first
            run()
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        g["graph"] = torch.cuda.CUDAGraph()
        before = _lib.launches()
        with torch.cuda.graph(g["graph"]):
            g["logits"] = run()
        g["launches"] = _lib.launches() - before
        self._graphs[(size, bound)] = g
        return g

    # ------------------------------------------------------------ a fixed batch that advances together
    def reset(self):
        if self.pooled:
            raise RuntimeError("a pooled engine opens and closes sequences one by one")
        self.cache.reset()
        self._fresh = True

    @torch.no_grad()
    def forward(self, tokens: torch.Tensor, commit: bool = False) -> torch.Tensor:
        """tokens [batch, T] at positions lengths[b] + t -> logits [batch, T, V] (fp32).  The cache lengths move only
        with ``commit`` (a verify pass followed by a partial commit rolls the rejected positions back)."""
        if self.pooled:
            raise RuntimeError("forward() needs an engine whose sequences own their pages (pool_tokens=None)")
        B, T = tokens.shape
        dev = self.device
        fresh, self._fresh = self._fresh and T >= self.PROMPT_MIN, False
        if T > self.max_seq_len:
            raise ValueError("the sequence exceeds the cache")
        pos = (self.cache.lengths[:, None] + torch.arange(T, device=dev, dtype=torch.int32)[None]).reshape(-1)
        slot = torch.arange(B, device=dev, dtype=torch.int32).repeat_interleave(T)
        batch = TokenBatch(tokens.reshape(-1).long(), pos, slot, max_len=self.max_seq_len)
        if T > 1:
            first = torch.arange(0, B * T, T, device=dev, dtype=torch.int32)
            batch.runs = torch.stack([first, torch.full_like(first, T)], 1)
        if fresh:
            batch.prompts, batch.single_from = [Segment(0, B, T, 0, 0)], B * T
        logits = self.model.logits(self.model.stream(batch, self.cache)).view(B, T, -1)
        if commit:
            self.cache.commit(T)
        return logits
