"""Continuous batching for models with per-sequence state slots.

A request waits for a slot, its prompt is run in portions of at most ``portion`` tokens beside the decode tokens of the
other requests, then it decodes one token per step until its length or an end token; its slot goes to the next request.
Every step is one packed ``model.step``; steps that only decode replay a CUDA graph (``graphs``), one for each of a few batch
sizes that smaller batches are filled up to.
"""
from __future__ import annotations

import itertools
from collections import deque
from dataclasses import dataclass, field
from typing import Deque, Dict, List, Optional, Sequence

import torch

from .generate import choose_tokens


@dataclass
class SequenceRequest:
    tokens: List[int]
    max_new_tokens: int
    eos_token_ids: Sequence[int] = ()
    temperature: float = 0.0
    top_p: Optional[float] = None
    seed: Optional[int] = None
    tag: object = None                       # the caller's
    id: int = -1
    output: List[int] = field(default_factory=list)
    fed: int = 0                             # prompt tokens already in the cache
    finished: bool = False


class Scheduler:
    def __init__(self, model, max_batch: int = 64, max_len: int = 8192, portion: int = 2048, step_tokens: int = 8192,
                 graphs: bool = True):
        self.model, self.max_batch, self.portion, self.step_tokens = model, max_batch, max(portion, 1), max(step_tokens, 1)
        self.cache = model.new_cache(max_batch, max_len)
        self.waiting: Deque[SequenceRequest] = deque()
        self.running: Dict[int, SequenceRequest] = {}
        self._ids = itertools.count()
        self._rng: Dict[int, torch.Generator] = {}
        self._graphs: Optional[dict] = {} if graphs and model.device.type == "cuda" else None
        self._seen: Dict[int, int] = {}
        self._pool = None

    # ------------------------------------------------------------------ requests
    def check(self, request: SequenceRequest) -> None:
        """Raises ``ValueError`` for a request that cannot be served."""
        if not request.tokens:
            raise ValueError("a request needs at least one token")
        if request.max_new_tokens < 1:
            raise ValueError("a request asks for at least one new token")
        if len(request.tokens) + request.max_new_tokens > self.cache.max_len:
            raise ValueError(f"{len(request.tokens)} + {request.max_new_tokens} tokens do not fit the {self.cache.max_len} a slot holds")
        if min(request.tokens) < 0 or max(request.tokens) >= self.model.config.vocab:
            raise ValueError("token id outside the vocabulary")

    def submit(self, request: SequenceRequest) -> int:
        self.check(request)
        request.id = next(self._ids)
        self.waiting.append(request)
        return request.id

    def cancel(self, request_id: int) -> None:
        self.waiting = deque(r for r in self.waiting if r.id != request_id)
        if self.running.pop(request_id, None) is not None:
            self.cache.release(request_id)
            self._rng.pop(request_id, None)

    @property
    def busy(self) -> bool:
        return bool(self.waiting or self.running)

    # ------------------------------------------------------------------ one step
    def _admit(self) -> None:
        while self.waiting and self.cache.free_slots:
            r = self.waiting.popleft()
            self.cache.acquire(r.id)
            self.running[r.id] = r
            if r.temperature and r.temperature > 0 and r.seed is not None:
                g = torch.Generator(device=self.model.device)
                g.manual_seed(r.seed)
                self._rng[r.id] = g

    def _plan(self):
        """(request, tokens, wanted places) of the next step: every decoding request's token, then prompt portions while
        the step's token budget lasts."""
        entries, budget = [], self.step_tokens
        for r in self.running.values():
            if r.fed == len(r.tokens):
                entries.append((r, [r.output[-1]], [0]))
                budget -= 1
        for r in self.running.values():
            left = len(r.tokens) - r.fed
            n = min(left, self.portion, max(budget, 0 if entries else 1))
            if left and n:
                entries.append((r, r.tokens[r.fed:r.fed + n], [n - 1] if n == left else []))
                budget -= n
        return entries

    def _decode_logits(self, entries) -> Optional[torch.Tensor]:
        """Logits of a decode-only step from the graph of the next batch size, captured once that has come up three times."""
        if self._graphs is None or any(len(r.tokens) != r.fed for r, _, _ in entries):
            return None
        n = len(entries)
        size = min(n if n <= 4 else (n + 7) // 8 * 8, self.max_batch)
        if size not in self._graphs:
            self._seen[size] = self._seen.get(size, 0) + 1
            if self._seen[size] < 3:
                return None
            from .hybrid import GraphedDecode
            if self._pool is None:
                self._pool = torch.cuda.graph_pool_handle()       # the graphs never run at once: one pool for all
            self._graphs[size] = GraphedDecode(self.model, self.cache, size, self._pool)
        c = self.cache
        logits = self._graphs[size].run([t[0] for _, t, _ in entries], [c.length(r.id) for r, _, _ in entries],
                                        [c.slot(r.id) for r, _, _ in entries])
        for r, _, _ in entries:
            c.advance(r.id, 1)
        return logits

    def step(self) -> List[SequenceRequest]:
        """Runs one step; returns the requests it finished."""
        self._admit()
        plan = self._plan()
        if not plan:
            return []
        logits = self._decode_logits(plan)
        if logits is None:
            logits = self.model.run([(r.id, t, w) for r, t, w in plan], self.cache)
        asked = [r for r, _, w in plan if w]
        for r, t, _ in plan:
            if r.fed < len(r.tokens):
                r.fed += len(t)
        if not asked:
            return []
        tokens = choose_tokens(logits, [r.temperature for r in asked], [r.top_p for r in asked],
                               [self._rng.get(r.id) for r in asked])
        done = []
        for r, tok in zip(asked, tokens):
            r.output.append(tok)
            if len(r.output) >= r.max_new_tokens or tok in r.eos_token_ids:
                r.finished = True
                del self.running[r.id]
                self.cache.release(r.id)
                self._rng.pop(r.id, None)
                done.append(r)
        return done

    def run(self) -> List[SequenceRequest]:
        """Steps until nothing is left; the finished requests in order of completion."""
        done: List[SequenceRequest] = []
        while self.busy:
            done += self.step()
        self.model.check_status()
        return done
