"""Requests in flight over one model and one paged cache.

:class:`Engine` owns the cache: a request holds one of its sequence slots from its first tokens to its release, and pages
of the shared pool as it grows.  :meth:`Engine.step` runs one mixed batch (portions of prompts beside single decoded tokens)
through the library's step call; :class:`Scheduler` composes such steps for submitted prompts - every running request decodes one
token per step, waiting prompts fill the rest of the step's token budget in portions - and samples with the library's own
token selection (repeat penalty, temperature, top-k, top-p).
"""
from __future__ import annotations

import ctypes as C
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from ._lib import check, lib
from .runtime import Model, _p

PAGE = 64  # FORGE_KV_PAGE


@dataclass
class Sampling:
    """Defaults of the generated main.rs except for the penalty (crates/forgellm-codegen-cpu/src/project.rs:608-613)."""
    temperature: float = 0.0
    top_k: int = 0
    top_p: float = 0.9
    repeat_penalty: float = 1.0
    seed: int = 0xDEADBEEF12345678


class Engine:
    def __init__(self, model: Model, pool_tokens: int, slots: int, max_seq: int | None = None):
        self.model = model
        self.cache = model.new_cache(max_seq=max_seq or pool_tokens, batch=slots, pool_tokens=pool_tokens)
        self._free = list(range(slots - 1, -1, -1))
        self._slot: dict = {}

    def admit(self, rid) -> int:
        """A sequence slot for request ``rid``."""
        if rid in self._slot:
            raise ValueError(f"request {rid!r} is already live")
        if not self._free:
            raise RuntimeError("no free sequence slot")
        self._slot[rid] = self._free.pop()
        return self._slot[rid]

    def release(self, rid) -> None:
        """The request is finished: its pages and its slot may be used again."""
        slot = self._slot.pop(rid)
        self.cache.free_seq(slot)
        self._free.append(slot)

    def live(self, rid) -> bool:
        return rid in self._slot

    def free_slots(self) -> int:
        return len(self._free)

    def length(self, rid) -> int:
        return self.cache.len(self._slot[rid])

    def step(self, entries) -> list[np.ndarray]:
        """``entries``: [(request id, tokens, wanted places among them)], one batch.  A request is admitted at its first entry.
        Returns the wanted logits of every entry, [wanted, vocab]."""
        for rid, _, _ in entries:
            if rid not in self._slot:
                self.admit(rid)
        return self.model.step([(self._slot[rid], toks, want) for rid, toks, want in entries], self.cache)

    def close(self) -> None:
        self.cache.close()


@dataclass
class _Request:
    rid: object
    prompt: list
    max_new: int
    sampling: Sampling
    eos: frozenset
    fed: int = 0                      # prompt tokens already in the cache
    out: list = field(default_factory=list)
    rng: C.c_uint64 | None = None
    next: int | None = None

    def pages(self) -> int:
        return -(-(len(self.prompt) + self.max_new) // PAGE)


class Scheduler:
    """Continuous batching: ``submit`` requests, ``run`` to the end (or ``tick`` once per step)."""

    def __init__(self, engine: Engine, step_tokens: int = 2048):
        self.engine = engine
        self.step_tokens = step_tokens
        self.waiting: deque[_Request] = deque()
        self.running: list[_Request] = []
        self.finished: dict = {}
        self._pool_pages = engine.cache.free_tokens() // PAGE
        self._reserved = 0

    def submit(self, rid, prompt, max_new: int, sampling: Sampling | None = None, eos=()) -> None:
        prompt = [int(t) for t in prompt]
        if not prompt or max_new < 1:
            raise ValueError("a request needs a prompt and at least one token to generate")
        r = _Request(rid, prompt, max_new, sampling or Sampling(), frozenset(eos))
        if r.pages() > self._pool_pages:
            raise ValueError("the request does not fit the cache pool")
        r.rng = C.c_uint64(r.sampling.seed)
        self.waiting.append(r)

    def _select(self, r: _Request, logits: np.ndarray) -> int:
        row = np.ascontiguousarray(logits, np.float32).copy()
        if r.out:   # like the reference's loop, the penalty starts with the second token
            recent = np.asarray(r.prompt + r.out, np.uint32)
            check(lib.forge_apply_repeat_penalty(_p(row), row.size, _p(recent), recent.size, r.sampling.repeat_penalty))
        tok = C.c_uint32()
        check(lib.forge_sample(_p(row), row.size, r.sampling.temperature, r.sampling.top_k, r.sampling.top_p, C.byref(r.rng), C.byref(tok)))
        return int(tok.value)

    def tick(self) -> bool:
        """One step; False when nothing is left to do."""
        while self.waiting and self.engine.free_slots() and self._reserved + self.waiting[0].pages() <= self._pool_pages:
            r = self.waiting.popleft()
            self.engine.admit(r.rid)
            self._reserved += r.pages()
            self.running.append(r)
        if not self.running:
            return False
        budget, entries, who = self.step_tokens, [], []
        for r in self.running:            # decoding requests first: one token each
            if r.fed == len(r.prompt):
                entries.append((r.rid, [r.next], [0]))
                who.append(r)
                budget -= 1
        for r in self.running:            # then portions of prompts
            left = len(r.prompt) - r.fed
            n = min(left, budget)
            if n > 0:
                part = r.prompt[r.fed:r.fed + n]
                r.fed += n
                entries.append((r.rid, part, [n - 1] if n == left else []))
                who.append(r)
                budget -= n
        for r, rows in zip(who, self.engine.step(entries)):
            if not len(rows):
                continue
            tok = self._select(r, rows[-1])
            done = tok in r.eos
            if not done:
                r.out.append(tok)
                r.next = tok
                done = len(r.out) == r.max_new
            if done:
                self.engine.release(r.rid)
                self._reserved -= r.pages()
                self.running.remove(r)
                self.finished[r.rid] = r.out
        return True

    def run(self) -> dict:
        """All submitted requests to their end: {request id: generated tokens}."""
        while self.tick():
            pass
        return self.finished
