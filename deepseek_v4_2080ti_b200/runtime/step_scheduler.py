"""Continuous batching over a runtime with a mixed-batch ``step`` (``models/paged.py``): every round is ONE pass in which
the running requests advance by one token each and waiting prompts are filled in portions beside them, bounded by a token
budget.  Greedy; requests are admitted first come first served once a slot and the pages of their worst case are free.

(Role of the background scheduler in cpp_engine/include/batch_scheduler.hpp:75-193; the C++ ``BatchScheduler`` of this
package drives engines that keep prefill and decode apart.)
"""
from __future__ import annotations

import time
from collections import deque
from dataclasses import dataclass, field


@dataclass
class _Request:
    index: int
    prompt: list[int]
    max_new: int
    pages: int = 0
    slot: int = -1
    fed: int = 0                                   # prompt tokens already in the cache
    out: list[int] = field(default_factory=list)
    t_admit: float = 0.0
    t_first: float = 0.0


class StepScheduler:
    def __init__(self, rt, eos_ids=(), max_batch: int = 8, token_budget: int = 8192):
        self.rt, self.eos = rt, set(eos_ids)
        self.max_batch = max(1, min(int(max_batch), rt.max_slots))
        self.budget = max(self.max_batch, int(token_budget))
        self.waiting: deque[_Request] = deque()
        self.running: list[_Request] = []
        self.reserved = 0
        self.rounds = self.mixed_rounds = 0

    def submit(self, index: int, prompt, max_new: int) -> None:
        prompt = [int(t) for t in prompt]
        if not prompt:
            raise ValueError("a request needs at least one prompt token")
        r = _Request(index, prompt, max(1, int(max_new)))
        total = len(prompt) + r.max_new - 1        # the last generated token is never fed back
        if total > self.rt.max_context:
            raise ValueError(f"request {index}: {total} tokens do not fit the context of {self.rt.max_context}")
        r.pages = self.rt.pages_held(total, min(len(prompt), self.budget))
        if r.pages > self.rt.num_blocks - 1:
            raise ValueError(f"request {index} needs {r.pages} pages, the pool has {self.rt.num_blocks - 1}")
        self.waiting.append(r)

    def _admit(self) -> None:
        while self.waiting and len(self.running) < self.max_batch and self.rt.free_slots:
            r = self.waiting[0]
            if self.reserved + r.pages > self.rt.num_blocks - 1:
                return                             # head of the line waits for pages
            self.waiting.popleft()
            r.slot, r.t_admit = self.rt.allocate(), time.perf_counter()
            self.reserved += r.pages
            self.running.append(r)

    def _finish(self, r: _Request):
        self.rt.free(r.slot)
        self.reserved -= r.pages
        self.running.remove(r)
        stop = r.out[-1] in self.eos
        now = time.perf_counter()
        return r.index, (r.out[:-1] if stop else r.out, "stop" if stop else "length",
                         {"prefill_seconds": r.t_first - r.t_admit, "decode_seconds": now - r.t_first,
                          "total_seconds": now - r.t_admit, "ttft_seconds": r.t_first - r.t_admit})

    def round(self) -> list[tuple[int, tuple]]:
        """One pass; returns the requests it finished as (index, (tokens, reason, timing))."""
        self._admit()
        entries, owners = [], []
        left = self.budget
        for r in self.running:
            if r.fed == len(r.prompt):
                entries.append((r.slot, [r.out[-1]], [0]))
                owners.append(r)
                left -= 1
        decoding = len(entries)
        for r in self.running:
            n = min(left, len(r.prompt) - r.fed)
            if n <= 0:
                continue
            r.fed += n
            left -= n
            last = r.fed == len(r.prompt)
            entries.append((r.slot, r.prompt[r.fed - n:r.fed], [n - 1] if last else []))
            if last:
                owners.append(r)
        if not entries:
            return []
        self.rounds += 1
        self.mixed_rounds += int(0 < decoding < len(entries))
        logits = self.rt.step(entries)
        done = []
        if owners:
            for r, tok in zip(owners, self.rt.greedy(logits)):
                if not r.out:
                    r.t_first = time.perf_counter()
                r.out.append(tok)
                if tok in self.eos or len(r.out) >= r.max_new:
                    done.append(r)
        return [self._finish(r) for r in done]

    def run(self) -> dict[int, tuple]:
        results: dict[int, tuple] = {}
        try:
            while self.waiting or self.running:
                results.update(self.round())
        finally:
            for r in self.running:                 # only after an error: give back what is held
                self.rt.free(r.slot)
            self.running, self.reserved = [], 0
        return results
