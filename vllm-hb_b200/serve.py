"""Continuous batching over Engine.step: requests are admitted while blocks and state slots last,
every step mixes single decoded tokens with portions of prompts under a token budget, finished
requests give back what they hold.

    sched = Scheduler(engine)
    sched.submit(Request("a", prompt_ids, max_tokens=32))
    sched.run()  -> {"a": [generated ids]}

Greedy requests take the step's arg-max; requests with a temperature are drawn on the device from
the logits the step left there.  Works with every model family (the engine's step is the same).
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Optional

BLOCK = 16


@dataclass
class Request:
    id: str
    prompt: list
    max_tokens: int = 16
    temperature: float = 0.0
    top_p: float = 1.0
    seed: int = 0
    stop_ids: tuple = ()
    output: list = field(default_factory=list)

    def total(self) -> int:
        """Tokens the engine will hold at most (the last generated token is never fed)."""
        return len(self.prompt) + self.max_tokens - 1


@dataclass
class _Live:
    req: Request
    seq: object
    fed: int = 0  # tokens of prompt + output already in the cache

    def tokens(self) -> list:
        return self.req.prompt + self.req.output

    def pending(self) -> int:
        return len(self.req.prompt) + len(self.req.output) - self.fed


class Scheduler:
    def __init__(self, engine, *, max_live: int = 64, step_tokens: int = 256):
        # a step is one batch of the engine, and every live request may hold a state slot
        slots = engine.num_free_state_slots()
        self.engine = engine
        self.max_live = min(max_live, slots) if slots > 0 else max_live
        self.step_tokens = min(step_tokens, engine.max_batch)
        self.waiting: deque[Request] = deque()
        self.live: list[_Live] = []
        self.done: dict[str, list] = {}
        self.total_blocks = engine.num_free_blocks()
        self.reserved = 0  # blocks promised to live requests

    def submit(self, req: Request) -> None:
        if not req.prompt or req.max_tokens < 1:
            raise ValueError("a request needs a prompt and at least one token to generate")
        if self._blocks(req) > self.total_blocks:
            raise ValueError(f"request {req.id} needs {self._blocks(req)} blocks, the pool has {self.total_blocks}")
        self.waiting.append(req)

    @staticmethod
    def _blocks(req: Request) -> int:
        return -(-req.total() // BLOCK)

    def _admit(self) -> None:
        # in order of arrival; a request holds a promise for every block it may come to need, so a
        # live request never runs out in the middle
        while self.waiting and len(self.live) < self.max_live:
            need = self._blocks(self.waiting[0])
            if self.reserved + need > self.total_blocks:
                return
            self.reserved += need
            req = self.waiting.popleft()
            self.live.append(_Live(req, self.engine.create_kv_cache()))

    def step(self) -> bool:
        """One engine step; False when there is nothing left to do."""
        self._admit()
        if not self.live:
            return False
        budget, plan = self.step_tokens, []
        for l in self.live:                     # decoded tokens first: they keep their pace
            if l.pending() == 1 and budget > 0:
                plan.append((l, 1))
                budget -= 1
        for l in self.live:                     # then portions of prompts, oldest first
            if l.pending() > 1 and budget > 0:
                n = min(l.pending(), budget)
                plan.append((l, n))
                budget -= n
        entries, asked = [], []
        for l, n in plan:
            last = n == l.pending()
            entries.append((l.seq, l.tokens()[l.fed:l.fed + n], [n - 1] if last else []))
            if last:
                asked.append(l)
        nxt, _ = self.engine.step(entries, logits=False)
        picked = [int(t) for t in nxt]
        groups: dict[tuple, list] = {}
        for i, l in enumerate(asked):
            if l.req.temperature > 0.0:
                groups.setdefault((l.req.temperature, l.req.top_p), []).append(i)
        for (temperature, top_p), rows in groups.items():
            # the draw of a token depends on its request's seed and its place, not on the batch
            seeds = [a.req.seed * 1000003 + len(a.req.output) for a in asked]
            drawn = self.engine.sample(seeds, temperature, top_p)
            for i in rows:
                picked[i] = int(drawn[i])
        for l, n in plan:
            l.fed += n
        for l, tok in zip(asked, picked):
            l.req.output.append(tok)
            if len(l.req.output) >= l.req.max_tokens or tok in l.req.stop_ids:
                self.done[l.req.id] = l.req.output
                l.seq.free()
                self.reserved -= self._blocks(l.req)
                self.live.remove(l)
        return True

    def run(self) -> dict:
        while self.step():
            pass
        return self.done


def generate(engine, prompts, max_tokens: int = 16, *, max_live: int = 64, step_tokens: int = 256,
             temperature: float = 0.0, top_p: float = 1.0, seed: Optional[int] = 0) -> list:
    """Generated token ids of every prompt, batched by a Scheduler."""
    sched = Scheduler(engine, max_live=max_live, step_tokens=step_tokens)
    for i, p in enumerate(prompts):
        sched.submit(Request(str(i), [int(t) for t in p], max_tokens, temperature, top_p, (seed or 0) + i))
    out = sched.run()
    return [out[str(i)] for i in range(len(prompts))]
