"""Continuous batching over an engine: waiting requests are admitted while slots and pages last, prompts are fed in
portions of at most ``prefill_budget`` tokens per step, everything that has finished its prompt is decoded together
(scheduler/scheduler.py and scheduler/prefill.py of the reference play this part)."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Deque, Dict, Iterable, List, Optional, Sequence

from ..core import Req
from .engine import Engine
from .sample import greedy


@dataclass(frozen=True)
class SamplingParams:
    max_new_tokens: int = 16
    stop_ids: tuple = ()


@dataclass(eq=False)
class GenerationRequest:
    uid: int
    prompt: List[int]
    params: SamplingParams
    output: List[int] = field(default_factory=list)
    fed: int = 0                          # tokens of prompt + output already run
    req: Optional[Req] = None
    pages: int = 0                        # reserved

    @property
    def finished(self) -> bool:
        return len(self.output) >= self.params.max_new_tokens or (bool(self.output) and self.output[-1] in self.params.stop_ids)


class Scheduler:
    def __init__(self, engine: Engine, prefill_budget: Optional[int] = None):
        self.engine = engine
        self.budget = min(prefill_budget or engine.max_portion, engine.max_portion)
        self.waiting: Deque[GenerationRequest] = deque()
        self.prefilling: List[GenerationRequest] = []
        self.decoding: List[GenerationRequest] = []
        self._reserved = 0
        self._next_uid = 0

    def add(self, prompt: Sequence[int], params: SamplingParams = SamplingParams()) -> GenerationRequest:
        if not prompt or params.max_new_tokens < 1:
            raise ValueError("a request needs a prompt and at least one new token")
        total = len(prompt) + params.max_new_tokens
        if total > self.engine.max_len:
            raise ValueError(f"prompt and new tokens ({total}) exceed the engine's max_len {self.engine.max_len}")
        g = GenerationRequest(self._next_uid, list(prompt), params)
        # the last new token is never run
        g.pages = self.engine.manager.pages_for(total - 1, min(len(prompt), self.budget))
        if g.pages > self.engine.manager.num_pages:
            raise ValueError(f"the request needs {g.pages} pages, the cache has {self.engine.manager.num_pages}")
        self._next_uid += 1
        self.waiting.append(g)
        return g

    @property
    def busy(self) -> bool:
        return bool(self.waiting or self.prefilling or self.decoding)

    def _admit(self) -> None:
        m = self.engine.manager
        while self.waiting and m.free_slots and self._reserved + self.waiting[0].pages <= m.num_pages:
            g = self.waiting.popleft()
            g.req = self.engine.open()
            self._reserved += g.pages
            self.prefilling.append(g)

    def _retire(self, g: GenerationRequest) -> None:
        self.engine.close(g.req)
        g.req = None
        self._reserved -= g.pages

    def step(self) -> List[GenerationRequest]:
        """One forward: prompt portions if any are left, else one token for every running request.  Returns the requests
        that finished."""
        self._admit()
        if self.prefilling:
            work, left = [], self.budget
            for g in self.prefilling:
                n = min(left, len(g.prompt) - g.fed)
                if n <= 0:
                    break
                work.append((g, g.prompt[g.fed:g.fed + n]))
                left -= n
        else:
            work = [(g, [g.output[-1]]) for g in self.decoding]
        if not work:
            return []
        complete = [g.fed + len(t) >= len(g.prompt) for g, t in work]
        logits = self.engine.step([g.req for g, _ in work], [t for _, t in work], [[len(t) - 1] if c else [] for (_, t), c in zip(work, complete)])
        tokens = greedy(logits).tolist() if logits is not None else []
        self.engine.check_status()
        done, k = [], 0
        for (g, t), c in zip(work, complete):
            g.fed += len(t)
            if not c:
                continue
            g.output.append(tokens[k])
            k += 1
            if g in self.prefilling:
                self.prefilling.remove(g)
                self.decoding.append(g)
            if g.finished:
                self.decoding.remove(g)
                self._retire(g)
                done.append(g)
        return done

    def generate(self, prompts: Iterable[Sequence[int]], params: SamplingParams = SamplingParams()) -> List[List[int]]:
        """New tokens of every prompt, in order."""
        gs = [self.add(p, params) for p in prompts]
        finished: Dict[int, bool] = {}
        while self.busy:
            for g in self.step():
                finished[g.uid] = True
        assert all(finished.get(g.uid) for g in gs)
        return [g.output for g in gs]
