"""Scheduler of step engines: decides which tokens of which request go into the next batch.

Every step carries one token of each request that is generating, plus portions of waiting prompts up to a row budget, so prompts
never stall the requests that are already producing tokens. A request is admitted when a slot is free and the cache pool has
pages for the whole sequence it may grow to (prompt + new tokens, or the window when every layer has one); what it holds is given
back when it finishes.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Sequence

from .engine import KV_PAGE, ResidentEngine, Sampling, StepEntry

__all__ = ["StepRequest", "StepScheduler"]


@dataclass
class StepRequest:
    id: int
    prompt: list[int]
    max_new_tokens: int
    sampling: Sampling
    eos_token: int | None
    slot: int = -1
    fed: int = 0                       # prompt tokens already run
    out: list[int] = field(default_factory=list)
    reserved: int = 0                  # pages set aside at admission


class StepScheduler:
    """``step_rows``: most rows of one step (prompt portions are cut to fit); default: the engine's own limit."""

    def __init__(self, engine: ResidentEngine, *, step_rows: int | None = None) -> None:
        if not engine.has_steps:
            raise ValueError("this engine runs whole prompts and decode steps only")
        self.engine = engine
        cfg = engine.config
        self.step_rows = max(1, min(step_rows or cfg.max_step_rows, cfg.max_step_rows))
        self._free = list(range(cfg.max_batch))[::-1]
        self._waiting: list[StepRequest] = []
        self._live: list[StepRequest] = []
        self._done: dict[int, list[int]] = {}
        self._total = self._pages = engine.free_tokens // KV_PAGE
        self._next_id = 0

    def submit(self, prompt: Sequence[int], max_new_tokens: int, sampling: Sampling | None = None, eos_token: int | None = None) -> int:
        cfg = self.engine.config
        if not prompt or len(prompt) >= cfg.max_seq:
            raise ValueError("the prompt must hold between 1 and max_seq - 1 tokens")
        r = StepRequest(self._next_id, [int(t) for t in prompt], int(max_new_tokens), sampling or Sampling(), eos_token)
        if self._pages_for(r) > self._total:
            raise ValueError("the request does not fit the cache pool")
        self._next_id += 1
        if r.max_new_tokens <= 0:
            self._done[r.id] = []
        else:
            self._waiting.append(r)
        return r.id

    def _pages_for(self, r: StepRequest) -> int:
        cfg = self.engine.config
        tokens = min(len(r.prompt) + r.max_new_tokens, cfg.max_seq)
        if cfg.window:   # pages behind the window go back while the sequence grows
            tokens = min(tokens, cfg.window + min(self.step_rows, max(len(r.prompt), 1)) + KV_PAGE)
        return (tokens + KV_PAGE - 1) // KV_PAGE

    def _admit(self) -> None:
        while self._waiting and self._free:
            need = self._pages_for(self._waiting[0])
            if need > self._pages:
                return
            r = self._waiting.pop(0)
            self._pages -= need
            r.reserved, r.slot = need, self._free.pop()
            self.engine.release(r.slot)
            self._live.append(r)

    def step(self) -> bool:
        """Runs one batch; False when nothing is left to do."""
        self._admit()
        if not self._live:
            return False
        room = self.step_rows
        batch: list[tuple[StepRequest, StepEntry]] = []
        for r in self._live:                               # generating requests first: one row each
            if r.fed == len(r.prompt) and room > 0:
                batch.append((r, StepEntry(r.slot, [r.out[-1]], (0,), r.sampling)))
                room -= 1
        for r in self._live:                               # then prompts, in order of arrival
            n = min(len(r.prompt) - r.fed, room)
            if n > 0:
                part = r.prompt[r.fed:r.fed + n]
                batch.append((r, StepEntry(r.slot, part, (n - 1,) if r.fed + n == len(r.prompt) else (), r.sampling)))
                room -= n
        drawn, _ = self.engine.step([e for _, e in batch])
        for (r, e), toks in zip(batch, drawn):
            if r.fed < len(r.prompt):
                r.fed += len(e.tokens)
            if toks:
                r.out.append(toks[0])
                full = len(r.prompt) + len(r.out) >= self.engine.config.max_seq
                if len(r.out) >= r.max_new_tokens or full or (r.eos_token is not None and toks[0] == r.eos_token):
                    self._finish(r)
        return True

    def _finish(self, r: StepRequest) -> None:
        self.engine.release(r.slot)
        self._free.append(r.slot)
        self._pages += r.reserved
        self._live.remove(r)
        self._done[r.id] = r.out

    def run(self) -> dict[int, list[int]]:
        """Until every submitted request is finished; request id -> generated tokens."""
        while self.step():
            pass
        done, self._done = self._done, {}
        return done
