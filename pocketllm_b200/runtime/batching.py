"""Continuous batching over a step function that takes mixed batches (`runtime.mixer_runtime.MixerRuntime`): requests join
and leave between steps, every running generation advances by one token per step, and prompts fill the rest of the step's
token budget in portions.

Who goes next is `PDScheduler.next_batch` (generations before prompts, prompts in order); room is taken when a request is
admitted, for its prompt and everything it may generate, so a running request never runs out of pages. Greedy requests
without anybody waiting run bursts of steps on the device; sampled ones take every step's logits through the sampler of
the servers.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Sequence

import torch

from ..server.engine import SamplingParams, apply_penalties, sample_token, token_logprobs
from .mixer_runtime import StepEntry
from .pd_scheduler import PDScheduler
from .request_cache import CacheFull


@dataclass(eq=False)
class Request:
    rid: int
    prompt: list[int]
    params: SamplingParams
    limit: int                                   # tokens it may generate
    done: int = 0                                # prompt tokens that have run
    out: list[int] = field(default_factory=list)
    generator: torch.Generator | None = None

    @property
    def greedy(self) -> bool:
        p = self.params
        return p.temperature <= 0 and p.logprobs < 0 and p.repetition_penalty == 1.0 and p.frequency_penalty == 0 and p.presence_penalty == 0

    @property
    def finished(self) -> bool:
        return len(self.out) >= self.limit or bool(self.out and self.out[-1] in self.params.stop_token_ids)


class BatchEngine:
    def __init__(self, runtime, *, token_budget: int = 2048, burst: int = 8, max_pending: int = 1 << 16, max_batch: int | None = None):
        self.rt, self.token_budget, self.burst = runtime, token_budget, burst
        self.max_batch = min(max_batch or runtime.max_requests, runtime.max_requests)
        self.sched = PDScheduler(max_pending=max_pending)
        self.requests: dict[int, Request] = {}
        self._next = 0
        self.stats = {"steps": 0, "burst_steps": 0, "mixed_steps": 0, "tokens": 0}

    def submit(self, prompt: Sequence[int], params: SamplingParams) -> int:
        """Queue a request; returns its id. A prompt that can never fit is refused here."""
        prompt = [int(t) for t in prompt]
        room = self.rt.max_tokens - len(prompt) + 1               # the last generated token is not run
        if not prompt:
            raise ValueError("an empty prompt")
        if room < 1:
            raise ValueError(f"{len(prompt)} prompt tokens exceed the cache of {self.rt.max_tokens}")
        if any(not 0 <= t < self.rt.vocab for t in prompt):
            raise ValueError("token id outside the vocabulary")
        r = Request(self._next, prompt, params, max(1, min(params.max_tokens, room)))
        if params.seed is not None:
            r.generator = torch.Generator().manual_seed(int(params.seed))
        if not self.sched.submit(r):
            raise RuntimeError("too many waiting requests")
        self._next += 1
        self.requests[r.rid] = r
        return r.rid

    def _admit(self, r: Request) -> bool:
        try:
            self.rt.cache.reserve({r.rid: len(r.prompt) + r.limit - 1})
        except CacheFull:
            return False
        return True

    def _end(self, r: Request) -> None:
        self.sched.finish(r)
        self.requests.pop(r.rid, None)
        if r.rid in self.rt.cache:
            self.rt.release(r.rid)

    def cancel(self, rid: int) -> None:
        r = self.requests.get(rid)
        if r is not None:
            self.sched.drop(r)
            self._end(r)

    def abort_all(self) -> None:
        for rid in list(self.requests):
            self.cancel(rid)

    @property
    def idle(self) -> bool:
        return not self.requests

    def step(self) -> list[tuple[int, object, bool]]:
        """Run one batch (or a burst of greedy steps). Returns (request id, token, finished) in order; tokens are `TokenInfo`
        where log-probabilities were asked for."""
        work = self.sched.next_batch(self.max_batch, self.token_budget, lambda r: len(r.prompt) - r.done, self._admit)
        if not work:
            if self.requests:
                raise CacheFull("no waiting request fits into the cache")
            return []
        self.stats["steps"] += 1
        if all(ph == "decode" and r.greedy for r, ph, _ in work) and self.sched.pending() == (0, 0) and len(work) <= 8:
            return self._burst([r for r, _, _ in work])
        entries, rows = [], []
        for r, phase, n in work:
            if phase == "decode":
                entries.append(StepEntry(r.rid, [r.out[-1]], (0,)))
            else:
                end = r.done + n
                entries.append(StepEntry(r.rid, r.prompt[r.done:end], (n - 1,) if end == len(r.prompt) else ()))
                r.done = end
            if entries[-1].want:
                rows.append(r)
        self.stats["mixed_steps"] += int(len({ph for _, ph, _ in work}) > 1)
        logits = self.rt.step(entries)
        self.rt.check_status()
        best = logits.argmax(-1).tolist() if rows else []
        events = []
        for i, r in enumerate(rows):
            p = r.params
            if r.greedy:
                tok: object = best[i]
            else:
                raw = logits[i].float().cpu()
                t = sample_token(apply_penalties(raw.clone(), r.out, p), p, r.generator)
                tok = token_logprobs(raw, t, p.logprobs) if p.logprobs >= 0 else t
            r.out.append(int(tok))
            events.append((r.rid, tok, r.finished))
            if r.finished:
                self._end(r)
            else:
                self.sched.prefill_done(r)
        for r, phase, _ in work:
            if phase == "prefill" and r.done < len(r.prompt):
                self.sched.prefill_more(r)
        self.stats["tokens"] += len(events)
        return events

    def _burst(self, reqs: list[Request]) -> list[tuple[int, object, bool]]:
        n = min([self.burst] + [r.limit - len(r.out) for r in reqs])
        toks = self.rt.decode_greedy([r.rid for r in reqs], [r.out[-1] for r in reqs], n)
        self.rt.check_status()
        events = []
        self.stats["burst_steps"] += n
        for i in range(n):                                        # step by step, as the requests would have produced them
            for r, row in zip(reqs, toks):
                if r.finished:
                    continue
                r.out.append(row[i])
                events.append((r.rid, row[i], r.finished))
        for r in reqs:
            if r.finished:
                self._end(r)
            else:
                self.sched.requeue_decode(r)
        self.stats["tokens"] += len(events)
        return events

    def run(self, prompts: Sequence[Sequence[int]], params: Sequence[SamplingParams]) -> list[list]:
        """All of these requests to their end; the generated tokens of each."""
        ids = [self.submit(p, q) for p, q in zip(prompts, params)]
        got: dict[int, list] = {i: [] for i in ids}
        left = set(ids)
        while left:
            for rid, tok, fin in self.step():
                if rid in got:
                    got[rid].append(tok)
                    if fin:
                        left.discard(rid)
        return [got[i] for i in ids]
