"""Steps whose batches and tokens come from outside: replay of token traces through the engine's own parts.

``ImposedSession`` feeds given token ids through an engine step by step and reads logits; nothing is sampled.  Requests,
pages and slots are the scheduler's (``ContinuousScheduler.imposed_plan`` reserves them, ``release`` gives them back),
the step is the executor's (``GpuExecutor.execute_logits``).  All entries of a step run as one batch: portions of prompts
beside single decoded tokens.
"""
from __future__ import annotations

import numpy as np

from ..executor.gpu_executor import Segment
from .scheduler import Request, SamplingParams


class ImposedSession:
    def __init__(self, engine) -> None:
        if engine.prefix.enabled:
            raise ValueError("a session of imposed steps runs without the prefix cache: every step computes its tokens")
        self.engine = engine
        self.vocab = engine.executor.cfg.vocab_size

    def step(self, entries: list[tuple[str, list[int], list[int]]]) -> list[np.ndarray]:
        """``entries``: (request id, its next tokens, places among them whose logits are wanted).  Returns the fp32 logits
        ``[wanted, vocab]`` of every entry."""
        eng = self.engine
        batch = []
        if len({rid for rid, _, _ in entries}) != len(entries):
            raise ValueError("a request has one entry in a step")
        for rid, tokens, want in entries:
            tokens = [int(t) for t in tokens]
            if not tokens or min(tokens) < 0 or max(tokens) >= self.vocab:
                raise ValueError(f"request {rid}: an entry has at least one token and ids in [0, {self.vocab})")
            if any(not 0 <= int(w) < len(tokens) for w in want):
                raise ValueError(f"request {rid}: a wanted place is not among the entry's tokens")
            r = eng.requests.get(rid)
            if r is None:
                r = eng.requests[rid] = Request(rid, tokens, SamplingParams())
            else:
                r.tokens.extend(tokens)
            batch.append((r, len(tokens)))
        plan = eng.scheduler.imposed_plan(batch)
        segs = [Segment(s.request.slot, s.request.tokens[s.start:s.start + s.count], s.start, s.request.pages, sample=False,
                        uid=s.request.arrival << 16, logit_offsets=[int(w) for w in want])
                for s, (_, _, want) in zip(plan.segments, entries)]
        if plan.copies:
            eng.executor.copy_pages(plan.copies)
        out = eng.executor.execute_logits(segs)
        eng.scheduler.commit(plan, {})
        eng.steps += 1
        return out

    def end(self, request_ids) -> None:
        """Requests that are finished: what they hold is given back."""
        for rid in request_ids:
            r = self.engine.requests.pop(rid, None)
            if r is None:
                raise ValueError(f"request {rid} is not live")
            self.engine.scheduler.release(r)
