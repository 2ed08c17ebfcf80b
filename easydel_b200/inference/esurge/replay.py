"""Teacher-forced replay: steps whose tokens and batch composition are given instead of scheduled and sampled.

:class:`TraceReplayer` drives an :class:`.engine.eSurge` step by step: every entry of a step names a request and its next
tokens, the whole step runs as one batch through the engine's own page pools, state slots and model runner, and the
logits of the asked-for places come back. Requests take pages and a slot at their first entry and give them back when
they end. Useful to compare the serving path with another implementation, or to reproduce a recorded schedule.
"""

from __future__ import annotations

import typing as tp

import torch

from ..sampling_params import SamplingParams
from .scheduler import EngineRequest, RequestStatus, ScheduledRequest, SchedulerOutput


def engine_limits(max_tokens: int, max_requests: int, page_size: int, granule: int = 64) -> dict[str, int]:
    """Engine sizes for requests that never hold more than ``max_tokens`` tokens together, each request's count rounded
    up to a multiple of ``granule``: the page pool covers those tokens in pages of ``page_size`` (each request can waste
    up to ``page_size - granule`` more than the rounded count) plus the null page."""
    pages = -(-(max_tokens + max_requests * max(0, page_size - granule)) // page_size)
    return {"num_pages": pages + 1, "max_num_seqs": max_requests, "max_model_len": -(-max_tokens // page_size) * page_size,
            "max_num_batched_tokens": max(max_tokens, max_requests)}


class TraceReplayer:
    def __init__(self, engine):
        if engine.scheduler.has_unfinished():
            raise RuntimeError("the engine is serving requests")
        self.engine = engine
        self.requests: dict[str, EngineRequest] = {}

    def _request(self, rid: str) -> EngineRequest:
        req = self.requests.get(rid)
        if req is None:
            sch = self.engine.scheduler
            if sch.num_running >= sch.config.max_num_seqs:
                raise RuntimeError(f"request {rid!r}: all {sch.config.max_num_seqs} state slots are taken")
            req = EngineRequest(rid, [], SamplingParams(max_tokens=None, temperature=0.0))
            sch.requests[rid] = req
            req.status = RequestStatus.RUNNING
            sch.running.append(req)
            self.requests[rid] = req
        return req

    def step(self, entries: tp.Sequence[dict], end: tp.Sequence[str] = ()) -> torch.Tensor | None:
        """``entries``: ``{"id", "tokens", "want"}``; returns fp32 logits ``[wanted, vocab]`` in the order of the entries
        and of their ``want`` lists (None when nothing is wanted). ``end``: requests that are finished after the step."""
        eng = self.engine
        sched, wants = [], []
        for e in entries:
            tokens = [int(t) for t in e["tokens"]]
            if not tokens:
                raise ValueError(f"request {e['id']!r}: an entry without tokens")
            req = self._request(e["id"])
            start = req.num_computed_tokens
            req.prompt_token_ids.extend(tokens)
            if not eng.scheduler._try_allocate(req, start + len(tokens)):
                raise RuntimeError(f"request {e['id']!r}: no free page for {start + len(tokens)} tokens")
            sched.append(ScheduledRequest(req, len(tokens), start, False))
            wants.append([int(w) for w in e.get("want") or ()])
        logits = None
        if sched:
            # the scheduler's own order: single-token rows lead the batch
            order = sorted(range(len(sched)), key=lambda i: (sched[i].num_new_tokens > 1, sched[i].request.order))
            out = SchedulerOutput([sched[i] for i in order], [], sum(s.num_new_tokens for s in sched),
                                  sum(1 for s in sched if s.num_new_tokens == 1))
            first, at = {}, 0
            for i in order:
                first[i] = at
                at += sched[i].num_new_tokens
            eng._assign_slots(out)
            logits = eng.runner.step_logits(out, [first[i] + w for i, ws in enumerate(wants) for w in ws])
            for s in sched:
                s.request.num_computed_tokens += s.num_new_tokens
        for rid in end:
            req = self.requests.pop(rid)
            eng.scheduler.finish_request(req, RequestStatus.FINISHED_STOPPED)
            eng._return_slot(req)
        return logits
