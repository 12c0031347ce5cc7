"""Replay policy: the caller says which requests run how many tokens in the next step.

Admission, block allocation and the life cycle of a request are the scheduler's own; only the choice that a
serving policy makes (who runs, in which portions) comes from outside.  Used by ``engine/replay.py``."""
from __future__ import annotations

from ..engine.request import RequestStatus
from ..engine.scheduler import Scheduler, SchedulerOutput


class ReplayScheduler(Scheduler):
    def __init__(self, *a, **kw):
        super().__init__(*a, **kw)
        if self.async_mode or self.kv.pool.enable_caching or self.connector is not None:
            raise ValueError("a replay runs synchronously, without prefix caching and without a KV connector")
        self.plan: list = []            # (request id, number of tokens) of the next step, in batch order

    def schedule(self) -> SchedulerOutput:
        scheduled = []
        plan, self.plan = self.plan, []
        for rid, n in plan:
            req = self.requests[rid]
            if req.num_computed_tokens + n > req.num_tokens:
                raise ValueError(f"request {rid}: the step runs tokens that were not given")
            if req in self.waiting:
                if len(self.running) >= self.cfg.max_num_seqs:
                    raise RuntimeError(f"request {rid}: {self.cfg.max_num_seqs} requests are live already")
                self.waiting.remove(req)
                req.status = RequestStatus.RUNNING
                self.running.append(req)
            first = req.request_id not in self._in_batch
            new_blocks = self.kv.allocate_slots(req, n)
            if new_blocks is None:
                raise RuntimeError(f"request {rid}: the KV pool of {self.kv.pool.num_blocks - 1} blocks is full")
            scheduled.append(self._make_sched(req, n, list(req.block_ids) if first else new_blocks))
        total = sum(s.num_new_tokens for s in scheduled)
        if total > self.cfg.max_num_batched_tokens:
            raise RuntimeError(f"step of {total} tokens exceeds max_num_batched_tokens {self.cfg.max_num_batched_tokens}")
        self.stats["scheduled_tokens"] += total
        out = SchedulerOutput(self.step_id, scheduled, self.finished_since_last, [], total)
        self.finished_since_last = []
        self.step_id += 1
        self._update_after_schedule(out)
        return out

    def finish(self, rid: str) -> None:
        """Give back what the request holds; its id may be used again."""
        req = self.requests.pop(rid)
        self._finish(req, RequestStatus.FINISHED_STOPPED)
