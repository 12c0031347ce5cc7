"""Step-by-step replay of given tokens through an engine, with the logits of chosen positions.

Nothing is sampled into the sequences: every token comes from the caller.  The steps run through the engine's
scheduler bookkeeping, cache, batch preparation, CUDA graphs and kernels like generated ones."""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from ..sampling_params import SamplingParams
from .llm_engine import LLMEngine
from .request import Request


class TraceReplay:
    def __init__(self, engine: LLMEngine):
        from ..schedulers.replay import ReplayScheduler
        if not isinstance(engine.scheduler, ReplayScheduler):
            raise ValueError("replay needs an engine with scheduler_cls='replay'")
        self.engine = engine

    def step(self, entries: Sequence, end: Sequence = ()) -> Optional[torch.Tensor]:
        """One batch.  entries: (request id, its next tokens, places among them whose logits are wanted); end: ids
        of requests that are finished after the step.  Returns [wanted, vocab] fp32 on the host in the order of the
        entries, None when nothing is wanted."""
        sch, runner = self.engine.scheduler, self.engine.runner
        want = {}
        for rid, tokens, places in entries:
            if not tokens:
                raise ValueError(f"request {rid}: an entry without tokens")
            if rid in want:
                raise ValueError(f"request {rid} appears twice in one step")
            req = sch.requests.get(rid)
            if req is None:
                sch.add_request(Request(rid, list(tokens), SamplingParams(temperature=0.0, max_tokens=1)))
            else:
                req.prompt_token_ids.extend(tokens)
                for t in tokens:
                    runner.batch.append_token(runner.batch.slot_of[rid], t)
            sch.plan.append((rid, len(tokens)))
            want[rid] = list(places)
        rows = None
        if want:
            out = sch.schedule()
            out.logit_places = want
            res = runner.execute_model(out)
            res.get()
            if res.place_logits:
                rows = torch.cat([res.place_logits[rid] for rid, _, _ in entries if rid in res.place_logits])
        for rid in end:
            sch.finish(rid)
        return rows
