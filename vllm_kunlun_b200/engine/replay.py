"""Replay of a prescribed schedule: given token ids run through the engine step by step, in given portions and batches,
and the logits at chosen places come back.  Everything below the choice of the batch is the engine's own - scheduler
bookkeeping, block pool, state slots, model runner, captured decode steps."""
from __future__ import annotations

from typing import Sequence

import torch

from .llm import LLM
from .request import Request, RequestStatus, SamplingParams


class ScheduleReplay:
    def __init__(self, model, dtype: str, max_tokens: int, max_requests: int = 4, block_size: int = 64, **kw):
        """``max_tokens``: the cache pool holds this many tokens (whole blocks) over all live requests."""
        blocks = -(-max_tokens // block_size)
        span = blocks * block_size
        self.llm = LLM(model, dtype=dtype, block_size=block_size, num_gpu_blocks=blocks, max_model_len=span,
                       max_num_seqs=max_requests, max_num_batched_tokens=span + max_requests, **kw)
        self.engine = self.llm.engine
        self.live: dict = {}

    def step(self, entries: Sequence[dict], end: Sequence[str] = ()) -> torch.Tensor:
        """``entries``: ``{"id", "tokens", "want"}`` per request, all of them one batch.  Returns fp32 logits on the
        host, one row per wanted place, in the order of the entries and of their ``want``.  Requests named in ``end``
        give back what they hold."""
        vocab = self.engine.cfg.model.vocab_size
        portions = []
        for e in entries:
            req = self.live.get(e["id"])
            if req is None:
                req = self.live[e["id"]] = Request(e["id"], [], SamplingParams(max_tokens=1))
            toks = [int(t) for t in e["tokens"]]
            if not toks or min(toks) < 0 or max(toks) >= vocab:
                raise ValueError(f"request {e['id']}: a portion needs tokens inside the vocabulary [0, {vocab})")
            rows = [int(w) for w in e.get("want", ())]
            if rows and (min(rows) < 0 or max(rows) >= len(toks)):
                raise ValueError(f"request {e['id']}: wanted places outside the portion")
            req.prompt_token_ids.extend(toks)
            portions.append((req, len(toks), rows))
        out = torch.empty(0, vocab)
        if portions:
            sched = self.engine.scheduler.schedule_portions(portions)
            handle = self.engine.runner.execute(sched)
            handle.wait()
            by_req, row = {}, 0
            for sr in sched.scheduled:
                n = len(sr.logit_rows)
                by_req[sr.req.request_id] = handle.logits[row:row + n]
                row += n
            out = torch.cat([by_req[req.request_id] for req, _, _ in portions])
        for rid in end:
            req = self.live.pop(rid)
            req.status = RequestStatus.FINISHED_STOPPED
            self.engine.scheduler.finish(req)
        return out
