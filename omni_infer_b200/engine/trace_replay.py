"""Replay of a given token trace through the engine's own step: the caller decides which tokens of which requests make up
every step and which rows' logits it wants; nothing is sampled.

Requests hold pages and state slots of the engine's block manager and every step is one ``execute_model`` call of the
engine's runner, so a replay runs what generation runs: a step in which every request brings one token is a decode step
(with its CUDA graph), any other is a ragged batch of portions."""
from __future__ import annotations

from typing import Optional

import torch

from .engine_core import EngineCore
from .request import Request, ScheduledRequest, SchedulerOutput


class TraceReplay:
    def __init__(self, engine: EngineCore):
        self.engine = engine
        self.live: dict = {}

    def step(self, entries: list, end=()) -> Optional[torch.Tensor]:
        """``entries``: dicts ``{"id", "tokens", "want"}``; ``end``: ids that are finished after this step.  Returns the
        logits [rows wanted, vocab] (fp32, CPU) in the order of the entries and their ``want``, None if nothing is wanted."""
        eng, vocab = self.engine, self.engine.model_cfg.vocab_size
        scheduled = []
        for e in entries:
            toks = [int(t) for t in e["tokens"]]
            want = [int(w) for w in e.get("want") or ()]
            if not toks or min(toks) < 0 or max(toks) >= vocab:
                raise ValueError(f"request {e['id']}: tokens must be a non-empty list of ids in [0, {vocab})")
            if want and not (0 <= min(want) and max(want) < len(toks)):
                raise ValueError(f"request {e['id']}: rows wanted lie outside its tokens")
            req = self.live.get(e["id"])
            if req is None:
                if len(self.live) >= eng.cfg.max_num_seqs:
                    raise RuntimeError(f"more than {eng.cfg.max_num_seqs} live requests")
                req = self.live[e["id"]] = Request(str(e["id"]), [])
            if req.num_computed_tokens + len(toks) > eng.cfg.max_model_len:
                raise RuntimeError(f"request {e['id']} outgrows the context of {eng.cfg.max_model_len} tokens")
            req.prompt_token_ids.extend(toks)
            if eng.kv.allocate_slots(req, len(toks)) is None:
                raise RuntimeError("the cache pool is exhausted")
            scheduled.append(ScheduledRequest(req, len(toks), True, want_logits=want))
        logits = None
        if scheduled:
            total = sum(s.num_scheduled_tokens for s in scheduled)
            single = total == len(scheduled)
            for s in scheduled:
                s.is_prefill = not single
            out = eng.worker.execute_model(SchedulerOutput(scheduled, not single, 1, total))
            logits = out.logits.float().cpu() if out.logits is not None else None
            for s in scheduled:
                s.request.num_computed_tokens += s.num_scheduled_tokens
        for rid in end:
            self.engine.kv.free(self.live.pop(rid))
        return logits
