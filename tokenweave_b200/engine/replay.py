"""Replays given steps through the engine: every step brings its tokens, nothing is sampled.

The replayer takes the scheduler's place. It admits requests, takes cache blocks and state slots from the engine
core's own manager, and hands the workers the same step messages the scheduler's decisions become, with two additions:
the tokens a request brings, and the places whose logits come back. Model, caches, batch layout and kernels are those
of generation. Used to compare a served model with recorded logits, and to reproduce a schedule exactly.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from ..sampling_params import SamplingParams
from ..worker.model_runner import NewRequestData, StepData
from .core import EngineCore
from .request import Request, RequestStatus


class StepReplayer:
    def __init__(self, core: EngineCore):
        self.core = core
        self.requests: dict[str, Request] = {}
        self._finished: list[str] = []
        self._step = 0

    def step(self, entries: Sequence[tuple], end: Sequence[str] = ()) -> Optional[torch.Tensor]:
        """``entries``: (request id, its next tokens, places among them whose logits are wanted), all one batch.
        ``end``: requests that are finished after this step. Returns fp32 logits ``[wanted, vocab]`` on the host, in
        the order of the entries and places, or None when nothing is wanted."""
        kv = self.core.kv
        vocab = self.core.config.model.vocab_size
        data = StepData(step_id=self._step, finished_req_ids=self._finished, given_tokens={}, want_logits={})
        self._finished = []
        self._step += 1
        for rid, tokens, want in entries:
            tokens = [int(t) for t in tokens]
            if not tokens or rid in data.want_logits:
                raise ValueError(f"request {rid}: one entry with at least one token per step")
            if any(t < 0 or t >= vocab for t in tokens):
                raise ValueError(f"request {rid}: token id outside [0, {vocab})")
            if any(w < 0 or w >= len(tokens) for w in want):
                raise ValueError(f"request {rid}: a wanted place outside its {len(tokens)} tokens")
            req = self.requests.get(rid)
            new = req is None
            if new:
                req = self.requests[rid] = Request(rid, [], SamplingParams(), status=RequestStatus.RUNNING)
            computed, held = req.num_computed_tokens, len(req.block_ids)
            if computed + len(tokens) > self.core.config.scheduler.max_model_len:
                raise ValueError(f"request {rid} grows beyond {self.core.config.scheduler.max_model_len} tokens")
            if not kv.allocate_slots(req, len(tokens)):
                raise RuntimeError(f"request {rid}: no cache block or state slot is free")
            req.prompt_token_ids.extend(tokens)
            if new:
                data.new_requests.append(NewRequestData(rid, list(tokens), len(tokens), req.sampling_params,
                                                        list(req.block_ids), None, req.state_slot))
            else:
                data.given_tokens[rid] = tokens
            data.scheduled.append((rid, computed, len(tokens), [] if new else list(req.block_ids[held:])))
            data.want_logits[rid] = list(want)
            data.total_num_tokens += len(tokens)
        result = self.core.executor.execute_model(data) if entries else None
        for rid, tokens, _ in entries:
            self.requests[rid].num_computed_tokens += len(tokens)
        for rid in end:
            kv.free(self.requests.pop(rid))
            self._finished.append(rid)
        return result.logits if result is not None else None
