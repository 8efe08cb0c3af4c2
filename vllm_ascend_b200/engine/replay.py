"""Replay of given token sequences: the caller decides which tokens of which requests form each step, and
reads logits instead of sampled tokens.  Steps run through the engine's own scheduler bookkeeping (block
pool, batch rows), model runner, caches and kernels."""
from __future__ import annotations

import numpy as np
import torch

from .request import Request, SamplingParams


class TraceReplayer:
    def __init__(self, llm):
        self.llm = llm
        self.scheduler = llm.engine.scheduler
        self.runner = llm.engine.runner
        self.live: dict[str, Request] = {}

    def step(self, entries: list[dict], end: list[str]):
        """``entries``: [{"id", "tokens", "want"}], one per request of this step: its next tokens and the
        places among them whose logits are asked for.  ``end``: requests that are over after the step.
        Returns fp32 logits [wanted, vocab] in the order of the entries and of their places, or None."""
        portions, want = [], {}
        if len({e["id"] for e in entries}) != len(entries):
            raise ValueError("a step lists a request twice")
        for e in entries:
            tokens = np.asarray(e["tokens"], dtype=np.int32)
            if tokens.size == 0:
                raise ValueError(f"request {e['id']}: a portion holds at least one token")
            if tokens.min() < 0 or tokens.max() >= self.llm.cfg.model.vocab_size:
                raise ValueError(f"request {e['id']}: token id outside the vocabulary")
            if any(not 0 <= int(k) < tokens.size for k in e["want"]):
                raise ValueError(f"request {e['id']}: wanted place outside the portion")
            req = self.live.get(e["id"])
            if req is None:
                req = Request(e["id"], tokens, SamplingParams(max_tokens=1, temperature=0.0))
                self.live[e["id"]] = req
            else:
                self.runner.append_tokens(req, tokens)
                req.prompt_token_ids = np.concatenate([req.prompt_token_ids, tokens])
            portions.append((req, int(tokens.size)))
            want[e["id"]] = [int(k) for k in e["want"]]
        logits = None
        if portions:
            so = self.scheduler.schedule_portions(portions)
            at, first = 0, {}
            for req, n in so.scheduled:
                first[req.request_id] = at
                at += n
            rows = [first[e["id"]] + k for e in entries for k in want[e["id"]]]
            logits = self.runner.execute_logits(so, rows)
            self.scheduler.update_from_output(so, {})
        for rid in end:
            req = self.live.pop(rid, None)
            if req is not None:
                if req.row >= 0:             # the id may come back with other tokens
                    self.runner.row_owner[req.row] = None
                self.scheduler.abort_request(rid)
                self.scheduler.requests.pop(rid, None)
        return logits


def make_replay_engine(model: str, dtype: str, max_tokens: int, max_requests: int = 4, page: int = 64,
                       device: str = "cuda"):
    """Engine whose cache pool holds ``max_tokens`` tokens (in pages) and whose batch has ``max_requests``
    rows."""
    from .llm import LLM
    pages = (max_tokens + page - 1) // page
    if dtype == "float32" and device == "cuda":
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
        torch.set_float32_matmul_precision("highest")
    return LLM(model, dtype=dtype, device=device, block_size=page, max_model_len=pages * page,
               max_num_seqs=max_requests, max_num_batched_tokens=pages * page, num_gpu_blocks_override=pages + 1,
               cudagraph_capture_sizes=[s for s in (1, 2, 4, 8) if s <= max_requests])
