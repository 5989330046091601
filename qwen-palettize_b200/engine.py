"""Serving loop over any registered model: requests with their own state, a step that feeds one request's next tokens, a
first-come scheduler that cuts prompts into portions and interleaves decoding, and token sampling.

`Engine.step` is the only place that runs a model; generation (`submit` / `run` / `generate`) and trace replay both go through it.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field

import torch

import seq_ops as S
from seq_state import StatePool


@dataclass
class SamplingParams:
    max_new: int = 16
    temperature: float = 0.0     # 0: greedy
    top_k: int = 0               # 0: all tokens
    seed: int = 0
    stop: tuple = ()             # token ids that end the request (kept in the output)


@dataclass
class Request:
    rid: object
    prompt: list
    params: SamplingParams
    fed: int = 0                                   # prompt tokens already run
    out: list = field(default_factory=list)
    done: bool = False


class Engine:
    def __init__(self, model, max_tokens: int, portion: int = 2048, max_live: int = 8):
        """max_tokens: capacity of one request's state; portion: most prompt tokens a step runs; max_live: requests with a state at once."""
        if portion < 1 or max_live < 1:
            raise ValueError("portion and max_live must be positive")
        self.model, self.portion, self.max_live = model, portion, max_live
        self.pool = StatePool(model, max_tokens)
        self.waiting, self.live, self.finished = deque(), deque(), {}
        self._next = 0

    # ---- the step ----------------------------------------------------------------------------------------------------
    def step(self, rid, tokens, want=(), end: bool = False):
        """Feed `tokens` to request rid (a new id starts a sequence) and return the fp32 logits at the places `want` among them, or None.
        end: the request is finished after this step and its state goes back to the pool."""
        V = self.model.vocab
        for t in tokens:
            if not 0 <= t < V:
                raise ValueError(f"token {t} outside the vocabulary of {V}")
        for w in want:
            if not 0 <= w < len(tokens):
                raise ValueError(f"place {w} among {len(tokens)} tokens")
        st = self.pool.get(rid) if rid in self.pool else self.pool.acquire(rid)
        out = self.model.forward(torch.tensor([list(tokens)], dtype=torch.int64), st, list(want)) if len(tokens) else None
        if end:
            self.pool.release(rid)
        return out

    def end(self, rid):
        if rid in self.pool:
            self.pool.release(rid)

    # ---- generation ----------------------------------------------------------------------------------------------------
    def submit(self, prompt, params: SamplingParams | None = None):
        params = params or SamplingParams()
        if not prompt:
            raise ValueError("empty prompt")
        if len(prompt) + params.max_new > self.pool.capacity:
            raise ValueError(f"{len(prompt)} + {params.max_new} tokens exceed the capacity {self.pool.capacity}")
        rid = ("gen", self._next)
        self._next += 1
        self.waiting.append(Request(rid, list(prompt), params))
        return rid

    def schedule(self):
        """The request that the next step serves: requests are admitted in order while there is room, a prompt that has started is
        finished first, then the live requests decode in turn."""
        while self.waiting and len(self.live) < self.max_live:
            self.live.append(self.waiting.popleft())
        for r in self.live:
            if r.fed < len(r.prompt):
                return r
        return self.live[0] if self.live else None

    def run_one(self) -> bool:
        """One scheduled step; False when there is nothing left to do."""
        r = self.schedule()
        if r is None:
            return False
        if r.fed < len(r.prompt):
            part = r.prompt[r.fed:r.fed + self.portion]
            r.fed += len(part)
            logits = self.step(r.rid, part, [len(part) - 1] if r.fed == len(r.prompt) else ())
        else:
            logits = self.step(r.rid, [r.out[-1]], [0])
        if logits is not None and r.params.max_new > 0:
            self._take(r, logits)
        if r.done or (r.fed == len(r.prompt) and len(r.out) >= r.params.max_new):
            self.live.remove(r)
            self.end(r.rid)
            self.finished[r.rid] = r.out
        elif r.fed == len(r.prompt):
            self.live.remove(r)          # to the back: the others decode next
            self.live.append(r)
        return True

    def _take(self, r: Request, logits: torch.Tensor):
        p = r.params
        at = torch.tensor([r.fed + len(r.out)], dtype=torch.int32, device=logits.device)
        tok = int(S.sample(logits, at, p.temperature, p.top_k, p.seed).item())
        r.out.append(tok)
        r.done = tok in p.stop

    def run(self) -> dict:
        """Until every submitted request is finished: {request id: generated tokens} of all finished so far."""
        while self.run_one():
            pass
        return self.finished

    def generate(self, prompts, params: SamplingParams | None = None):
        """Generated tokens of every prompt, in order."""
        ids = [self.submit(p, params) for p in prompts]
        done = self.run()
        return [done.pop(i) for i in ids]
