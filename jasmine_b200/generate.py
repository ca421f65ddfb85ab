"""Generation by continuous batching, for every registered model: prompts wait until a batch row and cache pages are free,
join the running batch between two steps, and leave it when they are done.

The scheduler only uses the calls all models share (admit / step_active / retire / pool_state / pages_for).  A sequence is
admitted when the pages it can ever hold fit beside what the running sequences can ever hold, so that no step runs out of
pages.  Tokens are the arg-max of the logits, or drawn by the library's sampler (temperature, top-k, top-p)."""
from __future__ import annotations

import ctypes as C
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from . import JsmError, SHAPE, check, lib


@dataclass
class Request:
    prompt: list
    max_new: int
    stop: frozenset = frozenset()
    tokens: list = field(default_factory=list)  # generated so far

    def done(self) -> bool:
        return len(self.tokens) >= self.max_new or bool(self.tokens and self.tokens[-1] in self.stop)


class Sampler:
    """Draws from logits in host memory with jsm_sample; temperature 0 = arg-max (no sampler is needed then)."""

    def __init__(self, rows, vocab, temperature, top_k=0, top_p=1.0, seed=0):
        self.vocab, self.args, self.seed, self.draws = vocab, (temperature, top_k, top_p), seed, 0
        self._logits, self._out = C.c_void_p(), C.c_void_p()
        check(lib().jsm_malloc(C.byref(self._logits), rows * vocab * 4))
        check(lib().jsm_malloc(C.byref(self._out), rows * 4))

    def __call__(self, logits) -> np.ndarray:
        n = logits.shape[0]
        out = np.empty(n, np.int32)
        check(lib().jsm_upload(self._logits, logits.ctypes.data, n * self.vocab * 4, None))
        check(lib().jsm_sample(self._logits, self.vocab, n, self.vocab, *self.args, self.seed, self.draws, self._out, None))
        check(lib().jsm_download(out.ctypes.data, self._out, n * 4, None))
        self.draws += 1
        return out

    def close(self):
        lib().jsm_free(self._logits)
        lib().jsm_free(self._out)


def generate(model, prompts, max_new, temperature=0.0, top_k=0, top_p=1.0, seed=0, stop=()):
    """Generated tokens of every prompt (lists of token ids), in the order of the prompts."""
    max_new = [max_new] * len(prompts) if isinstance(max_new, int) else list(max_new)
    reqs = [Request(list(p), n, frozenset(stop)) for p, n in zip(prompts, max_new)]
    for r in reqs:
        if len(r.prompt) + r.max_new > model.max_context:
            raise JsmError(SHAPE, f"a prompt of {len(r.prompt)} tokens and {r.max_new} new ones exceed the context of {model.max_context}")
        if model.pages_for(len(r.prompt) + r.max_new) > model.pool_state()[2]:
            raise JsmError(SHAPE, f"a sequence of {len(r.prompt) + r.max_new} tokens exceeds the page pool")
    waiting, rows = deque(r for r in reqs if r.max_new > 0), []
    sampler = Sampler(model.max_batch, model.vocab, temperature, top_k, top_p, seed) if temperature > 0 else None
    held = lambda r: model.pages_for(len(r.prompt) + r.max_new)
    try:
        with model.stream_scope():
            total = model.pool_state()[2]
            last = np.empty((1, model.vocab), np.float32) if sampler else None
            while waiting or rows:
                while waiting and len(rows) < model.max_batch and sum(map(held, rows)) + held(waiting[0]) <= total:
                    r = waiting.popleft()
                    row, tok = model.admit(np.asarray(r.prompt, np.int32), last)
                    assert row == len(rows)
                    r.tokens.append(int(sampler(last)[0]) if sampler else tok)
                    rows.append(r)
                for i in reversed(range(len(rows))):
                    if rows[i].done():
                        moved = model.retire(i)
                        gone = rows.pop()
                        if moved >= 0:
                            rows[i] = gone
                if not rows:
                    continue
                ids = np.asarray([r.tokens[-1] for r in rows], np.int32)
                nxt = np.empty(len(rows), np.int32)
                logits = np.empty((len(rows), model.vocab), np.float32) if sampler else None
                model.step_active(ids, nxt, logits)
                if sampler:
                    nxt = sampler(logits)
                for r, t in zip(rows, nxt):
                    r.tokens.append(int(t))
    finally:
        if sampler:
            sampler.close()
    return [r.tokens for r in reqs]
