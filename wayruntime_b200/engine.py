"""Serving loop over a device model of either kind: sessions, portions of prompts, decode batches, sampling.

The unit of work is `Engine.advance`: some sessions take their next tokens, from the cache and state that earlier
steps left.  Sessions with one token each go through one decode pass per WR_BATCH_MAX sessions
(include/wayruntime/wayruntime.h:423); a session with more goes through prefill passes of at most the model's
max_rows rows.  `Engine.step` schedules queued requests on top of it: one portion of a waiting prompt, then one
decode pass over the running requests.
"""
from __future__ import annotations

import itertools
from collections import deque
from dataclasses import dataclass, field

import numpy as np

from .binding import BATCH_MAX


@dataclass
class Sampling:
    """temperature 0: greedy (the lowest id wins a tie, as the reference's arg-max does, src/cli/wayrt.c:805)."""
    temperature: float = 0.0
    top_k: int = 0
    top_p: float = 1.0
    seed: int = 0


class Session:
    """One sequence: its cache and how many tokens it holds."""

    def __init__(self, model, max_ctx: int):
        self.kv = model.kv_create(max_ctx)
        self.max_ctx, self.pos = max_ctx, 0

    def close(self):
        self.kv.close()


@dataclass
class Request:
    prompt: list
    max_new: int
    sampling: Sampling = field(default_factory=Sampling)
    stop: frozenset = frozenset()
    id: int = 0
    output: list = field(default_factory=list)
    done: bool = False
    session: Session | None = None
    _rng: object = None


def sample(logits: np.ndarray, s: Sampling, rng) -> int:
    """One token id from a row of logits."""
    if s.temperature <= 0:
        return int(np.argmax(logits))
    z = logits.astype(np.float64) / s.temperature
    order = np.argsort(-z, kind="stable")
    if s.top_k > 0:
        order = order[:s.top_k]
    p = np.exp(z[order] - z[order[0]])
    p /= p.sum()
    if s.top_p < 1.0:
        keep = int(np.searchsorted(np.cumsum(p), s.top_p) + 1)
        order, p = order[:keep], p[:keep] / p[:keep].sum()
    return int(order[np.searchsorted(np.cumsum(p), rng.random() * p.sum(), side="right").clip(0, len(p) - 1)])


class Engine:
    def __init__(self, model, max_sessions: int = BATCH_MAX, portion: int | None = None):
        self.model = model
        self.max_sessions = max_sessions
        self.portion = min(portion or model.max_rows, model.max_rows)
        self.waiting, self.running = deque(), []
        self._ids = itertools.count()

    # ---- the step function

    def session(self, max_ctx: int) -> Session:
        return Session(self.model, max_ctx)

    def advance(self, sessions, tokens, want=None, argmax=False):
        """Run tokens[i] (a list of ids) on sessions[i].  want[i]: places among them whose logits are returned,
        default the last one; the result is one array [len(want[i]), vocab] per session — or, with argmax, the id of
        the first maximum after each session's last token."""
        want = [[len(t) - 1] for t in tokens] if want is None else want
        out = [None] * len(sessions)
        single = [i for i, t in enumerate(tokens) if len(t) == 1]
        for lo in range(0, len(single), BATCH_MAX):
            self._decode(single[lo:lo + BATCH_MAX], sessions, tokens, want, argmax, out)
        for i, t in enumerate(tokens):
            if len(t) > 1:
                out[i] = self._prefill(sessions[i], t, want[i], argmax)
        return out

    def _decode(self, rows, sessions, tokens, want, argmax, out):
        m = self.model
        asked = [j for j, i in enumerate(rows) if len(want[i])]
        res = m.forward(m.FWD_DECODE, [sessions[i].kv for i in rows], [sessions[i].pos for i in rows],
                        [tokens[i][0] for i in rows], logits=False if argmax else asked, argmax=argmax)
        for j, i in enumerate(rows):
            sessions[i].pos += 1
            if argmax:
                out[i] = int(res["argmax"][j])
            elif j in asked:
                out[i] = res["logits"][asked.index(j)][None, :].repeat(len(want[i]), axis=0)
            else:
                out[i] = np.empty((0, m.vocab), np.float32)

    def _prefill(self, s, tokens, want, argmax):
        m, parts = self.model, []
        rows_max = m.max_rows
        order = sorted(set(want))                    # (asked in any order, computed front to back, each once)
        for lo in range(0, len(tokens), rows_max):
            part = tokens[lo:lo + rows_max]
            last = lo + len(part) == len(tokens)
            here = [w - lo for w in order if lo <= w < lo + len(part)]
            if argmax:
                res = m.forward(m.FWD_PREFILL, [s.kv], [s.pos], part, out_from=len(part) - 1, argmax=last)
            elif here:
                first = here[0]
                res = m.forward(m.FWD_PREFILL, [s.kv], [s.pos], part, out_from=first, logits=[w - first for w in here])
                parts.append(res["logits"])
            else:
                res = m.forward(m.FWD_PREFILL, [s.kv], [s.pos], part, out_from=len(part))
            s.pos += len(part)
        if argmax:
            return int(res["argmax"][0])
        if not parts:
            return np.empty((0, m.vocab), np.float32)
        rows = np.concatenate(parts)
        return rows if order == list(want) else rows[[order.index(w) for w in want]]

    # ---- scheduling

    def submit(self, request: Request) -> Request:
        if not request.prompt:
            raise ValueError("a request needs at least one prompt token")
        request.id = next(self._ids)
        request._rng = np.random.default_rng(request.sampling.seed)
        self.waiting.append(request)
        return request

    def step(self) -> list:
        """One portion of the first waiting prompt (when a session is free), then one token for every running
        request; returns the requests that finished."""
        if self.waiting and len(self.running) < self.max_sessions:
            r = self.waiting[0]
            if r.session is None:
                r.session = self.session(len(r.prompt) + r.max_new)
            s = r.session
            part = r.prompt[s.pos:s.pos + self.portion]
            if s.pos + len(part) < len(r.prompt):
                self.advance([s], [part], [[]])
            else:
                self.waiting.popleft()
                self.running.append(r)
                self._take(r, self._next([r], [part])[0])
        ready = [r for r in self.running if not r.done]
        if ready:
            for r, t in zip(ready, self._next(ready, [[r.output[-1]] for r in ready])):
                self._take(r, t)
        finished = [r for r in self.running if r.done]
        self.running = [r for r in self.running if not r.done]
        for r in finished:
            r.session.close()
            r.session = None
        return finished

    def _next(self, reqs, tokens):
        sessions = [r.session for r in reqs]
        if all(r.sampling.temperature <= 0 for r in reqs):
            return self.advance(sessions, tokens, argmax=True)
        rows = self.advance(sessions, tokens)
        return [sample(row[-1], r.sampling, r._rng) for r, row in zip(reqs, rows)]

    def _take(self, r, token):
        r.output.append(token)
        if len(r.output) >= r.max_new or token in r.stop:
            r.done = True

    def run(self, requests) -> list:
        """Submit, step until all are done, return the requests."""
        for r in requests:
            self.submit(r)
        while self.waiting or self.running:
            self.step()
        return requests
