"""Step-wise serving of one model: requests get a slot, bring portions of prompts or single tokens, and leave.

`StepRunner` owns the cache and the slots and runs one ragged batch per call; `BatchEngine` puts a scheduler with
chunked prefill and sampling on top of it.  Speculative rounds with a draft model are engine.py's.
"""

from __future__ import annotations

from collections import deque
from typing import Optional

import numpy as np

from . import sampling
from .model import DeviceLM


class StepRunner:
    """Live requests by name.  A request is admitted with its first entry and holds a slot (recurrent states) and, as it
    grows, pages of the cache until it is ended; both are used again."""

    def __init__(self, model: DeviceLM, max_batch: int, max_seq: int, pool_tokens: int = 0):
        self.model, self.ctx = model, model.ctx
        self.max_batch, self.max_seq = int(max_batch), int(max_seq)
        self.cache = (model.new_cache(self.max_batch, self.max_seq, pool_tokens=pool_tokens) if pool_tokens
                      else model.new_cache(self.max_batch, self.max_seq))
        self._slot: dict = {}
        self._free = deque(range(self.max_batch))
        self.length: dict = {}

    @property
    def live(self):
        return list(self._slot)

    @property
    def free_slots(self) -> int:
        return len(self._free)

    def step(self, entries):
        """entries: (name, tokens, want) triples, each request once; `want`: places among its tokens.  The whole step is
        one batch.  Returns the logits of the wanted places in order, a (n, vocab) device array, or None."""
        slots, counts, tokens, rows, r0 = [], [], [], [], 0
        names = [e[0] for e in entries]
        if len(set(names)) != len(names):
            raise ValueError("a request may bring one entry per step")
        if sum(n not in self._slot for n in names) > len(self._free):
            raise RuntimeError(f"all {self.max_batch} slots are in use")
        for name, toks, want in entries:
            toks = np.asarray(toks, dtype=np.int64).reshape(-1)
            if toks.size == 0:
                raise ValueError(f"request {name!r} brings no tokens")
            if name not in self._slot:
                slot = self._free.popleft()
                self.cache.reset_seq(slot)
                self._slot[name], self.length[name] = slot, 0
            if any(w < 0 or w >= toks.size for w in want):
                raise IndexError(f"request {name!r}: wanted place outside its {toks.size} tokens")
            slots.append(self._slot[name])
            counts.append(toks.size)
            tokens.append(toks)
            rows += [r0 + int(w) for w in want]
            r0 += toks.size
        out = self.model.forward_ragged(self.cache, slots, counts, np.concatenate(tokens), rows)
        for name, n in zip(names, counts):
            self.length[name] += n
        return out

    def end(self, name):
        """The request is finished: its slot and pages are free again."""
        slot = self._slot.pop(name)
        del self.length[name]
        self.cache.reset_seq(slot)
        self._free.append(slot)


class BatchEngine(StepRunner):
    """Continuous batching: every step brings one token of each request that decodes and, within `step_tokens` rows in
    all, the next portions of the prompts that are not through yet."""

    def __init__(self, model: DeviceLM, max_batch: int, max_seq: int, pool_tokens: int = 0, step_tokens: int = 2048):
        super().__init__(model, max_batch, max_seq, pool_tokens)
        self.step_tokens = int(step_tokens)
        if self.step_tokens <= self.max_batch:
            raise ValueError("step_tokens must exceed max_batch")
        self.steps_run = 0

    def _plan(self, running, pos):
        """Entries of the next step: (request, first token, count)."""
        plan = [(r, p, 1) for r, p in pos.items() if p >= len(running[r]) - 1]
        budget = self.step_tokens - len(plan)
        for r, p in pos.items():
            left = len(running[r]) - p
            if left > 1 and budget > 0:
                n = min(left, budget)
                plan.append((r, p, n))
                budget -= n
        return plan

    def run(self, prompts, max_new_tokens, temperature: float = 0.0, top_k: int = 0, eos_id: Optional[int] = None, seed: int = 0):
        """Serve `prompts` (1-D token arrays, any number); returns each request's new tokens (EOS included), in order.
        `max_new_tokens`: an int, or one per request.  With a page pool a request is admitted when its pages for the
        prompt and all its new tokens are free beside those promised to the running ones."""
        seqs = [[int(t) for t in np.asarray(p).reshape(-1)] for p in prompts]
        n_prompt = [len(s) for s in seqs]
        limits = [int(max_new_tokens)] * len(seqs) if np.isscalar(max_new_tokens) else [int(x) for x in max_new_tokens]
        if len(limits) != len(seqs):
            raise ValueError("one max_new_tokens per request")
        if any(n < 1 for n in n_prompt):
            raise ValueError("a request needs at least one prompt token")
        for n, lim in zip(n_prompt, limits):
            if n + max(lim, 1) - 1 > self.max_seq:
                raise RuntimeError(f"a request of {n} + {lim} tokens does not fit the cache's {self.max_seq} positions")
        pages = self._page_need(n_prompt, limits)
        waiting = deque(i for i in range(len(seqs)) if limits[i] > 0)
        pos: dict = {}
        promised = 0
        total = self.cache.pages[0] if pages else 0
        while waiting or pos:
            while waiting and len(pos) < self.max_batch and (not pages or promised + pages[waiting[0]] <= total):
                i = waiting.popleft()
                pos[i] = 0
                promised += pages[i] if pages else 0
            if not pos:
                raise RuntimeError(f"request {waiting[0]} needs more pages than the pool of {total} has")
            plan = self._plan(seqs, pos)
            entries, sampled = [], []
            for r, p, n in plan:
                done = p + n == len(seqs[r])
                entries.append((("run", r), seqs[r][p:p + n], [n - 1] if done else []))
                pos[r] = p + n
                if done:
                    sampled.append(r)
            logits = self.step(entries)
            self.steps_run += 1
            if not sampled:
                continue
            toks = (sampling.argmax(self.ctx, logits) if temperature <= 0 else
                    sampling.sample(self.ctx, logits, temperature=temperature, top_k=top_k, seed=seed, offset=self.steps_run)).numpy()
            for r, t in zip(sampled, toks):
                seqs[r].append(int(t))
                if len(seqs[r]) - n_prompt[r] >= limits[r] or (eos_id is not None and int(t) == eos_id):
                    self.end(("run", r))
                    del pos[r]
                    promised -= pages[r] if pages else 0
        self.model.check()
        return [np.asarray(s[n:], dtype=np.int64) for s, n in zip(seqs, n_prompt)]

    def _page_need(self, n_prompt, limits):
        """Pages each request may come to hold, or None for a cache without a pool."""
        try:
            total, free = self.cache.pages
        except NotImplementedError:
            return None
        if total >= self.max_batch * -(-self.max_seq // 64):
            return None
        return [-(-(n + max(lim, 1) - 1) // 64) for n, lim in zip(n_prompt, limits)]
