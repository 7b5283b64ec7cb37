"""Requests over an engine's cache slots: admission, mixed steps, release, and a continuous-batching greedy loop.

:class:`RequestScheduler` gives every live request one cache slot and the pages its tokens need.  A step takes the next tokens
of any subset of the live requests - portions of prompts beside single decoded tokens - and runs them as one batch through
:meth:`DecoderEngine.run_step`; a finished request returns its slot and pages.  :meth:`generate` drives the same steps from
prompts: waiting requests are admitted while slots and pages last, decoding requests contribute one token per step, and what is
left of the step's token budget goes to prompt portions.
"""
from __future__ import annotations

from collections import deque
from typing import Deque, Dict, Hashable, List, Optional, Sequence, Tuple

import torch

from .errors import RPUBackendError
from .kv_cache import PAGE_TOKENS


class RequestScheduler:
    def __init__(self, engine, *, token_budget: Optional[int] = None):
        self.engine = engine
        self.budget = min(token_budget or engine.max_tokens, engine.max_tokens)
        self.slots: Dict[Hashable, int] = {}
        self._free: List[int] = list(range(engine.cache.batch_size))[::-1]
        for s in range(engine.cache.batch_size):
            engine.cache.release(s)

    # -- live requests ----------------------------------------------------------------------------
    def admit(self, request: Hashable) -> int:
        """Slot of ``request``, taking a free one at its first appearance."""
        if request not in self.slots:
            if not self._free:
                raise RPUBackendError(f"request {request!r}: all {self.engine.cache.batch_size} cache slots are taken")
            self.slots[request] = self._free.pop()
        return self.slots[request]

    def finish(self, request: Hashable) -> None:
        """Give the slot and pages of a live request back."""
        if request not in self.slots:
            raise RPUBackendError(f"request {request!r} is not live")
        slot = self.slots.pop(request)
        self.engine.cache.release(slot)
        self._free.append(slot)

    def length(self, request: Hashable) -> int:
        return int(self.engine.cache.lengths[self.slots[request]])

    def step(self, entries: Sequence[Tuple[Hashable, torch.Tensor, Sequence[int]]]):
        """Run ``(request, next tokens, rows whose logits are wanted)`` entries as one batch; returns
        ``(next token per entry [n] int32 on the device, logits per entry [wanted, vocab])``."""
        return self.engine.run_step([t for _, t, _ in entries], [self.admit(r) for r, _, _ in entries], [w for _, _, w in entries])

    # -- continuous batching ------------------------------------------------------------------------
    def _pages(self, tokens: int) -> int:
        return (tokens + PAGE_TOKENS - 1) // PAGE_TOKENS

    def generate(self, prompts: Sequence[torch.Tensor], max_new_tokens: int, *, eos_token_id: Optional[int] = None) -> List[List[int]]:
        """Greedy continuation of every prompt (1-D token ids of any lengths, more of them than slots if need be)."""
        if max_new_tokens < 1:
            raise RPUBackendError("max_new_tokens must be a positive integer")
        if self.slots:
            raise RPUBackendError("generate() needs an idle scheduler")
        cache = self.engine.cache
        prompts = [torch.as_tensor(p).reshape(-1).to("cpu", torch.int32) for p in prompts]
        total = [int(p.numel()) + max_new_tokens - 1 for p in prompts]
        for i, n in enumerate(total):
            if not prompts[i].numel():
                raise RPUBackendError(f"prompt {i} is empty")
            if self._pages(n) > cache.num_pages or n > cache.max_seq_len:
                raise RPUBackendError(f"prompt {i} needs {n} cached tokens; the cache holds {cache.max_seq_len} per request and "
                                      f"{cache.num_pages * PAGE_TOKENS} in all")
        waiting: Deque[int] = deque(range(len(prompts)))
        running: List[int] = []
        done_rows = [0] * len(prompts)
        out: List[List[int]] = [[] for _ in prompts]
        free_pages = cache.num_pages
        try:
            while waiting or running:
                # a request is admitted only with room for its whole life, so that no step can run out of pages
                while waiting and self._free and len(running) < cache.batch_size and self._pages(total[waiting[0]]) <= free_pages:
                    i = waiting.popleft()
                    free_pages -= self._pages(total[i])
                    self.admit(i)
                    running.append(i)
                entries, room = [], self.budget
                for i in running:                       # decoding requests first: one token each
                    if done_rows[i] >= prompts[i].numel() and room > 0:
                        entries.append((i, torch.tensor([out[i][-1]], dtype=torch.int32), ()))
                        room -= 1
                for i in running:
                    left = int(prompts[i].numel()) - done_rows[i]
                    if left > 0 and room > 0:
                        take = min(left, room)
                        entries.append((i, prompts[i][done_rows[i]:done_rows[i] + take], ()))
                        room -= take
                nxt = self.step(entries)[0].tolist()
                for (i, toks, _), t in zip(entries, nxt):
                    if done_rows[i] < prompts[i].numel():
                        done_rows[i] += int(toks.numel())
                        if done_rows[i] < prompts[i].numel():
                            continue
                    out[i].append(t)
                    if len(out[i]) >= max_new_tokens or (eos_token_id is not None and t == eos_token_id):
                        self.finish(i)
                        running.remove(i)
                        free_pages += self._pages(total[i])
            self.engine.check_status()
        finally:
            for r in list(self.slots):
                self.finish(r)
        return out


__all__ = ["RequestScheduler"]
