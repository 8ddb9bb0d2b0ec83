"""Requests over an engine's sequence slots: admission, mixed batches, reclaim.

Session maps request names to slots of a cache with a shared page pool and runs one batch per call (hm_step).
Scheduler drives a Session to completion for a list of prompts: long prompts go in portions beside the single
tokens of the requests that are already generating, finished requests give their slot and pages to waiting ones.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import numpy as np

from . import DType, HfModel, KvCacheFull, SamplingConfig, sample_token_device


class Session:
    """`slots` live requests at most, together at most `pool_tokens` tokens (each request rounded up to whole pages)."""

    def __init__(self, model: HfModel, slots: int, pool_tokens: int, kv_dtype: DType = DType.BF16, max_seq_len: Optional[int] = None):
        self.model = model
        limit = model.config().max_position_embeddings
        model.init_kv_cache(min(max_seq_len or pool_tokens, limit), batch=slots, kv_dtype=kv_dtype, pool_tokens=pool_tokens)
        self._free = list(range(slots - 1, -1, -1))
        self._slot: Dict[Hashable, int] = {}

    def live(self) -> int:
        return len(self._slot)

    def free_slots(self) -> int:
        return len(self._free)

    def length(self, name: Hashable) -> int:
        return self.model.kv_cache_len(self._slot[name])

    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]], want_logits: bool = True, want_greedy: bool = False):
        """entries: (request, its next tokens, wanted places).  A request is admitted at its first entry.
        Returns (logits [wanted, vocab] or None, greedy ids or None) in the order of the entries."""
        new = [name for name, _, _ in entries if name not in self._slot]
        if len(new) > len(self._free):
            raise RuntimeError(f"{len(new)} new requests, {len(self._free)} free slots")
        for name in new:
            self._slot[name] = self._free.pop()
        try:
            logits, greedy, _ = self.model.step([(self._slot[name], tokens, want) for name, tokens, want in entries], want_logits, want_greedy)
        except Exception:
            for name in new:
                self.end(name)
            raise
        return logits, greedy

    def end(self, name: Hashable):
        """Gives the request's slot and pages back."""
        slot = self._slot.pop(name)
        self.model.reset_kv_cache(slot)
        self._free.append(slot)


@dataclass
class _Request:
    index: int
    prompt: List[int]
    max_new: int
    fed: int = 0
    out: List[int] = field(default_factory=list)
    rng: int = 1


class Scheduler:
    """Continuous batching over a Session.  `portion` bounds the prompt tokens of one request in one batch, `batch_tokens`
    the tokens of a batch."""

    def __init__(self, session: Session, portion: int = 256, batch_tokens: int = 512):
        self.session, self.portion, self.batch_tokens = session, portion, batch_tokens
        self.page = 64 if session.model.architecture() else 16

    def _pages(self, r: _Request) -> int:
        return (len(r.prompt) + r.max_new + self.page - 1) // self.page

    def run(self, prompts: Sequence[Sequence[int]], max_new_tokens: int, sampling: Optional[SamplingConfig] = None, eos: Optional[int] = None) -> List[List[int]]:
        """Token ids generated for every prompt (without EOS).  sampling None: greedy."""
        eos = self.session.model.config().eos_token_id if eos is None else eos
        reqs = [_Request(i, [int(t) for t in p], max_new_tokens) for i, p in enumerate(prompts)]
        greedy = sampling is None or (sampling.temperature <= 0 and sampling.repetition_penalty == 1.0 and sampling.frequency_penalty == 0.0 and sampling.presence_penalty == 0.0)
        for r in reqs:
            if not r.prompt:
                raise ValueError("empty prompt")
            r.rng = ((sampling.seed or 0) + r.index if sampling else 0) | 1
        waiting, running = deque(r for r in reqs if r.max_new > 0), []
        free_pages = self.session.model.free_tokens() // self.page
        while waiting or running:
            # a request enters when its slot and all the pages it can come to need are free
            while waiting and self.session.free_slots() > len([r for r in running if r.fed == 0]) and self._pages(waiting[0]) <= free_pages:
                free_pages -= self._pages(waiting[0])
                running.append(waiting.popleft())
            if not running:
                raise KvCacheFull(3, f"a request of {len(waiting[0].prompt)} + {waiting[0].max_new} tokens does not fit the pool")
            budget, entries, batch = self.batch_tokens, [], []
            for r in sorted(running, key=lambda r: r.fed < len(r.prompt)):  # generating requests first
                if r.fed < len(r.prompt):
                    n = min(self.portion, len(r.prompt) - r.fed, budget)
                    tokens = r.prompt[r.fed : r.fed + n]
                else:
                    n, tokens = min(1, budget), r.out[-1:]
                if n == 0:
                    continue
                last = r.fed + n >= len(r.prompt)
                entries.append((r.index, tokens, [n - 1] if last else []))
                batch.append((r, n, last))
                budget -= n
            logits, ids = self.session.step(entries, want_logits=not greedy, want_greedy=greedy)
            k = 0
            for r, n, last in batch:
                r.fed += n
                if not last:
                    continue
                if greedy:
                    tok = int(ids[k])
                else:
                    tok, r.rng = sample_token_device(logits[k], sampling, r.out, r.rng)
                k += 1
                stop = eos is not None and tok == eos
                if not stop:
                    r.out.append(tok)
                if stop or len(r.out) >= r.max_new:
                    self.session.end(r.index)
                    running.remove(r)
                    free_pages += self._pages(r)
        return [r.out for r in reqs]
