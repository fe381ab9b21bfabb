"""Which sequences run in the next step (the part of nanovllm/engine/scheduler.py:25-84 that the models here need).

A step is either prefill or decode.  Waiting sequences are admitted first, whole prompts side by side up to the token
budget; a prompt that exceeds it is cut into portions.  When a running sequence needs a block and none is free, the most
recently admitted sequence gives everything back and is computed again later.
"""
from __future__ import annotations

from collections import deque

from .cache_manager import CacheManager


class Scheduler:

    def __init__(self, cache: CacheManager, max_num_seqs: int, max_num_batched_tokens: int):
        self.cache, self.max_num_seqs, self.max_tokens = cache, max_num_seqs, max_num_batched_tokens
        self.waiting: deque = deque()
        self.running: list = []

    def add(self, seq) -> None:
        self.waiting.append(seq)

    def done(self) -> bool:
        return not self.waiting and not self.running

    def schedule(self) -> tuple[list, list[int] | None]:
        """(sequences, tokens of each to compute) for a prefill step, (sequences, None) for a decode step."""
        batch, counts, budget = [], [], self.max_tokens
        while self.waiting and budget > 0 and len(self.running) + len(batch) < self.max_num_seqs:
            seq = self.waiting[0]
            todo = len(seq) - seq.num_cached_tokens
            n = min(todo, budget)
            if batch and n < todo:
                break  # only the first prompt of a step is cut
            if not self.cache.can_hold(seq, seq.num_cached_tokens + n):
                break
            self.cache.hold(seq, seq.num_cached_tokens + n)
            batch.append(seq)
            counts.append(n)
            budget -= n
            if n < todo:
                break  # stays at the head of the queue until its last portion has run
            self.waiting.popleft()
        if batch:
            return batch, counts
        ready, preempted = [], False
        for seq in list(self.running):
            if seq not in self.running:
                continue  # preempted for a sequence before it
            while not self.cache.can_hold(seq, len(seq)):
                victim = self.running[-1]
                self._preempt(victim)
                preempted = True
                if victim is seq:
                    break
            else:
                self.cache.hold(seq, len(seq))
                ready.append(seq)
        if ready:
            return ready, None
        # nothing fits: portions of prompts further back in the queue give way to the one in front
        for seq in reversed(self.waiting):
            if seq.block_table and seq is not self.waiting[0]:
                self.cache.release(seq)
                return self.schedule()
        if preempted:
            return self.schedule()
        raise RuntimeError("nothing to schedule" if not self.waiting else "the KV cache is too small for one sequence")

    def _preempt(self, seq) -> None:
        self.running.remove(seq)
        self.cache.release(seq)
        self.waiting.appendleft(seq)

    def prefilled(self, seq, n: int) -> bool:
        """Books n computed prompt tokens; True when the whole prompt is in the cache (the step's sample counts)."""
        seq.num_cached_tokens += n
        if seq.num_cached_tokens < len(seq):
            return False
        self.running.append(seq)
        return True

    def finish(self, seq) -> None:
        self.running.remove(seq)
        self.cache.release(seq)
