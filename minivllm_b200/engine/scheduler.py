"""Continuous-batching scheduler on the host, the policy of the reference's
src/myvllm/engine/scheduler.py:25-82: a prefill wave whenever waiting requests
fit (sequence and token budgets, free blocks), otherwise one decode token for
every running sequence, preempting from the tail when no block is free.

With `chunked_prefill` a step is mixed instead: one token for every decoding sequence, and portions of prompts up to
the token budget beside them.  `Sequence.num_cached_tokens` then counts the tokens that earlier steps have put into
the cache (and into the per-sequence state), `num_scheduled_tokens` those of the step being run.
"""
from collections import deque

from .block_manager import BlockManager
from .sequence import Sequence, SequenceStatus


class Scheduler:
    def __init__(self, max_num_seqs, max_num_batched_tokens, num_blocks, block_size, eos, num_slots=None,
                 prefix_caching=False, chunked_prefill=False):
        if chunked_prefill and prefix_caching:
            # a block's hash is published when its table is allocated, before a later portion has filled it
            raise ValueError("chunked prefill cannot be combined with prefix caching")
        self.chunked_prefill = chunked_prefill
        self.max_num_seqs = max_num_seqs
        self.max_num_batched_tokens = max_num_batched_tokens
        self.block_manager = BlockManager(num_blocks, block_size, num_slots or max_num_seqs, prefix_caching)
        self.eos = eos
        self.waiting: deque[Sequence] = deque()
        self.running: deque[Sequence] = deque()

    def is_finished(self):
        return not self.waiting and not self.running

    def add_sequence(self, seq):
        self.waiting.append(seq)

    def schedule(self):
        """Returns (sequences, is_prefill)."""
        if self.chunked_prefill:
            return self._schedule_mixed()
        picked, tokens = [], 0
        while self.waiting and len(self.running) < self.max_num_seqs:
            seq = self.waiting[0]
            if not self.block_manager.can_allocate(seq) or tokens + len(seq) > self.max_num_batched_tokens:
                break
            self.waiting.popleft()
            self.block_manager.allocate(seq)
            seq.status = SequenceStatus.RUNNING
            self.running.append(seq)
            picked.append(seq)
            tokens += len(seq)
        if picked:
            return picked, True
        # decode: every running sequence that can get a slot for its next token
        survivors = deque()
        while self.running:
            seq = self.running.popleft()
            while not self.block_manager.can_append(seq):
                if self.running:
                    self.preempt(self.running.pop())
                else:
                    self.preempt(seq)
                    seq = None
                    break
            if seq is None:
                break
            self.block_manager.append(seq)
            survivors.append(seq)
        self.running = survivors
        return list(survivors), False

    def _schedule_mixed(self):
        """Decoding sequences first (preempting from the tail when no block is free), then prompts in progress, then
        new ones.  A step in which every input token is already on the device is a decode step."""
        budget, picked, survivors = self.max_num_batched_tokens, [], deque()

        def take(seq):
            nonlocal budget
            seq.num_scheduled_tokens = min(len(seq) - seq.num_cached_tokens, budget)
            budget -= seq.num_scheduled_tokens
            if seq.num_scheduled_tokens:
                picked.append(seq)

        while self.running:
            seq = self.running.popleft()
            while seq is not None and not self.block_manager.can_append(seq):
                if self.running:
                    self.preempt(self.running.pop())
                else:
                    self.preempt(seq)
                    seq = None
            if seq is None:
                break
            self.block_manager.append(seq)
            survivors.append(seq)
        self.running = survivors
        for decoding in (True, False):
            for seq in self.running:
                if (len(seq) - seq.num_cached_tokens == 1) == decoding and budget:
                    take(seq)
        while self.waiting and budget and len(self.running) < self.max_num_seqs:
            seq = self.waiting[0]
            if not self.block_manager.can_allocate(seq):
                break
            self.waiting.popleft()
            self.block_manager.allocate(seq)
            seq.status = SequenceStatus.RUNNING
            self.running.append(seq)
            take(seq)
        return picked, not all(s.on_device for s in picked)

    def _advance_cached(self, seq):
        """Mixed steps: the scheduled tokens are in the cache now.  True when the sequence gets a next token."""
        if not self.chunked_prefill:
            return True
        seq.num_cached_tokens += seq.num_scheduled_tokens
        return seq.num_cached_tokens == len(seq)

    def preempt(self, seq):
        self.block_manager.deallocate(seq)
        seq.status = SequenceStatus.WAITING
        self.waiting.appendleft(seq)

    def postprocess(self, seqs, token_ids):
        for seq, tok in zip(seqs, token_ids):
            if not self._advance_cached(seq):
                continue
            seq.append_token(tok)
            seq.on_device = True
            if (not seq.ignore_eos and tok == self.eos) or seq.num_completion_tokens >= seq.max_tokens:
                self._finish(seq)

    def _finish(self, seq):
        seq.status = SequenceStatus.FINISHED
        self.block_manager.deallocate(seq)
        self.running.remove(seq)

    # ---- one step of lookahead: bookkeeping before the sampled tokens have reached the host ----
    def can_run_ahead(self, seqs):
        """True when the step after this one can be scheduled without knowing this step's tokens: no
        sequence of the batch can end on an EOS token, and no token value is hashed (prefix cache off)."""
        return not self.block_manager.prefix_caching and all(s.ignore_eos or self.eos < 0 for s in seqs)

    def no_preemption_next(self):
        """The next decode step finds a block for every running sequence, so nothing is preempted (a preempted
        sequence is prefilled again from its token ids, which must then be real)."""
        return len(self.block_manager.free_blocks) >= len(self.running)

    def advance(self, seqs):
        """postprocess() with the token values still unknown: appends a placeholder to every sequence and
        finishes those that reached max_tokens.  Returns the positions to hand to `fill_tokens`."""
        at = []
        for seq in seqs:
            if not self._advance_cached(seq):
                at.append(-1)            # a prompt in progress: nothing was sampled for it
                continue
            at.append(len(seq.token_ids))
            seq.append_token(-1)
            seq.on_device = True
            if seq.num_completion_tokens >= seq.max_tokens:
                self._finish(seq)
        return at

    @staticmethod
    def fill_tokens(seqs, positions, token_ids):
        for seq, pos, tok in zip(seqs, positions, token_ids):
            if pos >= 0:
                seq.token_ids[pos] = int(tok)
