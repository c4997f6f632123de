"""Continuous batching for token-by-token decoders.

Same queues, admission and pre-emption as the block-diffusion scheduler it derives from.  What differs: a request
also holds a state slot; a prompt runs in portions of whatever fits the step's token budget; a decode step feeds one
token per request; a pre-empted request gives pages and slot back and later runs its prompt and the tokens it has
produced once more.
"""
from __future__ import annotations

from .scheduler import Scheduler
from .sequence import Sequence, SequenceStatus
from .state_manager import StateManager


class CausalSequence(Sequence):
    """A request whose tokens are produced one at a time.  ``num_cached_tokens`` counts the tokens whose latents and
    state the engine holds; ``num_scheduled`` those the next step brings."""

    def __init__(self, token_ids, sampling_params=None):
        super().__init__(token_ids, sampling_params, denoising_block_size=0, mask_token_id=-1)
        self.state_slot = -1
        self.num_scheduled = 0
        self.next_token: int | None = None      # set by the runner when the step reached the last token

    @property
    def target_temperature(self) -> float:
        return 0.0 if self.sampling_params.greedy else self.temperature

    def append_token(self, token: int) -> None:
        self.token_ids.append(token)
        self.step_map.append(len(self.step_map))
        self.last_token = token
        self.num_tokens += 1


class CausalScheduler(Scheduler):

    def __init__(self, config):
        super().__init__(config)
        self.state_manager = StateManager(config.num_state_slots)

    def add(self, seq: CausalSequence):
        if not isinstance(seq, CausalSequence):
            raise TypeError("this design decodes CausalSequence requests")
        if seq.num_blocks > self.block_manager.num_blocks:
            raise ValueError("request needs more pages than the cache has")
        super().add(seq)

    def schedule(self) -> tuple[list[CausalSequence], bool]:
        picked: list[CausalSequence] = []
        budget = self.max_num_batched_tokens
        # prompts: first the ones already under way, then new requests
        for seq in self.running:
            left = len(seq) - seq.num_cached_tokens
            if left > 1 and budget > 0 and len(picked) < self.max_num_seqs:
                seq.num_scheduled = min(left, budget)
                budget -= seq.num_scheduled
                picked.append(seq)
        while self.waiting and budget > 0 and len(self.running) < self.max_num_seqs and len(picked) < self.max_num_seqs:
            seq = self.waiting[0]
            if not self.block_manager.can_allocate(seq) or not self.state_manager.can_allocate():
                break
            self.block_manager.allocate(seq)
            self.state_manager.allocate(seq)
            seq.status = SequenceStatus.RUNNING
            seq.num_scheduled = min(len(seq), budget)
            budget -= seq.num_scheduled
            self.running.append(self.waiting.popleft())
            picked.append(seq)
        if picked:
            return picked, True
        return self._schedule_decode(picked), False

    def _schedule_decode(self, picked: list[CausalSequence]) -> list[CausalSequence]:
        while self.running and len(picked) < self.max_num_seqs:
            seq = self.running.popleft()
            kept = True
            while kept and not self.block_manager.can_append(seq):
                if self.running:
                    self.preempt(self.running.pop())
                else:
                    self.preempt(seq)
                    kept = False
            if kept:
                self.block_manager.may_append(seq)
                seq.num_scheduled = 1
                picked.append(seq)
        if not picked:
            raise AssertionError("no request could be scheduled")
        self.running.extendleft(reversed(picked))
        return picked

    def preempt(self, seq: CausalSequence):
        super().preempt(seq)
        self.state_manager.deallocate(seq)

    def postprocess(self, seqs: list[CausalSequence]):
        for seq in seqs:
            seq.num_cached_tokens += seq.num_scheduled
            seq.num_scheduled = 0
            if seq.next_token is None:          # the prompt goes on in a later step
                continue
            token, seq.next_token = seq.next_token, None
            seq.append_token(token)
            stop = not seq.ignore_eos and (token == self.eos or token in seq.sampling_params.stop_token_ids)
            if stop or seq.num_completion_tokens >= seq.max_new_tokens:
                seq.status = SequenceStatus.FINISHED
                self.block_manager.deallocate(seq)
                self.state_manager.deallocate(seq)
                self.running.remove(seq)
