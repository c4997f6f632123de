"""Model runner of token-by-token decoders (``HybridConfig`` designs) on one B200.

Same boundary as the block-diffusion runner: built from a ``Config``, driven by ``call("run", seqs, is_prefill)``, it
sizes the cache from free memory, reads ``config.model`` or takes weights, and leaves its result on the sequences
(``next_token``).  ``execute`` underneath is the step function: any number of tokens of any number of sequences, from
the pages and state slots the sequences hold, and logits at the rows asked for.  Steps that bring one token per
sequence replay a CUDA graph per batch-size bucket.
"""
from __future__ import annotations

import numpy as np
import torch

from .. import loader, ops
from ..hybrid import PAGE, HybridEngine, HybridWeights, StepBatch, bytes_per_page, bytes_per_slot, pad128
from .causal_scheduler import CausalSequence
from .config import Config


class _StepInputs:
    """Inputs of a step in one pinned buffer with a device twin: one host->device copy per step.  Per-sequence fields
    come first, so the copy ends with the rows in use."""

    def __init__(self, max_rows: int, max_bs: int, max_pages: int, device):
        self.max_rows, self.max_bs, self.max_pages = max_rows, max_bs, max_pages
        fields = [("step", np.int32, (4,)), ("cu_q", np.int32, (max_bs + 1,)), ("cu_k", np.int32, (max_bs + 1,)),
                  ("start", np.int32, (max_bs,)), ("slot", np.int32, (max_bs,)), ("table", np.int32, (max_bs, max_pages)),
                  ("ids", np.int64, (max_rows,)), ("pos", np.int32, (max_rows,)), ("row_seq", np.int32, (max_rows,)),
                  ("slots", np.int32, (max_rows,)), ("want", np.int64, (max_rows,)), ("temp", np.float32, (max_rows,))]
        at, spans = 0, {}
        for name, dt, shape in fields:
            n = int(np.prod(shape)) * np.dtype(dt).itemsize
            spans[name] = (at, n, dt, shape)
            at += (n + 15) // 16 * 16
        self.nbytes = at
        self.host = torch.zeros(at, dtype=torch.uint8, pin_memory=True)
        self.dev = torch.zeros(at, dtype=torch.uint8, device=device)
        types = {np.int32: torch.int32, np.int64: torch.int64, np.float32: torch.float32}
        self.h = {k: self.host[o:o + n].view(types[dt]).numpy().reshape(shape) for k, (o, n, dt, shape) in spans.items()}
        self.d = {k: self.dev[o:o + n].view(types[dt]).view(shape) for k, (o, n, dt, shape) in spans.items()}

    def send(self):
        self.dev.copy_(self.host, non_blocking=True)

    def fill(self, seqs: list[CausalSequence], counts: list[int], pad_to: int = 0) -> tuple[int, int, int]:
        """Rows of every sequence's next tokens.  Returns (rows, longest portion, summed context lengths).  With
        ``pad_to`` the batch is filled up with one-row padding entries."""
        h, row, total_k, longest = self.h, 0, 0, 0
        h["cu_q"][0] = h["cu_k"][0] = 0
        for i, (seq, n) in enumerate(zip(seqs, counts)):
            lo = seq.num_cached_tokens
            hi = lo + n
            r = slice(row, row + n)
            h["ids"][r] = seq.token_ids[lo:hi]
            h["pos"][r] = np.arange(lo, hi)
            h["row_seq"][r] = i
            pages = np.asarray(seq.block_table, dtype=np.int64)
            p = np.arange(lo, hi)
            h["slots"][r] = pages[p // PAGE] * PAGE + p % PAGE
            h["table"][i, :len(pages)] = pages
            h["table"][i, len(pages):] = -1
            h["start"][i], h["slot"][i] = lo, seq.state_slot
            row += n
            total_k += hi
            longest = max(longest, n)
            h["cu_q"][i + 1], h["cu_k"][i + 1] = row, total_k
        for i in range(len(seqs), pad_to):
            h["ids"][row], h["pos"][row], h["row_seq"][row], h["slots"][row] = 0, -1, i, -1
            h["start"][i], h["slot"][i] = 0, -1
            row += 1
            h["cu_q"][i + 1], h["cu_k"][i + 1] = row, total_k
        return row, longest, total_k


class CausalModelRunner:

    def __init__(self, config: Config, rank: int = 0, event=None, weights: HybridWeights | None = None,
                 weight_seed: int = 20260320, noise_seed: int = 0, device: str | None = None):
        if not torch.cuda.is_available():
            raise RuntimeError("the decode path has no CPU implementation: a CUDA device is needed")
        if config.tensor_parallel_size != 1:
            raise NotImplementedError("this design runs on one GPU (more GPUs serve as request-parallel replicas)")
        self.config, self.rank, self.event = config, rank, event
        self.cfg = config.decoder_config
        self.device = torch.device(device or f"cuda:{rank}")
        torch.cuda.set_device(self.device)
        self.dtype = getattr(torch, config.dtype)
        if weights is not None:
            self.weights = weights
        elif loader.has_checkpoint(config.model):
            self.weights = loader.load_hybrid_weights(config.model, self.cfg, self.device, self.dtype)
        else:
            self.weights = HybridWeights.random_init(self.cfg, weight_seed, self.device, self.dtype)
        if self.weights.dtype != self.dtype:
            raise ValueError(f"weights are {self.weights.dtype}, the configuration says {self.dtype}")
        self.noise_seed = noise_seed
        self.step_index = 0
        self.max_bs = config.max_num_seqs
        self.max_rows = max(config.max_num_batched_tokens, self.max_bs)
        self.max_pages = (config.max_model_len + PAGE - 1) // PAGE
        self._size_cache()
        self.engine = HybridEngine(self.cfg, self.weights, config.num_kvcache_blocks, config.num_state_slots, self.max_rows,
                                   self.device)
        self.prompt_inputs = _StepInputs(self.max_rows, self.max_bs, self.max_pages, self.device)
        self.inputs = _StepInputs(self.max_bs, self.max_bs, self.max_pages, self.device)      # one token per sequence
        vp = pad128(self.cfg.vocab_size)
        self.max_want = self.max_bs
        self.logits_dev = torch.zeros(self.max_bs, vp, dtype=torch.float32, device=self.device)
        self.hidden_rows = torch.zeros(self.max_bs, self.engine.width_pad, dtype=self.dtype, device=self.device)
        # tokens of the step, then the device status word
        self.res_dev = torch.zeros(self.max_bs + 1, dtype=torch.int64, device=self.device)
        self.res_host = torch.zeros(self.max_bs + 1, dtype=torch.int64, pin_memory=True)
        self.graphs: dict[int, torch.cuda.CUDAGraph] = {}
        self.step_events = None         # benchmark: (start, end) CUDA events recorded around a step's GPU work
        if not config.enforce_eager:
            self.capture_cudagraph()

    # ------------------------------------------------------------------ control plane, memory
    def call(self, method_name, *args):
        return getattr(self, method_name)(*args)

    def exit(self):
        torch.cuda.synchronize(self.device)
        self.graphs.clear()

    def _size_cache(self):
        """Cache pages and state slots: as configured, else a slot per request in flight and what memory is left."""
        config = self.config
        if config.num_state_slots <= 0:
            config.num_state_slots = config.max_num_seqs
        page = bytes_per_page(self.cfg, self.dtype)
        if config.num_kvcache_blocks <= 0:
            if page == 0:                       # no attention: pages only bound the lengths
                config.num_kvcache_blocks = self.max_pages * config.max_num_seqs
                return
            free, total = torch.cuda.mem_get_info(self.device)
            budget = int(total * config.gpu_memory_utilization) - (total - free)
            budget -= config.num_state_slots * bytes_per_slot(self.cfg, self.dtype)
            reserve = 6 << 30                   # activation buffers allocated after the cache
            wanted = self.max_pages * config.max_num_seqs
            config.num_kvcache_blocks = min(wanted, (budget - reserve) // page)
        if config.num_kvcache_blocks <= 0:
            raise AssertionError("no memory left for the paged cache")

    # ------------------------------------------------------------------ the step function
    def _batch(self, inp: _StepInputs, m: int, bs: int, max_q: int, total_k: int, max_ctx: int) -> StepBatch:
        d = inp.d
        return StepBatch(m, bs, d["ids"][:m], d["pos"][:m], d["row_seq"][:m], d["slots"][:m], d["cu_q"][:bs + 1],
                         d["cu_k"][:bs + 1], d["start"][:bs], d["slot"][:bs], d["table"][:bs], max_q, total_k, max_ctx)

    def _check_counts(self, seqs, counts):
        if len(seqs) > self.max_bs:
            raise AssertionError("batch larger than max_num_seqs")
        for seq, n in zip(seqs, counts):
            end = seq.num_cached_tokens + n
            if n < 1 or end > len(seq) or end > PAGE * len(seq.block_table) or len(seq.block_table) > self.max_pages:
                raise AssertionError("a sequence brings tokens it does not have, or holds no pages for them")
            if seq.state_slot < 0:
                raise AssertionError("a sequence holds no state slot")

    def _one_token_body(self, bs: int):
        """All of a one-token step that depends only on device buffers, for a bucket of ``bs`` requests."""
        eng, d = self.engine, self.inputs.d
        h = eng.forward(self._batch(self.inputs, bs, bs, 1, 0, self.config.max_model_len))
        eng.logits(h, self.logits_dev[:bs])
        status = self.res_dev[bs:bs + 1].view(torch.int32)
        ops.pick_token(self.logits_dev[:bs], self.cfg.vocab_size, d["temp"][:bs], self.noise_seed, d["step"], self.res_dev[:bs],
                       status)

    @torch.inference_mode()
    def execute(self, seqs: list[CausalSequence], counts: list[int], want: list[tuple[int, int]] | None = None):
        """Runs the next ``counts[i]`` tokens of every sequence.  ``want`` lists (sequence index, place in its portion);
        returns (fp32 logits [len(want), vocab] on the device, sampled tokens [len(want)] list).  Without ``want`` the
        logits of every sequence's last token are meant.  The caller advances ``num_cached_tokens``."""
        self._check_counts(seqs, counts)
        bs = len(seqs)
        if want is None:
            want = [(i, n - 1) for i, n in enumerate(counts)]
        one_token = all(n == 1 for n in counts)
        nw = len(want)
        if one_token and [w[0] for w in want] == list(range(bs)) and self.graphs:
            gbs = next(x for x in sorted(self.graphs) if x >= bs)
            inp = self.inputs
            inp.fill(seqs, counts, pad_to=gbs)
            inp.h["temp"][:bs] = [s.target_temperature for s in seqs]
            inp.h["step"][0] = self.step_index
            self._mark(0)
            self.graphs[gbs].replay()
            self._mark(1)
            self._finish(gbs)
            return self.logits_dev[:bs, :self.cfg.vocab_size], self.res_host[:bs].tolist()
        inp = self.prompt_inputs
        m, max_q, total_k = inp.fill(seqs, counts)
        starts = np.concatenate([[0], np.cumsum(counts)])
        h = inp.h
        h["want"][:nw] = [int(starts[i]) + p for i, p in want]
        h["temp"][:nw] = [seqs[i].target_temperature for i, _ in want]
        h["step"][0] = self.step_index
        self._mark(0)
        inp.send()
        eng = self.engine
        max_ctx = max(s.num_cached_tokens + n for s, n in zip(seqs, counts))
        hidden = eng.forward(self._batch(inp, m, bs, max_q, total_k, max_ctx))
        logits, tokens = [], []
        for lo in range(0, nw, self.max_want) or [0]:
            n = min(self.max_want, nw - lo)
            if n > 0:
                rows = ops.copy_rows(hidden, inp.d["want"][lo:lo + n], self.hidden_rows[:n])
                eng.logits(rows, self.logits_dev[:n])
                ops.pick_token(self.logits_dev[:n], self.cfg.vocab_size, inp.d["temp"][lo:lo + n], self.noise_seed,
                               inp.d["step"], self.res_dev[:n], self.res_dev[n:n + 1].view(torch.int32))
                self.res_host[:n + 1].copy_(self.res_dev[:n + 1], non_blocking=True)
                self._mark(1)
                self._finish(n)
                part = self.logits_dev[:n, :self.cfg.vocab_size]
                logits.append(part if nw <= self.max_want else part.clone())
                tokens += self.res_host[:n].tolist()
        if nw == 0:
            torch.cuda.synchronize(self.device)
            from .._lib import device_status
            self._check_status(device_status(clear=True))
            return None, []
        return logits[0] if len(logits) == 1 else torch.cat(logits), tokens

    def _mark(self, which: int):
        if self.step_events is not None:
            self.step_events[which].record()

    def _finish(self, n: int):
        torch.cuda.current_stream().synchronize()
        self._check_status(int(self.res_host[n:n + 1].view(torch.int32)[0]))

    def _check_status(self, status: int):
        if status:
            raise RuntimeError(f"step {self.step_index}: device status word {status:#x} "
                               "(1 bad slot, 2 bad page, 4 bad token id, 16 wait timed out)")

    # ------------------------------------------------------------------ engine entry point
    def run(self, seqs: list[CausalSequence], is_prefill: bool) -> int:
        """One step of the scheduler's batch; returns the number of tokens produced."""
        counts = [seq.num_scheduled for seq in seqs]
        done = [i for i, (seq, n) in enumerate(zip(seqs, counts)) if seq.num_cached_tokens + n == len(seq)]
        _, tokens = self.execute(seqs, counts, [(i, counts[i] - 1) for i in done])
        for i, token in zip(done, tokens):
            seqs[i].next_token = token
        self.step_index += 1
        return len(done)

    # ------------------------------------------------------------------ CUDA graphs
    @torch.inference_mode()
    def capture_cudagraph(self):
        """One graph per batch-size bucket: copy of the step inputs, layers, logits, token choice, copy of the results.
        Padding entries carry slot -1, which every kernel treats as a no-op."""
        buckets = [x for x in (1, 2, 4, 8) if x <= self.max_bs] + list(range(16, self.max_bs + 1, 16))
        if buckets[-1] != self.max_bs:
            buckets.append(self.max_bs)
        pool = None
        for bs in reversed(buckets):
            self.inputs.fill([], [], pad_to=bs)
            self.inputs.h["temp"].fill(0.0)
            self.inputs.send()
            self._one_token_body(bs)        # sets kernel attributes and allocates buffers outside the capture
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph, pool):
                self.inputs.send()
                self._one_token_body(bs)
                self.res_host[:bs + 1].copy_(self.res_dev[:bs + 1], non_blocking=True)
            if pool is None:
                pool = graph.pool()
            self.graphs[bs] = graph
        torch.cuda.synchronize()
