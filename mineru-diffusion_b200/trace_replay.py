"""Replays a trace of given token ids through a model, step by step, and writes the logits asked for.

Steps come as JSON lines: ``entries`` (request id, its next tokens, the places among them whose logits are wanted) and
``end`` (requests that give their pages and state slot back).  The requests are the engine's own ``CausalSequence``
objects, run by ``CausalModelRunner.execute`` on pages and slots of the engine's own managers.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from .engine import registry
from .engine.block_manager import BlockManager
from .engine.causal_scheduler import CausalSequence
from .engine.config import Config
from .engine.state_manager import StateManager

PAGE = 256
EXIT_UNSUPPORTED = 3


class TraceReplay:

    def __init__(self, model: str, dtype: str, max_tokens: int, max_seqs: int = 8):
        max_len = max(PAGE, (max_tokens + PAGE - 1) // PAGE * PAGE)
        self.config = Config(model=model, dtype=dtype, max_num_seqs=max_seqs, max_model_len=max_len,
                             max_num_batched_tokens=max_len, num_kvcache_blocks=max_len // PAGE + max_seqs)
        arch = registry.of_config(self.config.decoder_config)
        self.runner = arch.load("runner")(self.config)
        self.pages = BlockManager(self.config.num_kvcache_blocks, PAGE)
        self.slots = StateManager(self.config.num_state_slots)
        self.live: dict[str, CausalSequence] = {}

    def step(self, entries: list[dict], end: list[str]):
        """Runs one step; returns fp32 logits [wanted, vocab] on the host, or None when nothing is wanted."""
        seqs, counts, want = [], [], []
        for e in entries:
            seq = self.live.get(e["id"])
            if seq is None:
                seq = self.live[e["id"]] = CausalSequence(e["tokens"])
                self.slots.allocate(seq)
            else:
                for token in e["tokens"]:
                    seq.append_token(token)
            while len(seq) > PAGE * len(seq.block_table):
                seq.block_table.append(self.pages._take())
            want += [(len(seqs), place) for place in e["want"]]
            seqs.append(seq)
            counts.append(len(e["tokens"]))
        logits = self.runner.execute(seqs, counts, want)[0] if seqs else None
        out = None if logits is None else logits.cpu()
        for seq, n in zip(seqs, counts):
            seq.num_cached_tokens += n
        for name in end:
            seq = self.live.pop(name)
            self.pages.deallocate(seq)
            self.slots.deallocate(seq)
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--dtype", required=True, choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="folder for <step>.f32: little-endian fp32 [wanted, vocab]")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens the live requests hold at any time")
    a = ap.parse_args(argv)
    with open(os.path.join(a.model, "config.json")) as f:
        if a.dtype == "float32" and "architecture" not in json.load(f):
            print("this design runs in bfloat16 only", file=sys.stderr)
            return EXIT_UNSUPPORTED
    replay = TraceReplay(a.model, a.dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if logits is not None:
            part = os.path.join(a.out, f".{step['step']}.part")
            logits.numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(a.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    replay.runner.exit()
    return 0
