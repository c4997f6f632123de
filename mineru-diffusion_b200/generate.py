"""Command line: generates tokens from a model folder, for prompts given as token ids.

The folder's ``config.json`` decides the design; ``--greedy`` is for token-by-token designs.  One JSON line per prompt:
``{"prompt": [...], "tokens": [...]}``, in the order given.
"""
from __future__ import annotations

import argparse
import json
import sys

from .engine.config import Config
from .engine.llm_engine import LLMEngine
from .engine.sampling_params import SamplingParams


def parse(argv=None):
    ap = argparse.ArgumentParser(prog="generate", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--prompt", action="append", required=True, metavar="IDS", help="token ids with commas between them; repeatable")
    ap.add_argument("--max-new-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--greedy", action="store_true", help="always the most likely token")
    ap.add_argument("--seed", type=int, default=0, help="seed of the sampling noise")
    ap.add_argument("--stop", type=int, action="append", default=[], metavar="ID", help="token id that ends a request; repeatable")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--max-num-seqs", type=int, default=16, help="requests in flight")
    ap.add_argument("--max-model-len", type=int, default=4096)
    ap.add_argument("--max-num-batched-tokens", type=int, default=16384)
    ap.add_argument("--eager", action="store_true", help="no CUDA graphs")
    a = ap.parse_args(argv)
    a.prompt = [[int(t) for t in p.replace(",", " ").split()] for p in a.prompt]
    if not all(a.prompt):
        ap.error("a prompt needs at least one token")
    return a


def main(argv=None) -> int:
    a = parse(argv)
    config = Config(model=a.model, dtype=a.dtype, max_num_seqs=a.max_num_seqs, max_model_len=a.max_model_len,
                    max_num_batched_tokens=max(a.max_num_batched_tokens, a.max_model_len), enforce_eager=a.eager)
    longest = max(map(len, a.prompt)) + a.max_new_tokens
    if longest > config.max_model_len:
        print(f"a request may grow to {longest} tokens, --max-model-len is {config.max_model_len}", file=sys.stderr)
        return 2
    engine = LLMEngine.from_config(config, noise_seed=a.seed)
    requests = [engine.new_request(p, SamplingParams(temperature=a.temperature, max_new_tokens=a.max_new_tokens, greedy=a.greedy,
                                                     ignore_eos=not a.stop, stop_token_ids=a.stop)) for p in a.prompt]
    done, _ = engine.generate(requests)
    for prompt, request in zip(a.prompt, requests):
        print(json.dumps({"prompt": prompt, "tokens": done[request.seq_id][0]}), flush=True)
    engine.model_runner.exit()
    return 0
