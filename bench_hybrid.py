"""Speed of the causal decoder designs beside the framework's closest other models at equal width, layers and vocabulary.

``python bench.py --design hybrid [--size 2k|4k]`` sets the hybrid design (Zikunex) beside the block-diffusion decoder,
``--design nipadra`` the Nipadra design beside the hybrid one with dense feed-forwards and the block-diffusion decoder.
One JSON line: prefill and decode throughput of all (random
weights, synthetic tokens), and for every kernel-launching operation of a prompt and of a decode step the time of one
call and its fraction of the roofline.  Times are CUDA events on the launching stream, the median of several calls
with an L2 flush (a 256 MB write) before each.  Roofline of an operation: the slowest of its bytes at the copy rate,
its tensor flops at the cuBLAS rate and, for the recurrences (fp32 by design), its fp32 flops at the FMA rate.
"""
from __future__ import annotations

import json
import statistics
import sys

import torch

HBM_GBS, BF16_TFLOPS = 6650.0, 1590.0        # used when no measured peaks are at hand
FP32_TFLOPS = 148 * 128 * 2 * 1.965e-3       # nominal: 128 FMA per SM and cycle

SIZES = {
    # width, heads of 128, dense ff, expert ff, experts, top, shared ff, q_rank, kv_rank, vocab
    "2k": dict(width=2048, heads=16, ff=6144, eff=1024, experts=64, top=6, shared=2048, q_rank=1536, kv_rank=512, vocab=32768),
    "4k": dict(width=4096, heads=32, ff=12288, eff=1536, experts=64, top=6, shared=3072, q_rank=1536, kv_rank=512, vocab=32768),
}


def design_config(pkg, s: dict):
    """Eight layers: every mixer twice, the second latent layer on the first one's cache; dense and expert feed-forwards."""
    heads, dense = s["heads"], {"kind": "dense", "ff": s["ff"]}
    moe = {"kind": "moe", "expert": {"ff": s["eff"]}, "shared": {"ff": s["shared"]},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": 8, "keep": 4}}}
    delta = {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4)}
    mlstm = {"type": "mlstm", "mixer": dict(heads=heads // 2, dim=128, vdim=256, gate_cap=15.0)}
    latent = {"type": "latent_attention", "mixer": dict(heads=heads, dim=128, vdim=128, q_rank=s["q_rank"], kv_rank=s["kv_rank"],
                                                        scale=128 ** -0.5)}
    shared = {"type": "latent_attention", "mixer": dict(latent["mixer"], kv_from=2)}
    layers = [(delta, dense), (delta, moe), (latent, moe), (mlstm, dense), (delta, dense), (delta, moe), (shared, moe), (mlstm, dense)]
    return pkg.HybridConfig.from_json({
        "architecture": "Zikunex", "vocab": s["vocab"], "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
        "layers": [dict(l, mlp=m) for l, m in layers]})


def dense_hybrid_config(pkg, s: dict):
    """The hybrid design without experts: eight layers of mLSTM, latent attention and delta rule, dense feed-forwards."""
    heads, dense = s["heads"], {"kind": "dense", "ff": s["ff"]}
    delta = {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4)}
    mlstm = {"type": "mlstm", "mixer": dict(heads=heads // 2, dim=128, vdim=256, gate_cap=15.0)}
    latent = {"type": "latent_attention", "mixer": dict(heads=heads, dim=128, vdim=128, q_rank=s["q_rank"], kv_rank=s["kv_rank"],
                                                        scale=128 ** -0.5)}
    return pkg.HybridConfig.from_json({
        "architecture": "Zikunex", "vocab": s["vocab"], "width": s["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
        "layers": [dict(l, mlp=dense) for l in (mlstm, latent, mlstm, delta) * 2]})


def nipadra_config(pkg, s: dict):
    """Eight layers, lightning attention and the parallel mixer in turn: 128 channels a head, eight key heads, a window of
    1024, a Mamba-2 branch of twice the width; every second lightning layer without a feed-forward."""
    heads, dense = s["heads"], {"kind": "dense", "ff": s["ff"]}
    light = {"type": "lightning", "mixer": dict(heads=heads, dim=128, vdim=128, decay=[1 - 2.0 ** (-1 - 8 * h / heads) for h in range(heads)])}
    left = dict(heads=heads, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, mask={"size": 1024}, rot={"base": 1e4, "dims": 128})
    right = dict(heads=2 * s["width"] // 64, vdim=64, state=128, groups=8, conv=4, norm_groups=8)
    par = {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 0.9, "right_scale": 1.1}}
    return pkg.HybridConfig.from_json({
        "architecture": "Nipadra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-5}, "postln_alpha": 2.0,
        "layers": [dict(light, mlp=dense), dict(par, mlp=dense), dict(light, mlp=None), dict(par, mlp=dense)] * 2})


def closest_config(pkg, s: dict):
    return pkg.DecoderConfig(vocab_size=s["vocab"], hidden_size=s["width"], intermediate_size=s["ff"], num_hidden_layers=8,
                             num_attention_heads=s["heads"], num_key_value_heads=8, max_position_embeddings=16384)


# ----------------------------------------------------------------------------- per-operation times
class Recorder:
    """Swaps the functions of ``ops`` for ones that note every call."""
    NAMES = ("gemm", "gemm_heads", "gemm_experts", "gemm_splitk_partials", "linear", "gateup_swiglu", "residual_norm", "rms_rows",
             "add_rms_norm", "gated_norm", "delta_prep", "channel_decay", "mlstm_prep", "scan", "moe_route", "moe_plan", "moe_gather",
             "part_norm", "decay_prep", "chunk_scan", "rotary_commit", "window_attn", "latent_attn", "gather_latents", "causal_attn_varlen", "sparse_attn_varlen", "block_attn_with_kvcache",
             "qkv_proj_rope_commit", "qknorm_rope_commit", "pick_token", "lm_head_sample", "gather_rows")

    def __init__(self, ops):
        self.ops, self.calls = ops, []

    def __enter__(self):
        self.saved = {n: getattr(self.ops, n) for n in self.NAMES}
        for n, fn in self.saved.items():
            def noted(*a, _n=n, _fn=fn, **k):
                self.calls.append((_n, _fn, a, k))
                return _fn(*a, **k)
            setattr(self.ops, n, noted)
        return self

    def __exit__(self, *_):
        for n, fn in self.saved.items():
            setattr(self.ops, n, fn)


def time_call(fn, flush: torch.Tensor, reps: int = 7) -> float:
    fn()
    times = []
    for _ in range(reps):
        flush.zero_()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1) * 1e3)
    return statistics.median(times)


def work_of(name: str, a: tuple, k: dict, ctx: dict):
    """(label, bytes, tensor flops, fp32 flops) of a recorded call, or None where no roofline is worth stating."""
    e = 2
    if name in ("gemm", "linear", "gemm_splitk_partials"):
        x, w = a[0], a[1]
        m, kk, n = x.shape[0], w.shape[1], w.shape[0]
        glu, silu = k.get("act") == 2, k.get("act") == 3
        return f"{name} {m}x{n}x{kk}" + (" glu" if glu else " silu" if silu else ""), (m * kk + n * kk + m * (n // 2 if glu else n)) * e, 2 * m * n * kk, 0
    if name == "gateup_swiglu":
        m, kk, n = a[0].shape[0], a[1].shape[1], a[1].shape[0]
        return f"gateup {m}x{n}x{kk}", (m * kk + n * kk + m * n // 2) * e, 2 * m * n * kk, 0
    if name == "qkv_proj_rope_commit":
        m, kk, n = a[0].shape[0], a[1].shape[1], a[1].shape[0]
        return f"qkv+rope {m}x{n}x{kk}", (m * kk + n * kk + m * n) * e, 2 * m * n * kk, 0
    if name == "gemm_heads":
        h, n, kk = a[1].shape
        m = a[0].shape[0]
        return f"per-head {m}x{h}x{n}x{kk}", (m * h * (n + kk) + h * n * kk) * e, 2 * m * h * n * kk, 0
    if name == "gemm_experts":
        E, n, kk = a[1].shape
        pairs, touched = ctx["rows"] * ctx["top"], ctx["touched"]
        return f"experts {pairs}x{n}x{kk}", (pairs * (n + kk) + touched * n * kk) * e, 2 * pairs * n * kk, 0
    if name == "causal_attn_varlen":
        q, kv = a[0], a[1]
        h, cu_q, cu_k = q.shape[1], a[3].tolist(), a[4].tolist()
        pairs = sum((cu_k[i + 1] - cu_k[i]) * (cu_q[i + 1] - cu_q[i]) - (cu_q[i + 1] - cu_q[i]) ** 2 / 2 for i in range(a[5]))
        return "causal attention", (2 * q.shape[0] + 2 * kv.shape[0]) * h * 128 * e, 4 * 128 * h * pairs, 0
    if name == "sparse_attn_varlen":
        cu, q, kv, h = a[3].tolist(), a[0], a[1], a[0].shape[1]
        pairs = sum((cu[i + 1] - cu[i]) ** 2 / 2 for i in range(len(cu) - 1))
        return "staircase attention", (2 * q.shape[0] * h + 2 * kv.shape[0] * kv.shape[1]) * 128 * e, 4 * 128 * h * pairs, 0
    if name == "latent_attn":
        q, cache, heads, keys = a[0], a[1], a[5], int((a[4] + 1).sum())
        w = cache.shape[1]
        return "latent attention", (keys * w + 2 * q.shape[0] * heads * w) * e, 4 * keys * heads * w, 0
    if name == "block_attn_with_kvcache":
        q, kc, keys = a[0], a[1], int(a[3].sum())
        return "block attention", (2 * keys * kc.shape[2] + 2 * q.shape[0] * q.shape[1] * q.shape[2]) * 128 * e, \
            4 * keys * q.shape[1] * q.shape[2] * 128, 0
    if name == "scan":
        mode, bs, heads, kvh, dim, vdim, rows = a[0], a[2], a[3], a[4], a[5], a[6], a[7].shape[0]
        per = dim * vdim
        io = rows * heads * (vdim * 8 + dim * (8 * kvh / heads + (4 if mode == 0 else 0))) + 2 * bs * heads * per * 4
        return ("delta scan", "mlstm scan", f"decay scan {heads}x{dim}x{vdim}")[mode], io, 0, rows * heads * per * (8 if mode == 0 else 6)
    if name == "residual_norm":
        m, wp = a[0].shape
        n = sum(e for _ in k.get("add", ())) + (ctx["top"] * e if k.get("moe") else 0) + e
        return "residual + norm" + (" + experts" if k.get("moe") else ""), m * wp * (8 + n), 0, 0
    if name == "add_rms_norm":
        src = a[0] if a[0] is not None else k["partials"]
        return "add + norm", src.shape[-2] * src.shape[-1] * 8, 0, 0
    if name == "delta_prep":
        m, heads, kvh, dim, vdim = a[1], a[3], a[4], a[5], a[6]
        c = 2 * kvh * dim + heads * vdim
        return "delta inputs", m * c * (e + 4), 0, 0
    if name == "window_attn":
        q, kc, starts, cu, window = a[0], a[1], a[4][2].tolist(), a[4][1].tolist(), a[8]
        m, h, d, keys, reads = q.shape[0], q.shape[1], a[7], 0, 0
        for i, s0 in enumerate(starts):
            n = cu[i + 1] - cu[i]
            keys += sum(min(window or p + 1, p + 1) for p in range(s0, s0 + n))       # (query, key) pairs
            reads += min(s0 + n, (window or s0 + n) + n - 1)                            # keys anyone sees
        return "window attention", (2 * reads * kc.shape[1] + 2 * m * h) * d * e, 4 * d * h * keys, 0
    if name == "chunk_scan":
        heads, kvh, dim, vdim, rows = a[1], a[2], a[3], a[4], a[5].shape[0]
        io = rows * (heads * vdim * (e + 4) + 2 * kvh * dim * e) + 2 * a[0] * heads * dim * vdim * 4
        # products of a 64-token chunk: scores (lower half), weighted scores and values (lower half, two terms), state read-out
        # and state update (two terms each)
        return f"chunk scan {heads}x{dim}x{vdim}", io, rows * heads * (64 * dim + 2 * 64 * vdim + 8 * dim * vdim), 0
    if name == "rotary_commit":
        h, g, d, m = a[3], a[4], a[5], a[12].shape[0]
        return "rotation + cache rows", m * (2 * h + 3 * g) * d * e, 0, 0
    if name == "decay_prep":
        m, heads, kvh, dim, vdim = a[1], a[3], a[4], a[5], a[6]
        return f"decay inputs {heads}x{dim}x{vdim}", m * (2 * kvh * dim + heads * vdim) * (e + a[11][0].element_size()), 0, 0
    if name == "part_norm":
        return f"gated norm in {a[3]} parts", a[0].numel() * (4 + 2 * e), 0, 0
    if name == "mlstm_prep":
        m, heads, dim, vdim = a[1:5]
        return "mlstm inputs", m * heads * (2 * dim + vdim) * (e + 4), 0, 0
    if name == "channel_decay":
        m, heads, dp = a[7].shape          # projection in, decay out, key and query, for every second token the key before
        return "decay", m * heads * dp * 8 + m * a[3].shape[1] * dp * 10, 0, 0
    if name == "gated_norm":
        m, h, v = a[0].shape
        return "gated norm", m * h * v * (4 + 2 * e), 0, 0
    if name == "moe_gather":
        return "expert gather", 2 * ctx["rows"] * ctx["top"] * a[1].shape[1] * e, 0, 0
    if name == "gather_latents":
        return "latent gather", 2 * a[4].numel() * e, 0, 0
    if name == "rms_rows":
        return "latent norms", a[1] * sum(s.n_pad for s in a[0]) * 2 * e, 0, 0
    if name == "lm_head_sample":
        x, w = a[0], a[1]
        return "LM head + sampler", (x.numel() + w.numel()) * e, 2 * x.shape[0] * w.numel(), 0
    return name, None, 0, 0


def op_table(rec: Recorder, peaks: dict, ctx: dict) -> list[dict]:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    floor = time_call(lambda: None, flush)
    rows: dict[str, list] = {}
    for name, fn, a, k in rec.calls:
        label, nbytes, tflops, fflops = work_of(name, a, k, ctx)
        us = max(time_call(lambda: fn(*a, **k), flush) - floor, 0.1)
        roof = None if nbytes is None else max(nbytes / (peaks["hbm_gbs"] * 1e3), tflops / (peaks["bf16_tflops"] * 1e6),
                                               fflops / (FP32_TFLOPS * 1e6))
        rows.setdefault(label, []).append((us, roof))
    out = []
    for label, v in rows.items():
        us, roof = statistics.mean(x[0] for x in v), v[0][1]
        out.append(dict(op=label, calls=len(v), us=round(us, 1), **({} if roof is None else
                                                                    {"roofline_us": round(roof, 1), "fraction": round(roof / us, 3)})))
    return sorted(out, key=lambda r: -r["us"] * r["calls"])


def timed(fn, reps: int = 5, warmup: int = 3) -> float:
    for _ in range(warmup):
        fn()
    ms = []
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        ms.append(e0.elapsed_time(e1))
    return statistics.median(ms)


# ----------------------------------------------------------------------------- the two models
def measure_design(pkg, cfg, s: dict, peaks: dict, prompts, batches, context: int, tables: int) -> dict:
    max_seqs, max_len = max(batches), context + 512
    max_tokens = max(n * l for n, l in prompts)
    max_len = max(max_len, max(l for _, l in prompts))
    config = pkg.Config(max_num_seqs=max_seqs, max_model_len=max_len, max_num_batched_tokens=max(max_tokens, max_len),
                        num_kvcache_blocks=max_seqs * ((max_len + 255) // 256), decoder_config=cfg)
    runner = pkg.CausalModelRunner(config)
    pages = (max_len + 255) // 256

    def seqs(n, length, done):
        out = []
        for i in range(n):
            q = pkg.CausalSequence(torch.randint(0, s["vocab"], (length,), generator=torch.Generator().manual_seed(i)).tolist())
            q.block_table, q.state_slot, q.num_cached_tokens = list(range(i * pages, (i + 1) * pages)), i, done
            out.append(q)
        return out

    # random weights route unevenly: experts with work in the last table's step, for the byte counts
    res = {"prefill": {}, "decode": {}, "weights_gb": round(runner.weights.nbytes() / 1e9, 2)}
    eng = runner.engine
    for n, length in prompts:
        batch = seqs(n, length, 0)
        ms = timed(lambda: runner.execute(batch, [length] * n))
        res["prefill"][f"{n} x {length}"] = {"ms": round(ms, 3), "tokens_per_s": round(n * length / ms * 1e3)}
    for bs in batches:
        batch = seqs(bs, context + 1, context)
        ms = timed(lambda: runner.execute(batch, [1] * bs), reps=9)
        res["decode"][f"{bs} requests at {context}"] = {"ms": round(ms, 4), "tokens_per_s": round(bs / ms * 1e3)}
    if tables:
        n, length = prompts[-1]
        with torch.inference_mode():
            for label, batch, counts in ((f"prefill {n} x {length}", seqs(n, length, 0), [length] * n),
                                         (f"decode {tables} at {context}", seqs(tables, context + 1, context), [1] * tables)):
                graphs, runner.graphs = runner.graphs, {}
                with Recorder(pkg.ops) as rec:
                    runner.execute(batch, counts)
                runner.graphs = graphs
                ids = [a[0] for nm, _, a, _ in rec.calls if nm == "moe_plan"]
                ctx = dict(rows=sum(counts), top=s["top"], touched=int(torch.unique(ids[-1]).numel()) if ids else 0)
                res[label] = op_table(rec, peaks, ctx)
    assert pkg._lib.device_status(clear=True) == 0
    runner.exit()
    return res


def measure_closest(pkg, s: dict, peaks: dict, prompts, requests, context: int, tables: bool) -> dict:
    block, mask = 32, s["vocab"] - 1
    max_len = max(context + 512, max(l for _, l in prompts) + block)
    max_seqs = max(max(requests), max(n for n, _ in prompts))
    pages = (max_len + block + 255) // 256
    config = pkg.Config(max_num_seqs=max_seqs, max_model_len=max_len, max_num_batched_tokens=max(n * l for n, l in prompts) + max_len,
                        num_kvcache_blocks=max_seqs * pages, decoder_config=closest_config(pkg, s), mask_token_id=mask, block_size=block,
                        launch_ahead=False)
    runner = pkg.ModelRunner(config)

    def seqs(n, length):
        out = []
        for i in range(n):
            ids = torch.randint(0, s["vocab"] - 1, (length,), generator=torch.Generator().manual_seed(i)).tolist()
            q = pkg.Sequence(ids, pkg.SamplingParams(ignore_eos=True), denoising_block_size=block, mask_token_id=mask)
            q.block_table = list(range(i * pages, (i + 1) * pages))
            out.append(q)
        return out

    res = {"prefill": {}, "decode": {}}
    for n, length in prompts:
        batch = seqs(n, length)

        def prefill():
            for q in batch:
                q.current_denoising_block = q._fresh_block()
            runner.run(batch, True)
        ms = timed(prefill)
        res["prefill"][f"{n} x {length}"] = {"ms": round(ms, 3), "tokens_per_s": round(n * length / ms * 1e3)}
    for bs in requests:
        batch = seqs(bs, context)

        def step():
            for q in batch:
                q.current_denoising_block = q._fresh_block()
            runner.run(batch, False)
        ms = timed(step, reps=9)
        res["decode"][f"{bs} requests x {block} rows at {context}"] = {"ms": round(ms, 4), "rows_per_s": round(bs * block / ms * 1e3)}
    if tables:
        n, length = prompts[-1]
        for label, batch, is_prefill in ((f"prefill {n} x {length}", seqs(n, length), True), (f"decode 1 x {block} rows at {context}", seqs(1, context), False)):
            runner.enforce_eager = True
            with Recorder(pkg.ops) as rec:
                runner.run(batch, is_prefill)
            runner.enforce_eager = False
            res[label] = op_table(rec, peaks, {"rows": 0, "top": 0, "touched": 0})
    runner.exit()
    return res


def main(pkg, size: str, peaks: dict, sampler, which: str = "hybrid") -> dict:
    s = SIZES[size]
    peaks = {"hbm_gbs": float(peaks.get("hbm_gbs", HBM_GBS)), "bf16_tflops": float(peaks.get("bf16_tflops", BF16_TFLOPS)),
             "source": "measured" if peaks else "fallback", "fp32_tflops": round(FP32_TFLOPS, 1)}
    prompts, context = [(1, 1024), (1, 4096), (4, 2048)], 2048
    sampler.start()
    cfg = {"hybrid": design_config, "nipadra": nipadra_config}[which](pkg, s)
    design = measure_design(pkg, cfg, s, peaks, prompts, [1, 32, 128], context, tables=32)
    torch.cuda.empty_cache()
    hybrid = {}
    if which == "nipadra":
        hybrid["closest_causal"] = measure_design(pkg, dense_hybrid_config(pkg, s), s, peaks, prompts, [1, 32, 128], context, tables=32)
        torch.cuda.empty_cache()
    closest = measure_closest(pkg, s, peaks, prompts, [1, 4], context, tables=True)
    clocks = sampler.stop()
    return {"metric": f"{which} decoder design: decoded tokens/s, 32 requests", "unit": "tokens/s",
            "value": design["decode"][f"32 requests at {context}"]["tokens_per_s"], "higher_is_better": True, "dtype": "bf16",
            "data": "synthetic tokens, random weights", "n_gpus": 1, "peaks": peaks, "clocks": clocks,
            "config": {"model": f"8 {which} layers beside 8 block-diffusion layers, size {size}", **s,
                       "l2_policy": "operations: 256 MB written before each call; steps: weights exceed L2"},
            "design": design, **hybrid, "closest": closest}


if __name__ == "__main__":
    sys.exit("run: python bench.py --design hybrid")
