"""Layer stack of decoders whose layers mix recurrences, attention and experts (``HybridConfig``).

``HybridWeights`` holds the checkpoint's tensors in the layout the kernels read: every projection of a mixer that
takes the layer's normed input is stacked into one matrix, rows and columns are padded with zeros to multiples of
128, expert matrices of one layer are one tensor, and the small parameters are fp32.  ``HybridEngine.forward`` runs
the stack over a step's rows:

    residual += previous output, RMSNorm -> one GEMM for all inputs of the mixer -> mixer -> output projection
    residual += ..., RMSNorm -> feed-forward (dense, or router -> plan -> gather -> grouped GEMMs)

In designs with the norm behind the sum the same row kernel leaves norm(scale * residual + output) as the new residual.  Two
mixers side by side share the input GEMM and the output GEMM: each leaves its scaled output in its own columns of one
buffer, and the product with the joined output matrices is their sum.

The residual is fp32; activations are bf16 or, in the fp32 mode, fp32 throughout.  A step is ragged: it brings any
number of tokens of any number of sequences.  Steps of at most 64 rows leave their projections as fp32 split-k slices
that the next kernel sums; steps that bring one token per sequence take the fused one-token form of the recurrences.
Recurrent and convolution state lives in a slot per sequence, latents, keys and values in paged caches.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from . import ops
from .engine.hybrid_config import (ChannelDeltaSpec, DecayScanSpec, DenseSpec, HybridConfig, LatentAttentionSpec, MlstmSpec,
                                   MoeSpec, ParallelSpec, WindowAttentionSpec, parts_of)

PAGE = 256
SKINNY_MAX_ROWS = 64
# Prompt portions of at least this many tokens per sequence expand keys and values per head (tcgen05 attention);
# shorter ones, like decoding, attend in the latent space.
EXPAND_MIN_TOKENS = 32
# Steps with a portion of at least this many tokens run their decay scans in chunks on the tensor cores.
CHUNK_MIN_TOKENS = 8


def pad128(n: int) -> int:
    return (n + 127) // 128 * 128


def pad_head(dim: int) -> int:
    """Channels of an attention head as the paged K and V caches store them."""
    return (dim + 63) // 64 * 64


def key_parts(ctas: int, keys: int) -> int:
    """Key-range parts of an attention of ``ctas`` CTAs over up to ``keys`` keys each: about two CTAs per SM, parts of at least
    128 keys."""
    return max(1, min(296 // max(1, ctas), keys // 128, 64))


class MissingTensors(KeyError):
    pass


class _Source:
    """Checkpoint tensors by name, each to be taken exactly once and of the shape asked for (None: any size)."""

    def __init__(self, tensors: dict):
        self.tensors = tensors
        self.taken: set[str] = set()

    def __call__(self, name: str, *shape):
        if name not in self.tensors:
            raise MissingTensors(f"checkpoint lacks {name}")
        t = self.tensors[name]
        if t.dim() != len(shape) or any(s is not None and s != d for s, d in zip(shape, t.shape)):
            raise ValueError(f"{name}: checkpoint shape {tuple(t.shape)} does not fit {shape}")
        self.taken.add(name)
        return t

    def check_all_taken(self):
        left = sorted(set(self.tensors) - self.taken)
        if left:
            raise ValueError(f"{len(left)} tensors are not parameters of the configuration, first: {left[:4]}")


@dataclass
class HybridWeights:
    dtype: torch.dtype
    embed: torch.Tensor                 # [vocab, Wp]; [pad128(vocab), Wp] where it is the output matrix too
    head: torch.Tensor                  # [pad128(vocab), Wp]
    final_norm: torch.Tensor            # fp32 [Wp]
    layers: list[dict] = field(default_factory=list)

    def nbytes(self) -> int:
        tensors = [self.embed, self.final_norm] + ([] if self.head is self.embed else [self.head])
        tensors += [t for lw in self.layers for d in (lw, *lw.get("parts", ())) if d is not None for t in d.values()
                    if isinstance(t, torch.Tensor)]
        return sum(t.numel() * t.element_size() for t in tensors)

    @classmethod
    def build(cls, cfg: HybridConfig, tensors: dict, device, dtype: torch.dtype = torch.bfloat16) -> "HybridWeights":
        """``tensors``: name -> tensor in the checkpoint's names, on any device."""
        src = _Source(tensors)
        w, wp = cfg.hidden_size, pad128(cfg.hidden_size)

        def mat(t, rows: int, cols: int) -> torch.Tensor:
            out = torch.zeros(rows, cols, dtype=dtype, device=device)
            out[:t.shape[0], :t.shape[1]].copy_(t)
            return out

        def vec(t, n: int) -> torch.Tensor:
            out = torch.zeros(n, dtype=torch.float32, device=device)
            out[:t.numel()].copy_(t.reshape(-1))
            return out

        def stack(parts: list) -> tuple[torch.Tensor, list[int]]:
            """parts = (tensor [n, w], rows to reserve); returns the stacked matrix and every part's first row."""
            starts, at = [], 0
            for t, reserve in parts:
                starts.append(at)
                at += reserve
            out = torch.zeros(pad128(at), wp, dtype=dtype, device=device)
            for (t, _), s in zip(parts, starts):
                out[s:s + t.shape[0], :w].copy_(t)
            return out, starts

        def heads_cols(t, heads: int, d: int, dp: int) -> torch.Tensor:
            """Output projection [w, heads * d] with every head's columns padded to dp."""
            out = torch.zeros(wp, heads, dp, dtype=dtype, device=device)
            out[:w, :, :d].copy_(t.reshape(w, heads, d))
            return out.view(wp, heads * dp)

        def heads_rows(t, heads: int, d: int, dp: int, cols: int) -> torch.Tensor:
            out = torch.zeros(heads, dp, cols, dtype=dtype, device=device)
            out[:, :d, :t.shape[1]].copy_(t.reshape(heads, d, t.shape[1]))
            return out

        def four(n: int) -> int:
            return (n + 3) // 4 * 4

        def eight(n: int) -> int:
            return (n + 7) // 8 * 8

        def residual_norm(name: str) -> torch.Tensor:
            return vec(src(name, w).float() + cfg.design.norm_offset, wp)

        def window_attention(mx: WindowAttentionSpec, m: str) -> tuple[list, dict, torch.Tensor]:
            """(input projections, parameters, output projection) of a mixer whose tensors start with ``m``."""
            parts = [(src(m + "q", mx.heads * mx.dim, w), four(mx.heads * mx.dim)),
                     (src(m + "k", mx.kv_heads * mx.dim, w), four(mx.kv_heads * mx.dim)), (src(m + "g", mx.heads, w), four(mx.heads))]
            pairs = torch.arange(mx.rot_dims // 2, dtype=torch.float64)
            inv_freq = (mx.rot_base ** (-2.0 * pairs / max(1, mx.rot_dims))).to(device)
            params = {"q_norm": vec(src(m + "q.norm", mx.dim), four(mx.dim)), "k_norm": vec(src(m + "k.norm", mx.dim), four(mx.dim)),
                      "inv_freq": inv_freq}
            return parts, params, src(m + "o", w, mx.heads * mx.dim)

        def decay_scan(mx: DecayScanSpec, m: str) -> tuple[list, dict, torch.Tensor]:
            nv, nk = mx.heads * mx.vdim, mx.kv_heads * mx.dim
            params = {"norm": vec(src(m + "norm", nv), four(nv))}
            if mx.decay is not None:
                # in the order of the other form's inputs: gate, values, keys, queries
                parts = [(src(m + "g", nv, w), eight(nv)), (src(m + "v", nv, w), eight(nv)), (src(m + "k", nk, w), eight(nk)),
                         (src(m + "q", nk, w), eight(nk))]
                params["decay"] = torch.tensor(mx.decay, dtype=torch.float32, device=device)
                params["log_decay"] = torch.tensor(mx.decay, dtype=torch.float64).log().clamp_min(-104.0).to(device, torch.float32)
                params["step"] = torch.ones_like(params["decay"])
            else:
                z, x, b, c, dt = src(m + "in", 2 * nv + 2 * nk + mx.heads, w).split([nv, nv, nk, nk, mx.heads])
                parts = [(z, four(nv)), (x, four(nv)), (b, four(nk)), (c, four(nk)), (dt, four(mx.heads))]
                params["conv"] = src(m + "conv", nv + 2 * nk, mx.conv).to(device=device, dtype=torch.float32).contiguous()
                params["conv_bias"] = vec(src(m + "conv.b", nv + 2 * nk), four(nv + 2 * nk))
                for key, name in (("dt_bias", "dt_bias"), ("a_log", "A_log"), ("skip", "D")):
                    params[key] = vec(src(m + name, mx.heads), mx.heads)
            return parts, params, src(m + "o", w, nv)

        def joined(mixers: list) -> dict:
            """Weights of mixers that read one input and whose outputs are summed: both GEMMs are shared."""
            stacked, starts = stack([p for parts, _, _ in mixers for p in parts])
            offsets, at = [], 0
            for _, _, o in mixers:
                offsets.append(at)
                at += (o.shape[1] + 7) // 8 * 8
            out = torch.zeros(wp, pad128(at), dtype=dtype, device=device)
            subs = []
            for (parts, params, o), off in zip(mixers, offsets):
                out[:w, off:off + o.shape[1]].copy_(o)
                subs.append({**params, "starts": starts[:len(parts)], "out": off})
                starts = starts[len(parts):]
            return {"in": stacked, "o": out, "parts": subs}

        layers = []
        for i, layer in enumerate(cfg.layers):
            p, mx, lw = f"l{i}.", layer.mixer, {}
            lw["norm1"] = residual_norm(p + "norm1")
            if isinstance(mx, ParallelSpec):
                lw.update(joined([window_attention(mx.left, p + "mix.left."), decay_scan(mx.right, p + "mix.right.")]))
            elif isinstance(mx, WindowAttentionSpec):
                lw.update(joined([window_attention(mx, p + "mix.")]))
            elif isinstance(mx, DecayScanSpec):
                lw.update(joined([decay_scan(mx, p + "mix.")]))
            elif isinstance(mx, ChannelDeltaSpec):
                nq, nv = mx.kv_heads * mx.dim, mx.heads * mx.vdim
                a1, g1 = src(p + "mix.a1", None, w), src(p + "mix.g1", None, w)
                ra, rg = a1.shape[0], g1.shape[0]
                parts = [(a1, pad128(ra)), (g1, pad128(rg)), (src(p + "mix.q", nq, w), four(nq)),
                         (src(p + "mix.k", nq, w), four(nq)), (src(p + "mix.v", nv, w), four(nv)),
                         (src(p + "mix.b", mx.heads, w), four(mx.heads))]
                lw["in"], lw["starts"] = stack(parts)
                lw["a2"] = mat(src(p + "mix.a2", mx.heads * mx.dim, ra), pad128(mx.heads * mx.dim), pad128(ra))
                lw["g2"] = mat(src(p + "mix.g2", nv, rg), pad128(nv), pad128(rg))
                for name, n in (("q", nq), ("k", nq), ("v", nv)):
                    lw["conv_" + name] = src(p + f"mix.{name}.conv", n, mx.conv).to(device=device, dtype=torch.float32).contiguous()
                lw["a_log"] = vec(src(p + "mix.A_log", mx.heads), mx.heads)
                lw["dt_bias"] = vec(src(p + "mix.dt_bias", mx.heads * mx.dim), mx.heads * mx.dim)
                lw["norm"] = vec(src(p + "mix.norm", mx.vdim), mx.vdim)
                lw["o"] = mat(src(p + "mix.o", w, nv), wp, pad128(nv))
            elif isinstance(mx, MlstmSpec):
                nq, nv = mx.heads * mx.dim, mx.heads * mx.vdim
                parts = [(src(p + "mix.q", nq, w), four(nq)), (src(p + "mix.k", nq, w), four(nq)),
                         (src(p + "mix.v", nv, w), four(nv)), (src(p + "mix.g", nv, w), four(nv)),
                         (src(p + "mix.i", mx.heads, w), four(mx.heads)), (src(p + "mix.f", mx.heads, w), four(mx.heads))]
                lw["in"], lw["starts"] = stack(parts)
                lw["bias_i"] = vec(src(p + "mix.i.b", mx.heads), mx.heads)
                lw["bias_f"] = vec(src(p + "mix.f.b", mx.heads), mx.heads)
                lw["norm"] = vec(src(p + "mix.norm", nv), nv)
                lw["o"] = mat(src(p + "mix.o", w, nv), wp, pad128(nv))
            else:
                qr, kr = pad128(mx.q_rank), pad128(mx.kv_rank)
                dp, vp = pad128(mx.dim), pad128(mx.vdim)
                parts = [(src(p + "mix.dq", mx.q_rank, w), qr)]
                lw["dq_norm"] = vec(src(p + "mix.dq.norm", mx.q_rank), qr)
                if mx.kv_from is None:
                    parts.append((src(p + "mix.dkv", mx.kv_rank, w), kr))
                    lw["dkv_norm"] = vec(src(p + "mix.dkv.norm", mx.kv_rank), kr)
                lw["in"], lw["starts"] = stack(parts)
                lw["uq"] = heads_rows(src(p + "mix.uq", mx.heads * mx.dim, mx.q_rank), mx.heads, mx.dim, dp, qr).view(-1, qr)
                uk = heads_rows(src(p + "mix.uk", mx.heads * mx.dim, mx.kv_rank), mx.heads, mx.dim, dp, kr)
                uv = heads_rows(src(p + "mix.uv", mx.heads * mx.vdim, mx.kv_rank), mx.heads, mx.vdim, vp, kr)
                lw["uk_t"] = uk.transpose(1, 2).contiguous()       # [heads, kr, dp]: folds the key projection into q
                lw["uv"] = uv                                      # [heads, vp, kr]
                if dtype == torch.bfloat16 and dp == 128 and vp == 128:
                    lw["ukv"] = torch.cat([uk.view(-1, kr), uv.view(-1, kr)])      # keys and values of prompts, per head
                lw["o"] = heads_cols(src(p + "mix.o", w, mx.heads * mx.vdim), mx.heads, mx.vdim, vp)
            mlp = layer.mlp
            if mlp is not None:
                lw["norm2"] = residual_norm(p + "norm2")
            if isinstance(mlp, DenseSpec):
                fp = pad128(mlp.ff)
                lw["up"], lw["down"] = mat(src(p + "mlp.up", mlp.ff, w), fp, wp), mat(src(p + "mlp.down", w, mlp.ff), wp, fp)
                if mlp.act == "relu_glu":
                    lw["up"] = torch.cat([mat(src(p + "mlp.gate", mlp.ff, w), fp, wp), lw["up"]])
            elif isinstance(mlp, MoeSpec):
                fp = pad128(mlp.expert_ff)
                lw["router"] = mat(src(p + "mlp.router", mlp.experts, w), pad128(mlp.experts), wp)
                up = torch.zeros(mlp.experts, fp, wp, dtype=dtype, device=device)
                down = torch.zeros(mlp.experts, wp, fp, dtype=dtype, device=device)
                for e in range(mlp.experts):
                    up[e, :mlp.expert_ff, :w].copy_(src(p + f"mlp.e{e}.up", mlp.expert_ff, w))
                    down[e, :w, :mlp.expert_ff].copy_(src(p + f"mlp.e{e}.down", w, mlp.expert_ff))
                lw["e_up"], lw["e_down"] = up, down
                if mlp.shared_ff is not None:
                    sp = pad128(mlp.shared_ff)
                    lw["s_up"] = mat(src(p + "mlp.shared.up", mlp.shared_ff, w), sp, wp)
                    lw["s_down"] = mat(src(p + "mlp.shared.down", w, mlp.shared_ff), wp, sp)
            layers.append(lw)
        tied = cfg.design.tied_head
        embed = mat(src("embed", cfg.vocab_size, w), pad128(cfg.vocab_size) if tied else cfg.vocab_size, wp)
        head = embed if tied else mat(src("head", cfg.vocab_size, w), pad128(cfg.vocab_size), wp)
        out = cls(dtype, embed, head, residual_norm("final.norm"), layers)
        src.check_all_taken()
        return out

    @classmethod
    def random_init(cls, cfg: HybridConfig, seed: int, device, dtype: torch.dtype = torch.bfloat16, rank: int = 128,
                    **kw) -> "HybridWeights":
        return cls.build(cfg, random_tensors(cfg, seed, device, rank=rank, **kw), device, dtype)


def tensor_shapes(cfg: HybridConfig, rank: int = 128) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of ``cfg``; ``rank``: the low rank of the decay and gate projections."""
    w, shapes = cfg.hidden_size, {}
    shapes["embed"] = (cfg.vocab_size, w)
    for i, layer in enumerate(cfg.layers):
        p, mx, mlp = f"l{i}.", layer.mixer, layer.mlp
        shapes[p + "norm1"] = (w,)
        m = p + "mix."
        if isinstance(mx, (ParallelSpec, WindowAttentionSpec, DecayScanSpec)):
            subs = parts_of(mx)
            for sub, pre in zip(subs, (m + "left.", m + "right.") if len(subs) > 1 else (m,)):
                if isinstance(sub, WindowAttentionSpec):
                    nq, nk = sub.heads * sub.dim, sub.kv_heads * sub.dim
                    shapes.update({pre + "q": (nq, w), pre + "k": (nk, w), pre + "q.norm": (sub.dim,), pre + "k.norm": (sub.dim,),
                                   pre + "g": (sub.heads, w), pre + "o": (w, nq)})
                    continue
                nv, nk = sub.heads * sub.vdim, sub.kv_heads * sub.dim
                shapes.update({pre + "norm": (nv,), pre + "o": (w, nv)})
                if sub.decay is not None:
                    shapes.update({pre + "q": (nk, w), pre + "k": (nk, w), pre + "v": (nv, w), pre + "g": (nv, w)})
                else:
                    shapes.update({pre + "in": (2 * nv + 2 * nk + sub.heads, w), pre + "conv": (nv + 2 * nk, sub.conv),
                                   pre + "conv.b": (nv + 2 * nk,), pre + "dt_bias": (sub.heads,), pre + "A_log": (sub.heads,),
                                   pre + "D": (sub.heads,)})
        elif isinstance(mx, ChannelDeltaSpec):
            nq, nv = mx.kv_heads * mx.dim, mx.heads * mx.vdim
            for name, n in (("q", nq), ("k", nq), ("v", nv)):
                shapes[m + name], shapes[m + name + ".conv"] = (n, w), (n, mx.conv)
            shapes.update({m + "b": (mx.heads, w), m + "A_log": (mx.heads,), m + "norm": (mx.vdim,), m + "a1": (rank, w),
                           m + "a2": (mx.heads * mx.dim, rank), m + "dt_bias": (mx.heads * mx.dim,), m + "g1": (rank, w),
                           m + "g2": (nv, rank), m + "o": (w, nv)})
        elif isinstance(mx, MlstmSpec):
            nq, nv = mx.heads * mx.dim, mx.heads * mx.vdim
            shapes.update({m + "q": (nq, w), m + "k": (nq, w), m + "v": (nv, w), m + "g": (nv, w), m + "o": (w, nv),
                           m + "norm": (nv,), m + "i": (mx.heads, w), m + "i.b": (mx.heads,), m + "f": (mx.heads, w),
                           m + "f.b": (mx.heads,)})
        else:
            shapes.update({m + "dq": (mx.q_rank, w), m + "dq.norm": (mx.q_rank,), m + "uq": (mx.heads * mx.dim, mx.q_rank)})
            if mx.kv_from is None:
                shapes.update({m + "dkv": (mx.kv_rank, w), m + "dkv.norm": (mx.kv_rank,)})
            shapes.update({m + "uk": (mx.heads * mx.dim, mx.kv_rank), m + "uv": (mx.heads * mx.vdim, mx.kv_rank),
                           m + "o": (w, mx.heads * mx.vdim)})
        m = p + "mlp."
        if mlp is not None:
            shapes[p + "norm2"] = (w,)
        if isinstance(mlp, DenseSpec):
            shapes.update({m + "up": (mlp.ff, w), m + "down": (w, mlp.ff)})
            if mlp.act == "relu_glu":
                shapes[m + "gate"] = (mlp.ff, w)
        elif isinstance(mlp, MoeSpec):
            for e in range(mlp.experts):
                shapes.update({m + f"e{e}.up": (mlp.expert_ff, w), m + f"e{e}.down": (w, mlp.expert_ff)})
            shapes[m + "router"] = (mlp.experts, w)
            if mlp.shared_ff is not None:
                shapes.update({m + "shared.up": (mlp.shared_ff, w), m + "shared.down": (w, mlp.shared_ff)})
    shapes["final.norm"] = (w,)
    if not cfg.design.tied_head:
        shapes["head"] = (cfg.vocab_size, w)
    return shapes


def random_tensors(cfg: HybridConfig, seed: int, device, rank: int = 128, std: float | None = None) -> dict[str, torch.Tensor]:
    """Seeded checkpoint: matrices N(0, std) (std None: 1 / sqrt(columns)), norms around 1, decays of moderate length."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        if name.endswith(("norm1", "norm2", "final.norm")):
            t = 1.0 - cfg.design.norm_offset + 0.1 * t
        elif name.endswith("norm") or ".norm" in name:
            t = 1.0 + 0.1 * t
        elif name.endswith("A_log"):
            t = t - 2.0
        elif name.endswith("f.b"):
            t = t + 3.0
        elif name.endswith(".D"):
            t = 1.0 + 0.3 * t
        elif name.endswith((".b", ".dt_bias")) and len(shape) == 1:
            pass
        elif name.endswith(".conv"):
            t = t * (0.5 / shape[1] ** 0.5) + 0.25
        else:
            t = t * (std if std is not None else shape[-1] ** -0.5)
        out[name] = t.to(torch.bfloat16)
    return out


@dataclass
class StepBatch:
    """Device tensors of one step (all int32 but ids).  A portion is the run of rows one sequence brings."""
    m: int
    bs: int
    ids: torch.Tensor            # int64 [m]
    row_pos: torch.Tensor        # [m] position in the sequence; -1: padding row
    row_seq: torch.Tensor        # [m] index of the row's sequence in this step
    slots: torch.Tensor          # [m] latent-cache row; -1: padding row
    cu_q: torch.Tensor           # [bs + 1]
    cu_k: torch.Tensor           # [bs + 1] context lengths after the step, summed
    start: torch.Tensor          # [bs] position of the first token brought
    state_slot: torch.Tensor     # [bs]; -1: padding
    table: torch.Tensor          # [bs, pages]
    max_q: int                   # longest portion
    total_k: int                 # cu_k[-1]; 0 in steps of one token per sequence
    max_ctx: int = 1             # longest context after the step (a bound)


class HybridEngine:

    def __init__(self, cfg: HybridConfig, weights: HybridWeights, num_pages: int, num_slots: int, max_tokens: int, device):
        self.cfg, self.w, self.device = cfg, weights, torch.device(device)
        self.dtype = weights.dtype
        self.max_tokens = max_tokens
        self.width_pad = pad128(cfg.hidden_size)
        self.num_pages, self.num_slots = num_pages, num_slots
        self._bufs: dict[tuple, torch.Tensor] = {}
        self._outgrown: list[torch.Tensor] = []
        self._one_token = False                  # the step in progress brings one token per sequence
        self.collect: list | None = None         # tests: receives the residual after every layer
        self.latents: dict[int, torch.Tensor] = {}
        self.kv: dict[int, tuple] = {}
        self.state: dict[int, dict] = {}
        for i, layer in enumerate(cfg.layers):
            for mx in parts_of(layer.mixer):
                caches = [torch.zeros(num_pages * PAGE, *shape, dtype=self.dtype, device=device) for shape in cache_shapes(mx)]
                if isinstance(mx, WindowAttentionSpec):
                    self.kv[i] = tuple(caches)
                elif caches:
                    self.latents[i] = caches[0]
                if state_shapes(mx, self.dtype):
                    self.state[i] = {k: torch.zeros(num_slots, *shape, dtype=dt, device=device)
                                     for k, (shape, dt) in state_shapes(mx, self.dtype).items()}
        self.residual = torch.zeros(max_tokens, self.width_pad, dtype=torch.float32, device=device)

    # ------------------------------------------------------------------ buffers
    def buf(self, name: str, m: int, *cols, dtype=None) -> torch.Tensor:
        """Rows [0, m) of a named activation buffer, allocated on first use for the longest step.  Buffers are zeroed
        then, so that padding columns no kernel writes stay zero: a name must not be shared by different layouts."""
        dtype = dtype or self.dtype
        key = (name, cols, dtype)
        t = self._bufs.get(key)
        if t is None:
            t = self._bufs[key] = torch.zeros(self.max_tokens, *cols, dtype=dtype, device=self.device)
        return t[:m]

    def scratch(self, name: str, n: int, dtype) -> torch.Tensor:
        """n elements of a named work buffer that grows with demand.  One-token steps have their own set, whose outgrown
        buffers are kept: captured graphs may still point at them."""
        key = (name, self._one_token, dtype)
        t = self._bufs.get(key)
        if t is None or t.numel() < n:
            if t is not None and self._one_token:
                self._outgrown.append(t)
            t = self._bufs[key] = torch.empty(n, dtype=dtype, device=self.device)
        return t[:n]

    def _linear(self, name: str, x: torch.Tensor, w: torch.Tensor, parts: bool = True, f32: bool = False, silu_from: int | None = None) -> ops.Rows:
        """x w^T as its consumer takes it: split-k slices for a short bf16 step, else rows, whose columns from ``silu_from`` on
        are activated."""
        m, n = x.shape[0], w.shape[0]
        if parts and m <= SKINNY_MAX_ROWS and self.dtype == torch.bfloat16:
            ks = ops.pick_ksplit(m, n, w.shape[1])
            out = self.scratch("parts_" + name, ks * SKINNY_MAX_ROWS * n, torch.float32)[:ks * m * n].view(ks, m, n)
            ops.gemm_splitk_partials(x, w, ks, out)
            return ops.Rows(parts=out)
        out = self.buf("rows_" + name, m, n, dtype=torch.float32 if f32 else None)
        return ops.Rows(ops.gemm(x, w, out) if silu_from is None else ops.gemm(x, w, out, act=ops.ACT_SILU, act_from=silu_from))

    # ------------------------------------------------------------------ forward
    def forward(self, b: StepBatch) -> torch.Tensor:
        """Final-norm rows [m, width_pad] of the step (an internal buffer)."""
        cfg, m = self.cfg, b.m
        if m > self.max_tokens:
            raise AssertionError(f"step of {m} rows exceeds the activation buffers ({self.max_tokens} rows)")
        self._one_token = b.max_q == 1
        h = self.buf("h", m, self.width_pad)
        res = self.residual[:m]

        post = cfg.design.post_norm

        def norm(weight, **kw):
            ops.residual_norm(res, cfg.hidden_size, cfg.rms_norm_eps, self.dtype, weight=weight, out=h, **kw)

        first = self.w.final_norm if not cfg.layers else (None if post else self.w.layers[0]["norm1"])
        norm(first, ids=b.ids, embed=self.w.embed[:cfg.vocab_size], embed_scale=cfg.embed_scale)
        for i, (layer, lw) in enumerate(zip(cfg.layers, self.w.layers)):
            mx, last = layer.mixer, i + 1 == len(cfg.layers)
            if "parts" in lw:
                y = self._joined(i, mx, lw, h, b)
            elif isinstance(mx, ChannelDeltaSpec):
                y = self._channel_delta(i, mx, lw, h, b)
            elif isinstance(mx, MlstmSpec):
                y = self._mlstm(i, mx, lw, h, b)
            else:
                y = self._latent_attention(i, mx, lw, h, b)
            after = {"add": (y,)}

            def feed_forward():
                return self._dense(layer.mlp, lw, h) if isinstance(layer.mlp, DenseSpec) else self._moe(layer.mlp, lw, h, b)

            if post:
                # every sum is normalised into the residual; the last one also meets the final norm
                behind = dict(post=True, res_scale=cfg.residual_scale)
                final = self.w.final_norm if last else None
                norm(lw["norm1"], weight2=final if layer.mlp is None else None, **behind, **after)
                if layer.mlp is not None:
                    norm(lw["norm2"], weight2=final, **behind, **feed_forward())
            else:
                if layer.mlp is not None:
                    norm(lw["norm2"], **after)
                    after = feed_forward()
                norm(self.w.final_norm if last else self.w.layers[i + 1]["norm1"], **after)
            if self.collect is not None:
                self.collect.append(res[:, :cfg.hidden_size].clone())
        return h

    def logits(self, rows: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        """fp32 logits [n, pad128(vocab)] of final-norm rows."""
        return ops.gemm(rows, self.w.head, out)

    # ------------------------------------------------------------------ mixers
    def _portions(self, b: StepBatch):
        return b.row_seq, b.cu_q, b.start, b.state_slot

    def _joined(self, li: int, mx, lw: dict, h: torch.Tensor, b: StepBatch) -> ops.Rows:
        """One mixer, or several side by side, on one input product; their outputs meet in one output product."""
        scales = (mx.left_scale, mx.right_scale) if isinstance(mx, ParallelSpec) else (1.0,)
        # plain projections of a chunked scan take their silu in the product's epilogue and go into the scan as they are
        silu_from = None
        if isinstance(mx, DecayScanSpec) and mx.decay is not None and mx.dim % 8 == 0 and self._chunks(mx, b) and b.m > SKINNY_MAX_ROWS:
            silu_from = lw["parts"][0]["starts"][1]
        x = self._linear("mix_in", h, lw["in"], silu_from=silu_from)
        widths = tuple(part.heads * (part.dim if isinstance(part, WindowAttentionSpec) else part.vdim) for part in parts_of(mx))
        y = self.buf("joined_o_" + "_".join(map(str, widths)), b.m, lw["o"].shape[1])
        for part, pw, n, scale in zip(parts_of(mx), lw["parts"], widths, scales):
            run = self._window_attention if isinstance(part, WindowAttentionSpec) else self._decay_scan
            run(li, part, pw, x, y[:, pw["out"]:pw["out"] + n], scale, b, **({} if silu_from is None else {"activated": True}))
        return self._linear("mix_out", y, lw["o"])

    def _window_attention(self, li: int, mx: WindowAttentionSpec, pw: dict, x: ops.Rows, y: torch.Tensor, scale: float, b: StepBatch):
        m, (k_cache, v_cache) = b.m, self.kv[li]
        q0, k0, g0 = pw["starts"]
        q = self.buf(f"window_q_{mx.dim}", m, mx.heads, k_cache.shape[2])
        ops.rotary_commit(x.cols(q0), x.cols(k0), x.cols(k0), mx.heads, mx.kv_heads, mx.dim, pw["q_norm"], pw["k_norm"],
                          self.cfg.rms_norm_eps, pw["inv_freq"], b.row_pos, b.slots, q, k_cache, v_cache)
        keys = min(b.max_ctx, mx.window) if mx.window else b.max_ctx
        nsplit = key_parts(m * mx.kv_heads * -(-mx.heads // mx.kv_heads // 16), keys)
        ws = self.scratch("window_ws", max(16, ops.window_attn_workspace_bytes(m, mx.heads, q.shape[2], nsplit)), torch.uint8)
        ops.window_attn(q, k_cache, v_cache, b.table, self._portions(b), b.row_pos, b.max_q, mx.dim, mx.window, mx.sink, mx.scale, y,
                        gate=x.cols(g0), out_scale=scale, nsplit=nsplit, workspace=ws)

    def _chunks(self, mx: DecayScanSpec, b: StepBatch) -> bool:
        return self.dtype == torch.bfloat16 and b.max_q >= CHUNK_MIN_TOKENS and ops.chunk_scan_supported(ops.scan_dim_pad(mx.dim), mx.vdim)

    def _decay_scan(self, li: int, mx: DecayScanSpec, pw: dict, x: ops.Rows, y: torch.Tensor, scale: float, b: StepBatch,
                    activated: bool = False):
        m, st, f32 = b.m, self.state[li], torch.float32
        heads, kvh, dim, vdim = mx.heads, mx.kv_heads, mx.dim, mx.vdim
        dp, one_token = ops.scan_dim_pad(dim), b.max_q == 1
        chunks = self._chunks(mx, b)
        act = self.dtype if chunks else f32
        z0, v0, k0, q0, *dt0 = pw["starts"]
        o = self.buf("scan_o", m, heads, vdim, dtype=f32)

        def leave():
            # lightning attention gates behind its norm, Mamba-2 in front of it
            ops.part_norm(o.view(m, heads * vdim), x.cols(z0), pw["norm"], mx.norm_groups, mx.decay is None, self.cfg.rms_norm_eps, y,
                          out_scale=scale)

        if activated:
            rows = x.x
            ops.chunk_scan(b.bs, heads, kvh, dim, vdim, rows[:, q0:], rows[:, k0:], rows[:, v0:], pw["log_decay"], pw["step"], st["s"],
                           self._portions(b), b.max_q, o)
            return leave()
        outs = (self.buf("scan_q", m, kvh, dp, dtype=act), self.buf("scan_k", m, kvh, dp, dtype=act),
                self.buf("scan_v", m, heads, vdim, dtype=act), self.buf("scan_s0", m, heads, dtype=f32),
                self.buf("scan_s1", m, heads, dtype=f32))
        scalars = dict(decay=pw["decay"]) if mx.decay is not None else dict(
            dt=x.cols(dt0[0]), a_log=pw["a_log"], dt_bias=pw["dt_bias"], conv=pw["conv"], conv_bias=pw["conv_bias"],
            conv_state=st["conv"], shift_state=one_token)
        ops.decay_prep(self.dtype, m, b.bs, heads, kvh, dim, vdim, x.cols(q0), x.cols(k0), x.cols(v0), self._portions(b), outs, **scalars)
        if chunks:
            q, k, v, *scalars = outs
            ops.chunk_scan(b.bs, heads, kvh, dp, vdim, q.view(m, -1), k.view(m, -1), v.view(m, -1), *scalars, st["s"], self._portions(b),
                           b.max_q, o, skip=pw.get("skip"))
        else:
            ops.scan(ops.SCAN_DECAY, self.dtype, b.bs, heads, kvh, dim, vdim, *outs, st["s"], self._portions(b), out=o,
                     skip=pw.get("skip"), one_token=one_token and ops.scan_fusable(dp, vdim))
        leave()

    def _channel_delta(self, li: int, mx: ChannelDeltaSpec, lw: dict, h: torch.Tensor, b: StepBatch) -> ops.Rows:
        m, st, f32 = b.m, self.state[li], torch.float32
        heads, kvh, dim, vdim = mx.heads, mx.kv_heads, mx.dim, mx.vdim
        dp, eps = ops.scan_dim_pad(dim), self.cfg.rms_norm_eps
        a0, g0, q0, k0, v0, b0 = lw["starts"]
        fused = b.max_q == 1 and ops.scan_fusable(dp, vdim)
        x = self._linear("mix_in", h, lw["in"])
        low = self.buf("delta_low", m, q0) if x.parts is not None else x.x[:, :q0]     # a1 | g1 columns as GEMM input
        outs = (self.buf("scan_q", m, kvh, dp, dtype=f32), self.buf("scan_k", m, kvh, dp, dtype=f32),
                self.buf("scan_v", m, heads, vdim, dtype=f32), self.buf("scan_s0", m, heads, dtype=f32))
        ops.delta_prep(self.dtype, m, b.bs, heads, kvh, dim, vdim, x.cols(q0), x.cols(k0), x.cols(v0), x.cols(b0),
                       (lw["conv_q"], lw["conv_k"], lw["conv_v"]), st["conv"], self._portions(b), outs, b.max_q == 1,
                       copy=x if x.parts is not None else None, copy_out=low if x.parts is not None else None)
        q, k, v, beta = outs
        raw = ops.gemm(low[:, a0:g0], lw["a2"], self.buf("delta_raw", m, lw["a2"].shape[0], dtype=f32))
        gate = self._linear("delta_gate", low[:, g0:q0], lw["g2"], parts=fused)
        y = self.buf(f"mix_o_{heads * vdim}", m, lw["o"].shape[1])
        common = (ops.SCAN_DELTA, self.dtype, b.bs, heads, kvh, dim, vdim, q, k, v, beta, None, st["s"], self._portions(b))
        if fused:
            ops.scan(*common, eps=eps, raw_decay=ops.Rows(raw), a_log=lw["a_log"], dt_bias=lw["dt_bias"], gate=gate,
                     norm=lw["norm"], y=y)
        else:
            g = self.buf("scan_g", m, heads, dp, dtype=f32)
            scalars = self.buf("scan_scalars", m, heads, 4, dtype=f32)
            ops.channel_decay(raw, lw["a_log"], lw["dt_bias"], q, k, beta, self._portions(b), g, scalars, dim)
            o = self.buf("scan_o", m, heads, vdim, dtype=f32)
            ops.scan(*common, g=g, scalars=scalars, out=o)
            ops.gated_norm(o, gate, lw["norm"], False, eps, y)
        return self._linear("mix_out", y, lw["o"])

    def _mlstm(self, li: int, mx: MlstmSpec, lw: dict, h: torch.Tensor, b: StepBatch) -> ops.Rows:
        m, st, f32 = b.m, self.state[li], torch.float32
        heads, dim, vdim = mx.heads, mx.dim, mx.vdim
        dp, eps = ops.scan_dim_pad(dim), self.cfg.rms_norm_eps
        q0, k0, v0, g0, i0, f0 = lw["starts"]
        fused = b.max_q == 1 and ops.scan_fusable(dp, vdim)
        x = self._linear("mix_in", h, lw["in"])
        outs = (self.buf("scan_q", m, heads, dp, dtype=f32), self.buf("scan_k", m, heads, dp, dtype=f32),
                self.buf("scan_v", m, heads, vdim, dtype=f32), self.buf("scan_s0", m, heads, dtype=f32),
                self.buf("scan_s1", m, heads, dtype=f32))
        ops.mlstm_prep(self.dtype, m, heads, dim, vdim, x.cols(q0), x.cols(k0), x.cols(v0), x.cols(i0), x.cols(f0),
                       lw["bias_i"], lw["bias_f"], mx.gate_cap, outs)
        y = self.buf(f"mix_o_{heads * vdim}", m, lw["o"].shape[1])
        args = (ops.SCAN_MLSTM, self.dtype, b.bs, heads, heads, dim, vdim, *outs, st["s"], self._portions(b))
        if fused:
            ops.scan(*args, eps=eps, gate=x.cols(g0), norm=lw["norm"], per_head_norm=True, y=y, mstate=st["m"])
        else:
            o = self.buf("scan_o", m, heads, vdim, dtype=f32)
            den = self.buf("scan_den", m, heads, dtype=f32)
            ops.scan(*args, out=o, den=den, mstate=st["m"])
            ops.gated_norm(o, x.cols(g0), lw["norm"], True, eps, y, den=den)
        return self._linear("mix_out", y, lw["o"])

    def _latent_attention(self, li: int, mx: LatentAttentionSpec, lw: dict, h: torch.Tensor, b: StepBatch) -> ops.Rows:
        m, heads, eps = b.m, mx.heads, self.cfg.rms_norm_eps
        cache = self.latents[li if mx.kv_from is None else mx.kv_from]
        kr, qr = cache.shape[1], lw["uq"].shape[1]
        vp, dp = lw["uv"].shape[1], lw["uk_t"].shape[2]
        x = self._linear("mix_in", h, lw["in"])
        cq = self.buf("latent_q", m, qr)
        segments = [ops.rms_segment(x.cols(lw["starts"][0]), mx.q_rank, qr, lw["dq_norm"], eps, cq)]
        if mx.kv_from is None:
            segments.append(ops.rms_segment(x.cols(lw["starts"][1]), mx.kv_rank, kr, lw["dkv_norm"], eps, cache, slots=b.slots))
        ops.rms_rows(segments, m, self.dtype)
        q = ops.gemm(cq, lw["uq"], self.buf("attn_q", m, heads * dp))
        o = self.buf("attn_o", m, heads * vp)
        if "ukv" in lw and b.max_q >= EXPAND_MIN_TOKENS:
            c = self.scratch("latent_ctx", b.total_k * kr, self.dtype).view(b.total_k, kr)
            ops.gather_latents(cache, b.table, b.cu_k, b.bs, c)
            n = lw["ukv"].shape[0]
            kv = self.scratch("attn_kv", b.total_k * n, self.dtype).view(b.total_k, n)
            ops.gemm(c, lw["ukv"], kv)
            k, v = kv[:, :heads * 128].unflatten(1, (heads, 128)), kv[:, heads * 128:].unflatten(1, (heads, 128))
            ops.causal_attn_varlen(q.view(m, heads, 128), k, v, b.cu_q, b.cu_k, b.bs, b.max_q, mx.scale, o.view(m, heads, 128))
        else:
            ql = ops.gemm_heads(q, lw["uk_t"], self.buf("latent_qk", m, heads * kr))
            ol = self.buf("latent_o", m, heads * kr)
            nsplit = key_parts(m * -(-heads // 16), b.max_ctx)
            ws = self.scratch("latent_ws", max(16, ops.latent_attn_workspace_bytes(m, heads, kr, nsplit)), torch.uint8)
            ops.latent_attn(ql, cache, b.table, b.row_seq, b.row_pos, heads, mx.scale, ol, nsplit, ws)
            ops.gemm_heads(ol, lw["uv"], o)
        return self._linear("mix_out", o, lw["o"])

    # ------------------------------------------------------------------ feed-forward
    def _dense(self, mlp: DenseSpec, lw: dict, h: torch.Tensor) -> dict:
        act = ops.gemm(h, lw["up"], self.buf("ff_act", h.shape[0], lw["down"].shape[1]),
                       act=ops.ACT_RELU_GLU if mlp.act == "relu_glu" else ops.ACT_RELU2)
        return {"add": (self._linear("ff_out", act, lw["down"]),)}

    def _moe(self, mlp: MoeSpec, lw: dict, h: torch.Tensor, b: StepBatch) -> dict:
        m, i32 = b.m, torch.int32
        z = self._linear("router", h, lw["router"], f32=True)
        ids = self.buf("moe_ids", m, mlp.top, dtype=i32)
        weights = self.buf("moe_w", m, mlp.top, dtype=torch.float32)
        slots = self.buf("moe_slot", m, mlp.top, dtype=i32)
        ops.moe_route(z, m, mlp.experts, mlp.top, mlp.groups, mlp.keep, ids, weights, row_slot=b.slots)
        tiles = ops.moe_max_tiles(m, mlp.top, mlp.experts)
        row_token = self.scratch("moe_row_token", tiles * 128, i32)
        tile_expert = self.scratch("moe_tile_expert", tiles, i32)
        num_tiles = self.scratch("moe_num_tiles", 4, i32)
        ops.moe_plan(ids, mlp.experts, tiles, slots, row_token, tile_expert, num_tiles)
        rows, wp, fp = tiles * 128, self.width_pad, lw["e_up"].shape[1]
        xs = self.scratch("moe_x", rows * wp, self.dtype).view(rows, wp)
        act = self.scratch("moe_act", rows * fp, self.dtype).view(rows, fp)
        ys = self.scratch("moe_y", rows * wp, self.dtype).view(rows, wp)
        ops.moe_gather(h, xs, row_token, num_tiles, tiles)
        ops.gemm_experts(xs, lw["e_up"], act, tile_expert, num_tiles, m, act=ops.ACT_RELU2)
        ops.gemm_experts(act, lw["e_down"], ys, tile_expert, num_tiles, m)
        out = {"moe": (ys, slots, weights)}
        if mlp.shared_ff is not None:
            sact = ops.gemm(h, lw["s_up"], self.buf("shared_act", m, lw["s_up"].shape[0]), act=ops.ACT_RELU2)
            out["add"] = (self._linear("shared_out", sact, lw["s_down"]),)
        return out


def cache_shapes(mx) -> list[tuple]:
    """What a mixer keeps per token in paged caches."""
    if isinstance(mx, WindowAttentionSpec):
        return [(mx.kv_heads, pad_head(mx.dim))] * 2
    if isinstance(mx, LatentAttentionSpec) and mx.kv_from is None:
        return [(pad128(mx.kv_rank),)]
    return []


def state_shapes(mx, dtype: torch.dtype) -> dict[str, tuple]:
    """Per-slot state of a recurrent mixer: name -> (shape, dtype)."""
    if isinstance(mx, (LatentAttentionSpec, WindowAttentionSpec)):
        return {}
    dp = ops.scan_dim_pad(mx.dim)
    if isinstance(mx, ChannelDeltaSpec):
        channels = 2 * mx.kv_heads * mx.dim + mx.heads * mx.vdim
        return {"s": ((mx.heads, mx.vdim, dp), torch.float32), "conv": ((mx.conv - 1, channels), dtype)}
    if isinstance(mx, DecayScanSpec):
        shapes = {"s": ((mx.heads, mx.vdim, dp), torch.float32)}
        if mx.conv:
            shapes["conv"] = ((mx.conv - 1, 2 * mx.kv_heads * mx.dim + mx.heads * mx.vdim), dtype)
        return shapes
    blocks = ops.scan_blocks(mx.vdim)
    return {"s": ((mx.heads, mx.vdim + 1, dp), torch.float32), "m": ((mx.heads, blocks), torch.float32)}


def _bytes(shape, dtype: torch.dtype) -> int:
    n = torch.empty(0, dtype=dtype).element_size()
    for s in shape:
        n *= s
    return n


def bytes_per_page(cfg: HybridConfig, dtype: torch.dtype) -> int:
    return sum(PAGE * _bytes(shape, dtype) for l in cfg.layers for mx in parts_of(l.mixer) for shape in cache_shapes(mx))


def bytes_per_slot(cfg: HybridConfig, dtype: torch.dtype) -> int:
    return sum(_bytes(shape, dt) for l in cfg.layers for mx in parts_of(l.mixer) for shape, dt in state_shapes(mx, dtype).values())
