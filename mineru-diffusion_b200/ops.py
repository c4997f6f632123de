"""Op-level interface of the decode hot path, named after the reference ops
they stand in for.  Each function takes CUDA tensors, checks what the C ABI
cannot (dtype, device, contiguity) and calls libmdb200 on the current stream.
torch is used for memory and streams only; no function here computes in torch
and none has a fallback.
"""
from __future__ import annotations


import torch

from . import _lib

_BF16 = torch.bfloat16


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def _need(t: torch.Tensor, dtype, name: str):
    if not t.is_cuda:
        raise RuntimeError(f"{name} must be a CUDA tensor (libmdb200 has no CPU path)")
    if t.dtype != dtype:
        raise TypeError(f"{name} must be {dtype}, got {t.dtype}")


def _rows(t: torch.Tensor, name: str) -> int:
    """Row stride (elements) of a 2-D view whose last dim is dense."""
    if t.stride(-1) != 1:
        raise ValueError(f"{name}: last dimension must be contiguous")
    return t.stride(0)


OPT_PDL = 1             # programmatic dependent launch between kernels (default on)
OPT_GEMM_PAIR = 3       # many-row GEMMs on CTA pairs (tcgen05.mma.cta_group::2): 1 from 2048 rows (default), 2 from 256, 0 never
OPT_WAIT_LIMIT_US = 4   # bound of every in-kernel wait in microseconds (default 2 s); expiry raises status bit 16


def set_option(option: int, value: int) -> None:
    _lib.check(_lib.lib().mdb_set_option(option, value), "mdb_set_option")


def get_option(option: int) -> int:
    return int(_lib.lib().mdb_get_option(option))


def pick_ksplit(m: int, n: int, k: int) -> int:
    """Split-k factor suited to the kernel that (m, n, k) will run on."""
    return int(_lib.lib().mdb_gemm_pick_ksplit(m, n, k))


# --------------------------------------------------------------------------
def store_kvcache(key: torch.Tensor, value: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                  slot_mapping: torch.Tensor) -> None:
    """``store_kvcache`` of the reference (nanovllm/layers/attention.py:33-40):
    key/value [N, Hkv, D] (or [bs, B, Hkv, D]), caches [pages, 256, Hkv, D],
    slot_mapping int32 with -1 = skip."""
    if key.dim() == 4:
        key = key.reshape(-1, *key.shape[2:])
        value = value.reshape(-1, *value.shape[2:])
    slot_mapping = slot_mapping.reshape(-1)
    n, h, d = key.shape
    for t, nm in ((key, "key"), (value, "value"), (k_cache, "k_cache"), (v_cache, "v_cache")):
        _need(t, _BF16, nm)
    _need(slot_mapping, torch.int32, "slot_mapping")
    if not (key.stride(-1) == 1 and value.stride(-1) == 1 and key.stride(1) == d and value.stride(1) == d):
        raise ValueError("key/value heads must be densely packed")
    if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise ValueError("caches must be contiguous")
    if slot_mapping.numel() != n:
        raise ValueError("slot_mapping must have one entry per row")
    num_slots = k_cache.numel() // (h * d)
    _lib.check(_lib.lib().mdb_kv_commit(key.data_ptr(), key.stride(0), value.data_ptr(), value.stride(0),
                                        k_cache.data_ptr(), v_cache.data_ptr(), slot_mapping.data_ptr(), n, h * d,
                                        num_slots, _stream()), "mdb_kv_commit")


def default_nsplit(bs: int, block: int, hq: int, hkv: int, max_ctx: int) -> int:
    """Key-range parts per request.  Measured on B200 over 1..32 requests and
    contexts of 0.6K..8K: the best part count fills the 148 SMs once and no
    more (a second wave of parts costs more than it saves, and from about 16
    requests up any split loses), with at most 16 parts; the kernels
    themselves never make a part shorter than 256 keys."""
    group = hq // hkv
    tokens_per_cta = max(1, min(block, (64 if group * block <= 64 else 128) // group))
    ctas = max(1, bs * hkv * -(-block // tokens_per_cta))
    want = 148 // ctas
    parts = max(1, max_ctx // 256)
    return int(max(1, min(want, parts, 16)))


def attn_workspace_bytes(bs: int, block: int, hq: int, nsplit: int) -> int:
    """Scratch bytes ``block_attn_with_kvcache`` needs for ``nsplit`` key-range parts (0 for one part)."""
    return int(_lib.lib().mdb_attn_paged_workspace_bytes(bs, block, hq, nsplit))


def _block_attn_args(q, k_cache, v_cache, cache_seqlens, block_table, out):
    """Shape, type and layout checks shared by the two paged-attention wrappers:
    the kernels hard-code head size 128 and 256-token pages and index the page
    table with unit stride inside a row."""
    if q.dim() != 4 or k_cache.dim() != 4:
        raise ValueError("q must be [bs, block, Hq, 128] and the caches [pages, 256, Hkv, 128]")
    bs, block, hq, d = q.shape
    pages, page, hkv, d2 = k_cache.shape
    if d != 128 or d2 != 128 or page != 256:
        raise ValueError("head_dim must be 128 and pages 256 tokens")
    if v_cache.shape != k_cache.shape:
        raise ValueError("k_cache and v_cache must have the same shape")
    tensors = [(q, "q"), (k_cache, "k_cache"), (v_cache, "v_cache")]
    if out is not None:
        if out.shape != q.shape:
            raise ValueError("out must have the shape of q")
        tensors.append((out, "out"))
    for t, nm in tensors:
        _need(t, _BF16, nm)
        if not t.is_contiguous():
            raise ValueError(f"{nm} must be contiguous")
    _need(cache_seqlens, torch.int32, "cache_seqlens")
    _need(block_table, torch.int32, "block_table")
    if cache_seqlens.numel() < bs or not cache_seqlens.is_contiguous():
        raise ValueError("cache_seqlens must hold one contiguous int32 per request")
    if block_table.dim() != 2 or block_table.shape[0] < bs or (block_table.shape[1] > 1 and block_table.stride(1) != 1):
        raise ValueError("block_table must be [bs, pages per request] with unit stride inside a row")
    return bs, block, hq, hkv, pages, d


def block_attn_with_kvcache(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                            cache_seqlens: torch.Tensor, block_table: torch.Tensor, softmax_scale: float | None = None,
                            nsplit: int | None = None, workspace: torch.Tensor | None = None,
                            out: torch.Tensor | None = None, max_ctx: int | None = None) -> torch.Tensor:
    """Stands in for ``flash_attn_with_kvcache(..., causal=False)`` as the
    reference calls it (nanovllm/layers/sdar_attention.py:50-55).
    q [bs, B, Hq, 128]; caches [pages, 256, Hkv, 128]."""
    bs, block, hq, hkv, pages, d = _block_attn_args(q, k_cache, v_cache, cache_seqlens, block_table, out)
    if softmax_scale is None:
        softmax_scale = d ** -0.5
    if nsplit is None:
        nsplit = default_nsplit(bs, block, hq, hkv, max_ctx if max_ctx is not None else block_table.shape[1] * 256)
    if out is None:
        out = torch.empty_like(q)
    need = _lib.lib().mdb_attn_paged_workspace_bytes(bs, block, hq, nsplit)
    if need and (workspace is None or workspace.numel() * workspace.element_size() < need):
        workspace = torch.empty(need, dtype=torch.uint8, device=q.device)
    ws_bytes = 0 if workspace is None else workspace.numel() * workspace.element_size()
    _lib.check(_lib.lib().mdb_attn_block_paged(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(),
                                               block_table.data_ptr(), block_table.stride(0), cache_seqlens.data_ptr(),
                                               bs, block, hq, hkv, pages, float(softmax_scale), nsplit,
                                               _ptr(workspace), ws_bytes, _stream()), "mdb_attn_block_paged")
    return out


def block_attn_with_kvcache_noalloc(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                                    cache_seqlens: torch.Tensor, block_table: torch.Tensor, out: torch.Tensor,
                                    softmax_scale: float | None = None, nsplit: int = 1) -> torch.Tensor:
    """``block_attn_with_kvcache`` for hosts that cannot hand over scratch memory
    (all device memory already given to the KV-cache pool, or a thread that must
    stay out of the allocator): the split partials use a fixed 8 MiB array
    inside the library, so neither this wrapper nor the call allocates -- the
    caller passes ``out``.  Raises ``MdbError`` when (bs, nsplit) need more than
    that array.  Calls share the array; keep them on one stream."""
    bs, block, hq, hkv, pages, d = _block_attn_args(q, k_cache, v_cache, cache_seqlens, block_table, out)
    if softmax_scale is None:
        softmax_scale = d ** -0.5
    _lib.check(_lib.lib().mdb_attn_block_paged_noalloc(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                                       out.data_ptr(), block_table.data_ptr(), block_table.stride(0),
                                                       cache_seqlens.data_ptr(), bs, block, hq, hkv, pages,
                                                       float(softmax_scale), nsplit, _stream()),
               "mdb_attn_block_paged_noalloc")
    return out


def sparse_attn_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens_q: torch.Tensor,
                       cu_seqlens_k: torch.Tensor, staircase_size: int = 4, max_seqlen: int | None = None,
                       out: torch.Tensor | None = None) -> torch.Tensor:
    """``sparse_attn_varlen`` of the reference
    (nanovllm/kernels/triton/attention/block_prefill_attention_v2.py:201-202):
    q [N, Hq, 128], k/v [N, Hkv, 128] packed; cu_seqlens int32 [nseq+1]."""
    n, hq, d = q.shape
    hkv = k.shape[1]
    if d != 128:
        raise ValueError("head_dim must be 128")
    if staircase_size not in (1, 2, 4, 8, 16, 32, 64, 128):
        raise AssertionError("staircase_size must be a power of two up to 128")
    for t, nm in ((q, "q"), (k, "k"), (v, "v")):
        _need(t, _BF16, nm)
        if t.stride(-1) != 1 or t.stride(1) != d:
            raise ValueError(f"{nm}: heads must be densely packed")
    _need(cu_seqlens_q, torch.int32, "cu_seqlens_q")
    if cu_seqlens_k is not cu_seqlens_q and cu_seqlens_k.data_ptr() != cu_seqlens_q.data_ptr():
        # the reference kernel assumes q and k lengths agree (self-attention)
        if not torch.equal(cu_seqlens_q, cu_seqlens_k):
            raise ValueError("query and key lengths must agree")
    nseq = cu_seqlens_q.numel() - 1
    if max_seqlen is None:
        max_seqlen = int((cu_seqlens_q[1:] - cu_seqlens_q[:-1]).max().item()) if nseq > 0 else 0
    if out is None:
        out = torch.empty((n, hq, d), dtype=_BF16, device=q.device)
    _lib.check(_lib.lib().mdb_attn_staircase_varlen(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(),
                                                    v.stride(0), out.data_ptr(), out.stride(0),
                                                    cu_seqlens_q.data_ptr(), nseq, max_seqlen, n, hq, hkv,
                                                    staircase_size, _stream()), "mdb_attn_staircase_varlen")
    return out


def linear(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``F.linear(x, weight)`` without bias for bf16 [.., K] x [N, K]."""
    _need(x, _BF16, "x")
    _need(weight, _BF16, "weight")
    if not weight.is_contiguous():
        raise ValueError("weight must be contiguous")
    lead = x.shape[:-1]
    x2 = x.reshape(-1, x.shape[-1])
    m, k = x2.shape
    n = weight.shape[0]
    if out is None:
        out = torch.empty((m, n), dtype=_BF16, device=x.device)
    _lib.check(_lib.lib().mdb_gemm_bf16(x2.data_ptr(), _rows(x2, "x"), weight.data_ptr(), out.data_ptr(),
                                        _rows(out, "out"), m, n, k, _stream()), "mdb_gemm_bf16")
    return out.reshape(*lead, n)


def gemm_splitk_partials(x: torch.Tensor, weight: torch.Tensor, ksplit: int, partials: torch.Tensor | None = None):
    """fp32 split-k slices [ksplit, m, n] of x W^T (m <= 64)."""
    m, k = x.shape
    n = weight.shape[0]
    if partials is None:
        partials = torch.empty((ksplit, m, n), dtype=torch.float32, device=x.device)
    _lib.check(_lib.lib().mdb_gemm_splitk_partials(x.data_ptr(), _rows(x, "x"), weight.data_ptr(), partials.data_ptr(),
                                                   m, n, k, ksplit, _stream()), "mdb_gemm_splitk_partials")
    return partials


def gateup_swiglu(x: torch.Tensor, w_gate_up: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """gate_up projection + SiLU*mul in one pass over the weight (m <= 64)."""
    m, k = x.shape
    inter = w_gate_up.shape[0] // 2
    if out is None:
        out = torch.empty((m, inter), dtype=_BF16, device=x.device)
    _lib.check(_lib.lib().mdb_gemm_gateup_swiglu(x.data_ptr(), _rows(x, "x"), w_gate_up.data_ptr(), out.data_ptr(),
                                                 _rows(out, "out"), m, inter, k, _stream()), "mdb_gemm_gateup_swiglu")
    return out


def silu_and_mul(x: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``SiluAndMul`` of the reference (nanovllm/layers/activation.py:12-15)."""
    _need(x, _BF16, "x")
    x2 = x.reshape(-1, x.shape[-1])
    m, two_i = x2.shape
    inter = two_i // 2
    if out is None:
        out = torch.empty((m, inter), dtype=_BF16, device=x.device)
    _lib.check(_lib.lib().mdb_silu_mul(x2.data_ptr(), _rows(x2, "x"), out.data_ptr(), _rows(out, "out"), m, inter,
                                       _stream()), "mdb_silu_mul")
    return out.reshape(*x.shape[:-1], inter)


def add_rms_norm(x: torch.Tensor | None, residual: torch.Tensor | None, weight: torch.Tensor, eps: float,
                 partials: torch.Tensor | None = None, out: torch.Tensor | None = None,
                 residual_out: torch.Tensor | None = None):
    """``RMSNorm.forward`` of the reference (nanovllm/layers/layernorm.py:42-50).
    Input rows come from ``x`` (bf16 [m, h]) or from fp32 split-k ``partials``
    [s, m, h].  Returns (y, new_residual); without ``residual`` the new
    residual is the input row itself."""
    src = x if x is not None else partials
    m, h = src.shape[-2], src.shape[-1]
    dev = src.device
    if out is None:
        out = torch.empty((m, h), dtype=_BF16, device=dev)
    if residual_out is None:
        residual_out = torch.empty((m, h), dtype=_BF16, device=dev)
    nparts = 0 if partials is None else partials.shape[0]
    _lib.check(_lib.lib().mdb_add_rmsnorm(_ptr(x), _ptr(partials), nparts, _ptr(residual), weight.data_ptr(),
                                          float(eps), out.data_ptr(), residual_out.data_ptr(), m, h, _stream()),
               "mdb_add_rmsnorm")
    return out, residual_out


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    y, _ = add_rms_norm(x.reshape(-1, x.shape[-1]), None, weight, eps)
    return y.reshape(x.shape)


def qknorm_rope_commit(qkv: torch.Tensor | None, positions: torch.Tensor, rope_table: torch.Tensor,
                       q_norm_w: torch.Tensor, k_norm_w: torch.Tensor, eps: float, hq: int, hkv: int,
                       slot_mapping: torch.Tensor | None = None, k_cache: torch.Tensor | None = None,
                       v_cache: torch.Tensor | None = None, partials: torch.Tensor | None = None,
                       q_out: torch.Tensor | None = None, k_out: torch.Tensor | None = None,
                       v_out: torch.Tensor | None = None, want_kv: bool = False):
    """q/k per-head RMSNorm, rotary embedding and KV store after qkv_proj
    (nanovllm/models/sdar.py:74-82, nanovllm/layers/sdar_attention.py:37-38)."""
    src = qkv if qkv is not None else partials
    m = src.shape[-2]
    dev = src.device
    d = 128
    _need(positions, torch.int64, "positions")
    _need(rope_table, torch.float32, "rope_table")
    if q_out is None:
        q_out = torch.empty((m, hq, d), dtype=_BF16, device=dev)
    if want_kv and k_out is None:
        k_out = torch.empty((m, hkv, d), dtype=_BF16, device=dev)
        v_out = torch.empty((m, hkv, d), dtype=_BF16, device=dev)
    num_slots = 0 if k_cache is None else k_cache.numel() // (hkv * d)
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
    nparts = 0 if partials is None else partials.shape[0]
    _lib.check(_lib.lib().mdb_qknorm_rope_commit(_ptr(qkv), 0 if qkv is None else _rows(qkv, "qkv"), _ptr(partials),
                                                 nparts, positions.data_ptr(), rope_table.data_ptr(),
                                                 rope_table.shape[0], q_norm_w.data_ptr(), k_norm_w.data_ptr(),
                                                 float(eps), _ptr(slot_mapping), q_out.data_ptr(), _ptr(k_out),
                                                 _ptr(v_out), _ptr(k_cache), _ptr(v_cache), num_slots, m, hq, hkv,
                                                 _stream()), "mdb_qknorm_rope_commit")
    return q_out, k_out, v_out


def qkv_rope_commit_supported(m: int, k: int) -> bool:
    """Whether ``qkv_proj_rope_commit`` takes this step: many rows, on the tcgen05 kernels."""
    return m > 64 and k % 64 == 0


def qkv_proj_rope_commit(x: torch.Tensor, w_qkv: torch.Tensor, positions: torch.Tensor, rope_table: torch.Tensor,
                         q_norm_w: torch.Tensor, k_norm_w: torch.Tensor, eps: float, hq: int, hkv: int,
                         slot_mapping: torch.Tensor | None = None, k_cache: torch.Tensor | None = None,
                         v_cache: torch.Tensor | None = None, q_out: torch.Tensor | None = None,
                         k_out: torch.Tensor | None = None, v_out: torch.Tensor | None = None):
    """``qkv_proj`` + ``qknorm_rope_commit`` as one kernel for many rows
    (nanovllm/models/sdar.py:73-82, nanovllm/layers/sdar_attention.py:37-38):
    the projection output stays in tensor memory."""
    _need(x, _BF16, "x")
    _need(w_qkv, _BF16, "w_qkv")
    _need(positions, torch.int64, "positions")
    _need(rope_table, torch.float32, "rope_table")
    m, k = x.shape
    d = 128
    if w_qkv.shape[0] != (hq + 2 * hkv) * d or w_qkv.shape[1] != k:
        raise ValueError("w_qkv must be [(hq + 2 hkv) * 128, k]")
    if q_out is None:
        q_out = torch.empty((m, hq, d), dtype=_BF16, device=x.device)
    num_slots = 0 if k_cache is None else k_cache.numel() // (hkv * d)
    if slot_mapping is not None:
        _need(slot_mapping, torch.int32, "slot_mapping")
    _lib.check(_lib.lib().mdb_gemm_qkv_rope_commit(x.data_ptr(), _rows(x, "x"), w_qkv.data_ptr(), m, k,
                                                   positions.data_ptr(), rope_table.data_ptr(), rope_table.shape[0],
                                                   q_norm_w.data_ptr(), k_norm_w.data_ptr(), float(eps),
                                                   _ptr(slot_mapping), q_out.data_ptr(), _ptr(k_out), _ptr(v_out),
                                                   _ptr(k_cache), _ptr(v_cache), num_slots, hq, hkv, _stream()),
               "mdb_gemm_qkv_rope_commit")
    return q_out, k_out, v_out


def gather_rows(table: torch.Tensor, ids: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``F.embedding`` row gather for bf16 tables and int64 ids."""
    _need(table, _BF16, "table")
    _need(ids, torch.int64, "ids")
    ids = ids.reshape(-1)
    m, h = ids.numel(), table.shape[1]
    if out is None:
        out = torch.empty((m, h), dtype=_BF16, device=table.device)
    _lib.check(_lib.lib().mdb_gather_rows(table.data_ptr(), table.shape[0], ids.data_ptr(), out.data_ptr(), m, h,
                                          _stream()), "mdb_gather_rows")
    return out


def lmhead_workspace_bytes(m: int, vocab: int) -> int:
    return int(_lib.lib().mdb_lmhead_workspace_bytes(m, vocab))


def lm_head_sample(hidden: torch.Tensor, weight: torch.Tensor, temperatures: torch.Tensor, block: int,
                   noise: torch.Tensor | None = None, seed: int | None = None, step: int = 0,
                   step_dev: torch.Tensor | None = None, workspace: torch.Tensor | None = None,
                   x0: torch.Tensor | None = None, conf: torch.Tensor | None = None):
    """LM head + ``Sampler.prepare`` fused (nanovllm/layers/embed_head.py:61-72,
    nanovllm/layers/sampler.py:11-22).  hidden [m, H]; weight [V, H];
    temperatures fp32 [m // block].  Noise: explicit fp32 [m, V] tensor, or a
    ``seed`` for the counter-based generator, or neither for plain argmax.
    Returns (x0 int32 [m], confidence fp32 [m])."""
    _need(hidden, _BF16, "hidden")
    _need(weight, _BF16, "weight")
    _need(temperatures, torch.float32, "temperatures")
    m, h = hidden.shape
    vocab = weight.shape[0]
    mode = 1 if noise is not None else (2 if seed is not None else 0)
    if noise is not None:
        _need(noise, torch.float32, "noise")
        if tuple(noise.shape) != (m, vocab) or not noise.is_contiguous():
            raise ValueError("noise must be a contiguous [m, vocab] tensor")
    need = lmhead_workspace_bytes(m, vocab)
    if workspace is None or workspace.numel() * workspace.element_size() < need:
        workspace = torch.empty(need, dtype=torch.uint8, device=hidden.device)
    if x0 is None:
        x0 = torch.empty(m, dtype=torch.int32, device=hidden.device)
    if conf is None:
        conf = torch.empty(m, dtype=torch.float32, device=hidden.device)
    _lib.check(_lib.lib().mdb_lmhead_sample(hidden.data_ptr(), _rows(hidden, "hidden"), weight.data_ptr(), m, vocab, h,
                                            temperatures.data_ptr(), block, mode, _ptr(noise), int(seed or 0) & 0xFFFFFFFF,
                                            int(step) & 0xFFFFFFFF, _ptr(step_dev), workspace.data_ptr(),
                                            workspace.numel() * workspace.element_size(), x0.data_ptr(),
                                            conf.data_ptr(), _stream()), "mdb_lmhead_sample")
    return x0, conf


def logits_sample(logits: torch.Tensor, temperatures: torch.Tensor, block: int, noise: torch.Tensor | None = None,
                  seed: int | None = None, step: int = 0):
    """``Sampler.prepare`` (nanovllm/layers/sampler.py:11-22) on bf16 logits [m, V]."""
    _need(logits, _BF16, "logits")
    m, vocab = logits.shape
    mode = 1 if noise is not None else (2 if seed is not None else 0)
    need = lmhead_workspace_bytes(m, vocab)
    workspace = torch.empty(need, dtype=torch.uint8, device=logits.device)
    x0 = torch.empty(m, dtype=torch.int32, device=logits.device)
    conf = torch.empty(m, dtype=torch.float32, device=logits.device)
    _lib.check(_lib.lib().mdb_logits_sample(logits.data_ptr(), _rows(logits, "logits"), m, vocab,
                                            temperatures.data_ptr(), block, mode, _ptr(noise),
                                            int(seed or 0) & 0xFFFFFFFF, int(step) & 0xFFFFFFFF, None,
                                            workspace.data_ptr(), need, x0.data_ptr(), conf.data_ptr(), _stream()),
               "mdb_logits_sample")
    return x0, conf


def gumbel_noise(m: int, vocab: int, seed: int, step: int, device) -> torch.Tensor:
    """The noise the counter-based generator adds for (seed, step)."""
    out = torch.empty((m, vocab), dtype=torch.float32, device=device)
    _lib.check(_lib.lib().mdb_gumbel_noise(out.data_ptr(), m, vocab, seed & 0xFFFFFFFF, step & 0xFFFFFFFF, _stream()),
               "mdb_gumbel_noise")
    return out


def unmask_decide(block_ids: torch.Tensor, x0: torch.Tensor, conf: torch.Tensor, mask_id: int, threshold: float,
                  quota: int = 1, transfer: torch.Tensor | None = None, counts: torch.Tensor | None = None,
                  quotas: torch.Tensor | None = None, status_out: torch.Tensor | None = None):
    """The unmask rule of ``Sampler.forward`` (nanovllm/layers/sampler.py:28-54)
    applied in place to block_ids int64 [bs, B]; returns (transfer uint8
    [bs, B], counts int32 [bs]).  ``quotas`` int32 [bs] gives every request its own
    quota (the HF twin's schedule, mineru_diffusion/modeling_mineru_diffusion.py:617-623).  ``status_out``
    (int32 [1], device) receives the device status word and clears it."""
    _need(block_ids, torch.int64, "block_ids")
    _need(x0, torch.int32, "x0")
    _need(conf, torch.float32, "conf")
    bs, block = block_ids.shape
    if quotas is not None:
        _need(quotas, torch.int32, "quotas")
        if quotas.numel() < bs or not quotas.is_contiguous():
            raise ValueError("quotas must be a contiguous int32 tensor with one entry per request")
    if transfer is None:
        transfer = torch.empty((bs, block), dtype=torch.uint8, device=block_ids.device)
    if counts is None:
        counts = torch.empty(bs, dtype=torch.int32, device=block_ids.device)
    _lib.check(_lib.lib().mdb_unmask_decide(block_ids.data_ptr(), x0.data_ptr(), conf.data_ptr(), bs, block,
                                            int(mask_id), float(threshold), int(quota), _ptr(quotas),
                                            transfer.data_ptr(), counts.data_ptr(), _ptr(status_out), _stream()),
               "mdb_unmask_decide")
    return transfer, counts


def num_transfer_tokens(block_length: int, steps: int) -> list[int]:
    """Quota of every denoising step of a block, ``get_num_transfer_tokens`` of the HF twin
    (mineru_diffusion/modeling_mineru_diffusion.py:617-623): ``block_length // steps`` tokens per step and
    one more in each of the first ``block_length % steps`` steps.  Step ``s`` of a block uses entry
    ``min(s, steps - 1)`` (:712)."""
    if steps < 1:
        raise ValueError("denoising_steps must be positive")
    base, rem = divmod(block_length, steps)
    return [base + (1 if s < rem else 0) for s in range(steps)]


# -------------------------------------------------------------------------- tensor-parallel pair
def gemm_splitk_partials_tp(x: torch.Tensor, weight: torch.Tensor, ksplit: int, local_ptr: int, peer_ptr: int,
                            peer_flags_ptr: int, tag: int, epoch: torch.Tensor) -> None:
    """Split-k slices of x W^T written to this rank's slice range locally and, over
    NVLink, in the peer's buffer; then the peer's flag slots are raised."""
    m, k = x.shape
    n = weight.shape[0]
    _lib.check(_lib.lib().mdb_gemm_splitk_partials_tp(x.data_ptr(), _rows(x, "x"), weight.data_ptr(), local_ptr,
                                                      peer_ptr, m, n, k, ksplit, peer_flags_ptr, tag,
                                                      epoch.data_ptr(), _stream()), "mdb_gemm_splitk_partials_tp")


def linear_tp_rows(x: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, peer_ptr: int, peer_flags_ptr: int,
                   tag: int, epoch: torch.Tensor) -> int:
    """Many-row x W^T stored into ``out`` and, over NVLink, into the peer's landing buffer at ``peer_ptr``
    (same leading dimension as ``out``); then the peer's flag slots are raised.  Returns the number of
    flag slots (= CTAs launched) the consumer has to wait for."""
    import ctypes as C
    m, k = x.shape
    n = weight.shape[0]
    grid = C.c_int(0)
    _lib.check(_lib.lib().mdb_gemm_bf16_tp(x.data_ptr(), _rows(x, "x"), weight.data_ptr(), out.data_ptr(), peer_ptr,
                                           _rows(out, "out"), m, n, k, peer_flags_ptr, tag, epoch.data_ptr(),
                                           C.byref(grid), _stream()), "mdb_gemm_bf16_tp")
    return int(grid.value)


def add_rms_norm_tp_rows(x: torch.Tensor, x_peer: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float,
                         out: torch.Tensor, residual_out: torch.Tensor, wait_flags_ptr: int, wait_count: int, tag: int,
                         epoch: torch.Tensor) -> None:
    """``add_rms_norm`` of bf16(x + x_peer) after the peer's flag slots show this launch's number."""
    m, h = x.shape
    _lib.check(_lib.lib().mdb_add_rmsnorm_tp_rows(x.data_ptr(), x_peer.data_ptr(), residual.data_ptr(),
                                                  weight.data_ptr(), float(eps), out.data_ptr(), residual_out.data_ptr(),
                                                  m, h, wait_flags_ptr, wait_count, tag, epoch.data_ptr(), _stream()),
               "mdb_add_rmsnorm_tp_rows")


def tp_grid_size(m: int, n: int, k: int, ksplit: int) -> int:
    return int(_lib.lib().mdb_tp_grid_size(m, n, k, ksplit))


def add_rms_norm_tp(partials: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float,
                    out: torch.Tensor, residual_out: torch.Tensor, wait_flags_ptr: int, wait_count: int, tag: int,
                    epoch: torch.Tensor) -> None:
    """``add_rms_norm`` over [2*S, m, h] slices of both ranks after the peer's flag slots show this launch's number."""
    m, h = partials.shape[-2], partials.shape[-1]
    _lib.check(_lib.lib().mdb_add_rmsnorm_tp(None, partials.data_ptr(), partials.shape[0], residual.data_ptr(),
                                             weight.data_ptr(), float(eps), out.data_ptr(), residual_out.data_ptr(),
                                             m, h, wait_flags_ptr, wait_count, tag, epoch.data_ptr(), _stream()),
               "mdb_add_rmsnorm_tp")


def lm_head_sample_tp(hidden: torch.Tensor, weight: torch.Tensor, temperatures: torch.Tensor, block: int,
                      workspace: torch.Tensor, peer_workspace_ptr: int, tile_begin: int, tile_count: int,
                      peer_flags_ptr: int, wait_flags_ptr: int, wait_count: int, tag: int, epoch: torch.Tensor,
                      x0: torch.Tensor, conf: torch.Tensor, noise: torch.Tensor | None = None,
                      seed: int | None = None, step: int = 0, step_dev: torch.Tensor | None = None):
    """LM head + sampler statistics with the vocabulary split by 128-row tiles between the two ranks."""
    m, h = hidden.shape
    vocab = weight.shape[0]
    mode = 1 if noise is not None else (2 if seed is not None else 0)
    _lib.check(_lib.lib().mdb_lmhead_sample_tp(hidden.data_ptr(), _rows(hidden, "hidden"), weight.data_ptr(), m, vocab,
                                               h, temperatures.data_ptr(), block, mode, _ptr(noise),
                                               int(seed or 0) & 0xFFFFFFFF, int(step) & 0xFFFFFFFF, _ptr(step_dev),
                                               workspace.data_ptr(), peer_workspace_ptr,
                                               workspace.numel() * workspace.element_size(), tile_begin, tile_count,
                                               peer_flags_ptr, wait_flags_ptr, wait_count, tag, epoch.data_ptr(),
                                               x0.data_ptr(), conf.data_ptr(), _stream()), "mdb_lmhead_sample_tp")
    return x0, conf


# --------------------------------------------------------------------------
# Decoders with an fp32 residual: recurrent mixers, latent attention, experts.  Activations are bf16 or fp32 tensors.

_DTYPES = {torch.bfloat16: 0, torch.float32: 1}
ACT_NONE, ACT_RELU2, ACT_RELU_GLU, ACT_SILU = 0, 1, 2, 3


class Rows:
    """A projection's output as its consumer takes it: rows of the activation type, or the fp32 split-k slices of a
    short step, which the consumer sums and rounds.  ``cols(c)`` is the view that starts at column ``c``."""
    __slots__ = ("x", "parts", "ld", "col")

    def __init__(self, x: torch.Tensor | None = None, parts: torch.Tensor | None = None, col: int = 0, ld: int | None = None):
        self.x, self.parts, self.col = x, parts, col
        self.ld = ld if ld is not None else (x.stride(0) if x is not None else parts.shape[-1])

    def cols(self, c: int) -> "Rows":
        return Rows(self.x, self.parts, self.col + c, self.ld)

    def c(self) -> _lib.Rows:
        if self.parts is not None:
            return _lib.Rows(None, self.parts.data_ptr(), self.ld, self.parts.stride(0), self.parts.shape[0], self.col)
        return _lib.Rows(self.x.data_ptr(), None, self.ld, 0, 0, self.col)


_NO_ROWS = _lib.Rows()


def _rows_c(r: Rows | None) -> _lib.Rows:
    return _NO_ROWS if r is None else r.c()


def _act_dtype(t: torch.Tensor, name: str) -> int:
    if not t.is_cuda:
        raise RuntimeError(f"{name} must be a CUDA tensor (libmdb200 has no CPU path)")
    if t.dtype not in _DTYPES:
        raise TypeError(f"{name} must be bfloat16 or float32, got {t.dtype}")
    return _DTYPES[t.dtype]


def gemm(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: int = ACT_NONE, act_from: int = 0) -> torch.Tensor:
    """out = act(x w^T); x [m, k] (row stride free), w [n, k]; out of the activation type, or fp32.  ACT_RELU_GLU: w is
    [2 n, k], gate rows first, and out = relu(gate) * up.  ACT_SILU activates the columns from act_from on."""
    m, k = x.shape
    n = w.shape[0] // 2 if act == ACT_RELU_GLU else w.shape[0]
    a = _lib.GemmArgs(_act_dtype(x, "x"), 0, act, int(out.dtype == torch.float32), x.data_ptr(), w.data_ptr(),
                      out.data_ptr(), _rows(x, "x"), _rows(out, "out"), m, n, k, 0, 0, 0, None, None, act_from)
    _lib.check(_lib.lib().mdb_gemm(a, _stream()), "mdb_gemm")
    return out


def gemm_heads(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Head h: out[:, h n : (h + 1) n] = x[:, h k : (h + 1) k] w[h]^T; w [heads, n, k]."""
    heads, n, k = w.shape
    a = _lib.GemmArgs(_act_dtype(x, "x"), 1, 0, int(out.dtype == torch.float32), x.data_ptr(), w.data_ptr(), out.data_ptr(),
                      _rows(x, "x"), _rows(out, "out"), x.shape[0], n, k, heads, 0, 0, None, None)
    _lib.check(_lib.lib().mdb_gemm(a, _stream()), "mdb_gemm (per head)")
    return out


def gemm_experts(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, tile_expert: torch.Tensor, num_tiles: torch.Tensor,
                 max_rows_per_expert: int = 0, act: int = ACT_NONE) -> torch.Tensor:
    """Rows of x / out laid out by expert in tiles of 128; w [experts, n, k]."""
    experts, n, k = w.shape
    a = _lib.GemmArgs(_act_dtype(x, "x"), 2, act, int(out.dtype == torch.float32), x.data_ptr(), w.data_ptr(),
                      out.data_ptr(), _rows(x, "x"), _rows(out, "out"), x.shape[0], n, k, 0, experts, max_rows_per_expert,
                      tile_expert.data_ptr(), num_tiles.data_ptr())
    _lib.check(_lib.lib().mdb_gemm(a, _stream()), "mdb_gemm (per expert)")
    return out


def residual_norm(residual: torch.Tensor, width: int, eps: float, dtype: torch.dtype, weight: torch.Tensor | None = None,
                  out: torch.Tensor | None = None, add: tuple = (), ids: torch.Tensor | None = None,
                  embed: torch.Tensor | None = None, embed_scale: float = 1.0, moe: tuple | None = None, post: bool = False,
                  res_scale: float = 1.0, weight2: torch.Tensor | None = None) -> None:
    """Folds projections (``add``), chosen experts' rows (``moe`` = rows, slots [m, top], weights [m, top]) or the scaled
    embedding (``ids``) into the fp32 residual and writes its RMSNorm to ``out`` (without ``weight``: the residual itself).
    ``post``: the residual, scaled by ``res_scale`` before the sum, becomes its own norm, and ``out`` receives it or its norm
    with ``weight2``."""
    m, wp = residual.shape
    a = _lib.ResidualNormArgs(dtype=_DTYPES[dtype], m=m, width=width, width_pad=wp, residual=residual.data_ptr(), eps=eps,
                              weight=_ptr(weight), y=_ptr(out), ldy=0 if out is None else _rows(out, "out"), post=int(post),
                              weight2=_ptr(weight2), res_scale=res_scale)
    if ids is not None:
        _need(ids, torch.int64, "ids")
        a.ids, a.embed, a.vocab, a.embed_scale = ids.data_ptr(), embed.data_ptr(), embed.shape[0], embed_scale
    for i, r in enumerate(add):
        a.add[i] = r.c()
    if moe is not None:
        rows, slots, weights = moe
        a.moe_rows, a.moe_ld, a.moe_slot, a.moe_weight, a.moe_top = (rows.data_ptr(), rows.stride(0), slots.data_ptr(),
                                                                     weights.data_ptr(), slots.shape[1])
    _lib.check(_lib.lib().mdb_residual_norm(a, _stream()), "mdb_residual_norm")


def rms_segment(src: Rows, n: int, n_pad: int, weight: torch.Tensor, eps: float, out: torch.Tensor,
                slots: torch.Tensor | None = None) -> _lib.RmsSegment:
    """Columns [0, n) of ``src``, RMS-normalised and zero-padded to n_pad, into rows of ``out`` ([rows, >= n_pad])."""
    return _lib.RmsSegment(src.c(), weight.data_ptr(), out.data_ptr(), out.stride(0), _ptr(slots), out.shape[0], n, n_pad, eps)


def rms_rows(segments: list, m: int, dtype: torch.dtype) -> None:
    arr = (_lib.RmsSegment * len(segments))(*segments)
    _lib.check(_lib.lib().mdb_rms_rows(_DTYPES[dtype], arr, len(segments), m, _stream()), "mdb_rms_rows")


def gated_norm(o: torch.Tensor, gate: Rows, weight: torch.Tensor, per_head_weight: bool, eps: float, out: torch.Tensor,
               den: torch.Tensor | None = None) -> None:
    """o [m, heads, vdim] fp32, divided by den [m, heads] if given, normalised per head, times weight, times sigmoid(gate),
    into out [m, heads * vdim]."""
    m, heads, vdim = o.shape
    a = _lib.GatedNormArgs(_act_dtype(out, "out"), m, heads, vdim, o.data_ptr(), _ptr(den), gate.c(), weight.data_ptr(),
                           out.data_ptr(), _rows(out, "out"), vdim if per_head_weight else 0, eps)
    _lib.check(_lib.lib().mdb_gated_norm(a, _stream()), "mdb_gated_norm")


def part_norm(o: torch.Tensor, gate: Rows, weight: torch.Tensor, parts: int, gate_first: bool, eps: float, out: torch.Tensor,
              out_scale: float = 1.0) -> None:
    """o [m, n] fp32 in ``parts`` equal parts, each by its own root mean square: norm(o * silu(gate)) * weight with
    ``gate_first``, else norm(o) * weight * sigmoid(gate); times out_scale into the first n columns of ``out``."""
    m, n = o.shape
    a = _lib.PartNormArgs(_act_dtype(out, "out"), m, n, parts, int(gate_first), out_scale, eps, o.data_ptr(), gate.c(),
                          weight.data_ptr(), out.data_ptr(), _rows(out, "out"))
    _lib.check(_lib.lib().mdb_part_norm(a, _stream()), "mdb_part_norm")


def scan_dim_pad(dim: int) -> int:
    p = int(_lib.lib().mdb_scan_dim_pad(dim))
    if p == 0:
        raise ValueError(f"recurrent heads of {dim} key channels are not supported (at most 512)")
    return p


def scan_blocks(vdim: int) -> int:
    return int(_lib.lib().mdb_scan_blocks(vdim))


def scan_fusable(dim_pad: int, vdim: int) -> bool:
    return bool(_lib.lib().mdb_scan_fusable(dim_pad, vdim))


def delta_prep(dtype: torch.dtype, m: int, bs: int, heads: int, kv_heads: int, dim: int, vdim: int, q: Rows, k: Rows, v: Rows,
               b: Rows, conv: tuple, conv_state: torch.Tensor, portions: tuple, outs: tuple, shift_state: bool,
               copy: Rows | None = None, copy_out: torch.Tensor | None = None) -> None:
    """``conv`` = fp32 [channels, taps] weights of q, k, v; ``conv_state`` [slots, taps - 1, channels]; ``portions`` =
    (row_seq, cu_q, start, state_slot); ``outs`` = fp32 (q, k [m, kv_heads, dim_pad], v [m, heads, vdim], beta [m, heads])."""
    qo, ko, vo, bo = outs
    row_seq, cu_q, start, slot = portions
    a = _lib.DeltaPrepArgs(
        dtype=_DTYPES[dtype], m=m, bs=bs, heads=heads, kv_heads=kv_heads, dim=dim, dim_pad=qo.shape[-1], vdim=vdim,
        taps=conv[0].shape[1], channels=conv_state.shape[-1], shift_state=int(shift_state),
        copy_cols=0 if copy is None else copy_out.shape[1], q=q.c(), k=k.c(), v=v.c(), b=b.c(), copy=_rows_c(copy),
        copy_out=_ptr(copy_out), copy_ld=0 if copy_out is None else copy_out.stride(0), conv_q=conv[0].data_ptr(),
        conv_k=conv[1].data_ptr(), conv_v=conv[2].data_ptr(), conv_state=conv_state.data_ptr() or None,
        conv_slot_stride=conv_state.stride(0), num_slots=conv_state.shape[0], row_seq=row_seq.data_ptr(),
        cu_q=cu_q.data_ptr(), start=start.data_ptr(), state_slot=slot.data_ptr(), q_out=qo.data_ptr(), k_out=ko.data_ptr(),
        v_out=vo.data_ptr(), beta_out=bo.data_ptr())
    _lib.check(_lib.lib().mdb_delta_prep(a, _stream()), "mdb_delta_prep")


def channel_decay(x: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, q: torch.Tensor, k: torch.Tensor,
                  beta: torch.Tensor, portions: tuple, out: torch.Tensor, scalars: torch.Tensor, dim: int) -> None:
    """out [m, heads, dim_pad] = exp(-exp(a_log) softplus(x + dt_bias)); x fp32 [m, >= heads * dim]; scalars [m, heads, 4] =
    (k.q, for a portion's odd tokens the products with the token before, beta); q, k, beta of ``delta_prep``."""
    m, heads, dp = out.shape
    row_seq, cu_q, _, _ = portions
    a = _lib.DecayArgs(m, heads, q.shape[1], dim, dp, x.data_ptr(), _rows(x, "x"), a_log.data_ptr(), dt_bias.data_ptr(),
                       q.data_ptr(), k.data_ptr(), beta.data_ptr(), out.data_ptr(), scalars.data_ptr(), row_seq.data_ptr(),
                       cu_q.data_ptr())
    _lib.check(_lib.lib().mdb_channel_decay(a, _stream()), "mdb_channel_decay")


def mlstm_prep(dtype: torch.dtype, m: int, heads: int, dim: int, vdim: int, q: Rows, k: Rows, v: Rows, i: Rows, f: Rows,
               bias_i: torch.Tensor, bias_f: torch.Tensor, cap: float, outs: tuple) -> None:
    qo, ko, vo, li, lf = outs
    a = _lib.MlstmPrepArgs(_DTYPES[dtype], m, heads, dim, qo.shape[-1], vdim, q.c(), k.c(), v.c(), i.c(), f.c(),
                           bias_i.data_ptr(), bias_f.data_ptr(), qo.data_ptr(), ko.data_ptr(), vo.data_ptr(), li.data_ptr(),
                           lf.data_ptr(), cap)
    _lib.check(_lib.lib().mdb_mlstm_prep(a, _stream()), "mdb_mlstm_prep")


def decay_prep(dtype: torch.dtype, m: int, bs: int, heads: int, kv_heads: int, dim: int, vdim: int, q: Rows, k: Rows, v: Rows,
               portions: tuple, outs: tuple, dt: Rows | None = None, a_log: torch.Tensor | None = None,
               dt_bias: torch.Tensor | None = None, decay: torch.Tensor | None = None, conv: torch.Tensor | None = None,
               conv_bias: torch.Tensor | None = None, conv_state: torch.Tensor | None = None, shift_state: bool = False) -> None:
    """Inputs of the decay scan: ``outs`` = fp32 (q, k [m, kv_heads, dim_pad], v [m, heads, vdim], decay, step [m, heads]); with
    q, k, v in bf16 the inputs of the chunk form, whose decay is the logarithm.
    ``conv`` fp32 [channels, taps] (v | k | q) with ``conv_bias`` and ``conv_state`` [slots, taps - 1, channels], or None: silu
    alone.  Scalars from ``dt`` with ``a_log`` and ``dt_bias``, or the fixed ``decay`` [heads] and step 1."""
    qo, ko, vo, do, so = outs
    row_seq, cu_q, start, slot = portions
    taps = 0 if conv is None else conv.shape[1]
    a = _lib.DecayPrepArgs(
        dtype=_DTYPES[dtype], m=m, bs=bs, heads=heads, kv_heads=kv_heads, dim=dim, dim_pad=qo.shape[-1], vdim=vdim, taps=taps,
        channels=0 if conv is None else conv.shape[0], shift_state=int(shift_state),
        for_chunks=int(qo.dtype == _BF16), q=q.c(), k=k.c(), v=v.c(), dt=_rows_c(dt),
        conv=_ptr(conv), conv_bias=_ptr(conv_bias), conv_state=(_ptr(conv_state) or None) if taps > 1 else None,
        conv_slot_stride=conv_state.stride(0) if taps > 1 else 0, num_slots=conv_state.shape[0] if taps > 1 else 1 << 30,
        row_seq=row_seq.data_ptr(), cu_q=cu_q.data_ptr(), start=start.data_ptr(), state_slot=slot.data_ptr(), a_log=_ptr(a_log),
        dt_bias=_ptr(dt_bias), decay_const=_ptr(decay), q_out=qo.data_ptr(), k_out=ko.data_ptr(), v_out=vo.data_ptr(),
        decay_out=do.data_ptr(), step_out=so.data_ptr())
    _lib.check(_lib.lib().mdb_decay_prep(a, _stream()), "mdb_decay_prep")


SCAN_DELTA, SCAN_MLSTM, SCAN_DECAY = 0, 1, 2


def scan(mode: int, dtype: torch.dtype, bs: int, heads: int, kv_heads: int, dim: int, vdim: int, q, k, v, s0, s1, state,
         portions: tuple, eps: float = 0.0, g=None, scalars=None, mstate=None, den=None, out=None, raw_decay: Rows | None = None,
         a_log=None, dt_bias=None, gate: Rows | None = None, norm=None, per_head_norm: bool = False, y=None, skip=None,
         one_token: bool = False) -> None:
    """The recurrence over every sequence's portion; ``state`` [slots, heads, vdim (mLSTM: + 1), dim_pad] fp32.  With ``y``
    the fused one-token form runs (decay from ``raw_decay``, gated norm into ``y``), else ``out`` [m, heads, vdim] fp32
    (mLSTM: and ``den`` [m, heads]) is written.  Decay scan: s0 = decay, s1 = step, ``skip`` [heads] times v is added to the
    read-out; ``one_token`` picks its one-token form."""
    _, cu_q, start, slot = portions
    a = _lib.ScanArgs(
        mode=mode, dtype=_DTYPES[dtype], fused=int(y is not None or one_token), bs=bs, heads=heads, kv_heads=kv_heads, dim=dim,
        dim_pad=q.shape[-1], vdim=vdim, eps=eps, q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), g=_ptr(g), s0=_ptr(s0),
        s1=_ptr(s1), state=state.data_ptr(), state_slot_stride=state.stride(0), num_slots=state.shape[0],
        mstate=_ptr(mstate), scalars=_ptr(scalars), den=_ptr(den), cu_q=cu_q.data_ptr(), start=start.data_ptr(), state_slot=slot.data_ptr(),
        out=_ptr(out), raw_decay=_rows_c(raw_decay), a_log=_ptr(a_log), dt_bias=_ptr(dt_bias), gate=_rows_c(gate),
        norm=_ptr(norm), norm_head_stride=vdim if per_head_norm else 0, y=_ptr(y), ldy=0 if y is None else _rows(y, "y"),
        skip=_ptr(skip))
    _lib.check(_lib.lib().mdb_scan(a, _stream()), "mdb_scan")


def chunk_scan_supported(dim_pad: int, vdim: int) -> bool:
    return bool(_lib.lib().mdb_chunk_scan_supported(dim_pad, vdim))


def chunk_scan(bs: int, heads: int, kv_heads: int, dim: int, vdim: int, q, k, v, log_decay, step, state, portions: tuple, max_q: int, out,
               skip=None) -> None:
    """The decay scan over prompt portions on the tensor cores: bf16 q, k [m, >= kv_heads * dim] and v [m, >= heads * vdim] (row
    strides free), logarithms of the decays (at least -104) and steps [m, heads], or [heads] for all tokens; ``state`` and
    ``out`` as in ``scan``."""
    _, cu_q, start, slot = portions
    for t, nm in ((q, "q"), (k, "k"), (v, "v")):
        _need(t, _BF16, nm)
    a = _lib.ChunkScanArgs(q.shape[0], bs, heads, kv_heads, dim, state.shape[-1], vdim, max_q, q.data_ptr(), k.data_ptr(), v.data_ptr(), _rows(q, "q"),
                           _rows(k, "k"), _rows(v, "v"), heads if log_decay.dim() > 1 else 0, log_decay.data_ptr(),
                           step.data_ptr(), _ptr(skip), state.data_ptr(), state.stride(0), state.shape[0], cu_q.data_ptr(),
                           start.data_ptr(), slot.data_ptr(), out.data_ptr())
    _lib.check(_lib.lib().mdb_chunk_scan(a, _stream()), "mdb_chunk_scan")


def moe_route(logits: Rows, m: int, experts: int, top: int, groups: int, keep: int, ids: torch.Tensor, weights: torch.Tensor,
              row_slot: torch.Tensor | None = None) -> None:
    a = _lib.MoeRouteArgs(m, experts, top, groups, keep, logits.c(), _ptr(row_slot), ids.data_ptr(), weights.data_ptr())
    _lib.check(_lib.lib().mdb_moe_route(a, _stream()), "mdb_moe_route")


def moe_max_tiles(m: int, top: int, experts: int) -> int:
    return int(_lib.lib().mdb_moe_max_tiles(m, top, experts))


def moe_plan(ids: torch.Tensor, experts: int, max_tiles: int, slot: torch.Tensor, row_token: torch.Tensor,
             tile_expert: torch.Tensor, num_tiles: torch.Tensor) -> None:
    m, top = ids.shape
    a = _lib.MoePlanArgs(m, top, experts, max_tiles, ids.data_ptr(), slot.data_ptr(), row_token.data_ptr(),
                         tile_expert.data_ptr(), num_tiles.data_ptr())
    _lib.check(_lib.lib().mdb_moe_plan(a, _stream()), "mdb_moe_plan")


def moe_gather(x: torch.Tensor, out: torch.Tensor, row_token: torch.Tensor, num_tiles: torch.Tensor, max_tiles: int) -> None:
    _lib.check(_lib.lib().mdb_moe_gather(_act_dtype(x, "x"), x.data_ptr(), _rows(x, "x"), out.data_ptr(), out.shape[1],
                                         row_token.data_ptr(), num_tiles.data_ptr(), max_tiles, _stream()), "mdb_moe_gather")


def latent_attn_workspace_bytes(m: int, heads: int, width: int, nsplit: int) -> int:
    return int(_lib.lib().mdb_latent_attn_workspace_bytes(m, heads, width, nsplit))


def latent_attn(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, row_seq: torch.Tensor, row_pos: torch.Tensor,
                heads: int, scale: float, out: torch.Tensor, nsplit: int = 1, workspace: torch.Tensor | None = None) -> None:
    """q, out [m, heads * width]; cache [pages * 256, width]; the row at position p sees keys 0 .. p (p = -1: no row)."""
    m, width = q.shape[0], cache.shape[1]
    _need(block_table, torch.int32, "block_table")
    _lib.check(_lib.lib().mdb_latent_attn(
        _act_dtype(q, "q"), q.data_ptr(), cache.data_ptr(), out.data_ptr(), block_table.data_ptr(), block_table.stride(0),
        row_seq.data_ptr(), row_pos.data_ptr(), m, heads, width, cache.shape[0] // 256, scale, nsplit, _ptr(workspace),
        0 if workspace is None else workspace.numel() * workspace.element_size(), _stream()), "mdb_latent_attn")


def gather_latents(cache: torch.Tensor, block_table: torch.Tensor, cu: torch.Tensor, nseq: int, out: torch.Tensor) -> None:
    """out [total, width] = the cached rows of every sequence in order (cu [nseq + 1] row offsets)."""
    _lib.check(_lib.lib().mdb_gather_latents(_act_dtype(cache, "cache"), cache.data_ptr(), block_table.data_ptr(),
                                             block_table.stride(0), cache.shape[0] // 256, cu.data_ptr(), nseq, out.shape[0],
                                             out.data_ptr(), cache.shape[1], _stream()), "mdb_gather_latents")


def causal_attn_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_q: torch.Tensor, cu_k: torch.Tensor, nseq: int,
                       max_q: int, scale: float, out: torch.Tensor) -> None:
    """Causal attention over packed rows, head size 128: q/out [total_q, hq, 128], k/v [total_k, hkv, 128] (row strides
    free); the queries of a sequence are its last ones."""
    for t, nm in ((q, "q"), (k, "k"), (v, "v"), (out, "out")):
        _need(t, _BF16, nm)
        if t.shape[-1] != 128 or t.stride(-1) != 1 or t.stride(1) != 128:
            raise ValueError(f"{nm}: heads of 128 must be densely packed")
    _lib.check(_lib.lib().mdb_attn_causal_varlen(
        q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), out.data_ptr(), out.stride(0),
        cu_q.data_ptr(), cu_k.data_ptr(), nseq, max_q, q.shape[0], k.shape[0], q.shape[1], k.shape[1], scale, _stream()),
        "mdb_attn_causal_varlen")


def rotary_commit(q: Rows, k: Rows, v: Rows, heads: int, kv_heads: int, dim: int, q_norm: torch.Tensor, k_norm: torch.Tensor,
                  eps: float, inv_freq: torch.Tensor, row_pos: torch.Tensor, slots: torch.Tensor, q_out: torch.Tensor,
                  k_cache: torch.Tensor, v_cache: torch.Tensor) -> None:
    """Per-head norms and interleaved rotation (of 2 * len(inv_freq) channels) of q and k; q_out [m, heads, dim_pad], caches
    [slots, kv_heads, dim_pad]; v goes to its cache as it comes."""
    m, _, dp = q_out.shape
    _need(inv_freq, torch.float64, "inv_freq")
    a = _lib.RotaryCommitArgs(_act_dtype(q_out, "q_out"), m, heads, kv_heads, dim, dp, 2 * inv_freq.numel(), eps, q.c(), k.c(), v.c(),
                              q_norm.data_ptr(), k_norm.data_ptr(), inv_freq.data_ptr() or None, row_pos.data_ptr(), slots.data_ptr(),
                              k_cache.shape[0], q_out.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr())
    _lib.check(_lib.lib().mdb_rotary_commit(a, _stream()), "mdb_rotary_commit")


def window_attn_workspace_bytes(m: int, heads: int, dim_pad: int, nsplit: int) -> int:
    return int(_lib.lib().mdb_window_attn_workspace_bytes(m, heads, dim_pad, nsplit))


def window_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor, portions: tuple,
                row_pos: torch.Tensor, max_q: int, dim: int, window: int, sink: bool, scale: float, out: torch.Tensor,
                gate: Rows | None = None, out_scale: float = 1.0, nsplit: int = 1, workspace: torch.Tensor | None = None) -> None:
    """q [m, heads, dim_pad]; caches [pages * 256, kv_heads, dim_pad]; head h of a row goes to columns [h * dim, (h + 1) * dim)
    of ``out``.  ``portions`` = (row_seq, cu_q, start, state_slot)."""
    m, heads, dp = q.shape
    row_seq, cu_q, start, _ = portions
    _need(block_table, torch.int32, "block_table")
    a = _lib.WindowAttnArgs(
        dtype=_act_dtype(q, "q"), m=m, bs=start.numel(), heads=heads, kv_heads=k_cache.shape[1], dim=dim, dim_pad=dp, window=window,
        sink=int(sink), max_q=max_q, nsplit=nsplit, scale=scale, out_scale=out_scale, q=q.data_ptr(), k_cache=k_cache.data_ptr(),
        v_cache=v_cache.data_ptr(), block_table=block_table.data_ptr(), row_seq=row_seq.data_ptr(), row_pos=row_pos.data_ptr(),
        cu_q=cu_q.data_ptr(), start=start.data_ptr(), table_stride=block_table.stride(0), num_pages=k_cache.shape[0] // 256,
        gate=_rows_c(gate), out=out.data_ptr(), ld_out=_rows(out, "out"), workspace=_ptr(workspace),
        workspace_bytes=0 if workspace is None else workspace.numel() * workspace.element_size())
    _lib.check(_lib.lib().mdb_window_attn(a, _stream()), "mdb_window_attn")


def pick_token(logits: torch.Tensor, vocab: int, temperatures: torch.Tensor, seed: int, step_dev: torch.Tensor | None,
               out: torch.Tensor, status_out: torch.Tensor | None = None) -> None:
    """Token per row of fp32 logits [m, >= vocab]: Gumbel-max at the row's temperature, or arg-max at temperature 0."""
    _need(logits, torch.float32, "logits")
    _lib.check(_lib.lib().mdb_pick_token(logits.data_ptr(), _rows(logits, "logits"), logits.shape[0], vocab,
                                         temperatures.data_ptr(), seed & 0xFFFFFFFF, _ptr(step_dev), out.data_ptr(),
                                         _ptr(status_out), _stream()), "mdb_pick_token")


def copy_rows(table: torch.Tensor, ids: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out[i] = table[ids[i]] for rows of either activation type (a byte copy)."""
    t, o = (table, out) if table.dtype == _BF16 else (table.view(_BF16), out.view(_BF16))
    gather_rows(t, ids, out=o)
    return out
