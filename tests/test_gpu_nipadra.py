"""Nipadra decoder design on the GPU against its plain restatement: each mechanism alone, then whole models -- prompts,
portions, batches, reuse of pages and slots, long decoding, generation through the engine."""
import io
import json
import sys
from importlib import import_module

import pytest
import torch

import hybrid_cases as hc
from hybrid_cases import hybrid, pkg, row_error, run_portions, sequence
from nipadra_cases import EVEN, MODELS, ODD, RAGGED, tensors
from oracle import nipadra_oracle as orc

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
DTYPES = [F32, BF]


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rand(*shape, seed=0, scale=1.0, dtype=BF):
    """CPU values that the activation type holds exactly."""
    return (torch.randn(*shape, generator=gen(seed)) * scale).to(dtype).float()


def rel(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    return float((got - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(1e-9))


def i32(x):
    return torch.as_tensor(x).to(torch.int32).to(DEV)


def portions_of(counts, starts=None, slots=None):
    """(row_seq, cu_q, start, state_slot) device tensors."""
    row_seq = torch.cat([torch.full((n,), i) for i, n in enumerate(counts)])
    return (i32(row_seq), i32(torch.tensor([0] + list(counts)).cumsum(0)), i32(starts or [0] * len(counts)),
            i32(slots if slots is not None else list(range(len(counts)))))


def rows(t, dtype, as_parts=False):
    """A projection's output as the kernels take it, padded to a multiple of four columns: rows, or two slices that sum to it."""
    t = torch.nn.functional.pad(t, (0, -t.shape[1] % 4))
    if as_parts:
        a = torch.randn(t.shape, generator=gen(99)).to(BF).float()
        return pkg.ops.Rows(parts=torch.stack([a, t - a]).to(DEV))
    return pkg.ops.Rows(t.to(dtype).to(DEV))


# --------------------------------------------------------------------------- row kernels and products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,m", [(160, 5), (1500, 70), (4096, 3)])
def test_norm_behind_the_sum(dtype, width, m):
    ops, wp = pkg.ops, hybrid.pad128(width)
    pad = lambda t: torch.nn.functional.pad(t, (0, wp - width))
    res, a, parts = torch.randn(m, width, generator=gen(1)), rand(m, width, seed=3), torch.randn(3, m, width, generator=gen(4))
    w, w2 = rand(width, seed=2, scale=0.3), rand(width, seed=6, scale=0.3)
    rd, y = pad(res).to(DEV), torch.zeros(m, wp, dtype=dtype, device=DEV)
    args = dict(post=True, res_scale=1.7, add=(ops.Rows(pad(a).to(dtype).to(DEV)), ops.Rows(parts=pad(parts).to(DEV))))
    ops.residual_norm(rd, width, 3e-6, dtype, weight=pad(1 + w).to(DEV), out=y, **args)
    ref = orc.post_norm(res.double(), (a + parts.sum(0).to(dtype).float()).double(), w.double(), 1.7, 3e-6)
    assert rel(rd[:, :width], ref) < 1e-6 and float(rd[:, width:].abs().sum()) == 0
    assert rel(y[:, :width], ref) < (1e-6 if dtype is F32 else 4e-3)
    ops.residual_norm(pad(res).to(DEV), width, 3e-6, dtype, weight=pad(1 + w).to(DEV), out=y, weight2=pad(1 + w2).to(DEV), **args)
    assert rel(y[:, :width], orc.rms(ref, 3e-6) * (1 + w2)) < (1e-6 if dtype is F32 else 4e-3)
    # embedding without a norm
    table, ids = rand(50, width, seed=8), torch.tensor([0, 49] * m)[:m]
    ops.residual_norm(rd, width, 3e-6, dtype, out=y, ids=ids.to(DEV), embed=pad(table).to(dtype).to(DEV))
    assert torch.equal(rd[:, :width].cpu(), table[ids]) and torch.equal(y[:, :width].float().cpu(), table[ids])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("as_parts", [False, True])
@pytest.mark.parametrize("n,parts", [(96, 4), (1000, 1), (66, 3), (3072, 2), (6144, 1)])
def test_norm_in_parts_with_gate(dtype, n, parts, as_parts):
    if as_parts and dtype is F32:
        pytest.skip("split-k slices exist in bf16 steps")
    m = 5
    o, z, w = torch.randn(m, n, generator=gen(1)) * 3, rand(m, n, seed=2), 0.5 + torch.rand(n, generator=gen(3))
    o[:, :n // parts] *= 50                              # parts of very different size
    zd = rows(z, dtype, as_parts)
    zr = (z if not as_parts else (zd.parts.sum(0).to(BF).float().cpu()[:, :n])).double()
    y = torch.full((m, hybrid.pad128(n)), 7.0, dtype=dtype, device=DEV)
    tol = 2e-6 if dtype is F32 else 4e-3
    pkg.ops.part_norm(o.to(DEV), zd, w.to(DEV), parts, True, 1e-5, y, out_scale=0.7)
    assert rel(y[:, :n], 0.7 * orc.gated_group_norm(o.double(), zr, w.double(), parts, 1e-5)) < tol
    pkg.ops.part_norm(o.to(DEV), zd, w.to(DEV), parts, False, 1e-5, y)
    ref = orc.rms(o.double().view(m, parts, -1), 1e-5).view(m, n) * w.double() * orc.sigmoid(zr)
    assert rel(y[:, :n], ref) < tol and float((y[:, n:] - 7).abs().sum()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k", [(1, 128, 128), (40, 256, 384), (65, 128, 256), (300, 384, 128), (2100, 256, 256)])
def test_gated_product(dtype, m, n, k):
    x, w = rand(m, k, seed=1), rand(2 * n, k, seed=2, scale=k ** -0.5)
    y = torch.zeros(m, n, dtype=dtype, device=DEV)
    pkg.ops.gemm(x.to(dtype).to(DEV), w.to(dtype).to(DEV), y, act=pkg.ops.ACT_RELU_GLU)
    z = x.double() @ w.double().T
    assert rel(y, torch.relu(z[:, :n]) * z[:, n:]) < (2e-6 if dtype is F32 else 4e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k,from_", [(65, 256, 2048, 72), (300, 384, 128, 0), (2100, 512, 256, 260), (130, 640, 1024, 128)])
def test_product_activated_from_a_column_on(dtype, m, n, k, from_):
    x, w = rand(m, k, seed=1), rand(n, k, seed=2, scale=k ** -0.5)
    y = torch.zeros(m, n, dtype=dtype, device=DEV)
    pkg.ops.gemm(x.to(dtype).to(DEV), w.to(dtype).to(DEV), y, act=pkg.ops.ACT_SILU, act_from=from_)
    ref = x.double() @ w.double().T
    ref[:, from_:] = orc.silu(ref[:, from_:])
    assert rel(y, ref) < (2e-6 if dtype is F32 else 4e-3)


@pytest.mark.parametrize("mq", [64, 150])
def test_chunk_scan_reads_columns_of_a_projection(mq):
    """Heads of 40 channels in rows of another matrix: missing channels of the stored state count as zeros."""
    ops, T, H, D, DV = pkg.ops, 150, 3, 40, 24
    x = rand(T, 8 + 2 * H * D + H * DV + 16, seed=1, scale=0.5)
    q, k, v = x[:, 8:8 + H * D], x[:, 128:128 + H * D], x[:, 248:248 + H * DV]
    log = torch.tensor([-0.5, -0.01, -3.0])
    decay = torch.exp(log.double()).expand(T, H)
    ref = orc.linear_scan(q.double().view(T, H, D), k.double().view(T, H, D), v.double().view(T, H, DV), decay, torch.ones_like(decay))
    xd = x.to(BF).to(DEV)
    state, o = torch.full((1, H, DV, 64), 5.0, device=DEV), torch.zeros(T, H, DV, device=DEV)
    ops.chunk_scan(1, H, H, D, DV, xd[:, 8:], xd[:, 128:], xd[:, 248:], log.to(DEV), torch.ones(H, device=DEV), state, portions_of([T], slots=[0]), mq, o)
    assert rel(o, ref) < 3e-5 and float(state[..., D:].abs().max()) == 0


# --------------------------------------------------------------------------- rotation and caches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("as_parts", [False, True])
@pytest.mark.parametrize("H,G,D,dims", [(4, 2, 64, 64), (3, 1, 40, 24), (2, 2, 30, 6), (5, 5, 128, 128), (2, 1, 262, 130), (2, 1, 12, 0),
                                        (2, 1, 200, 196)])
def test_rotary_commit(dtype, as_parts, H, G, D, dims):
    if as_parts and dtype is F32:
        pytest.skip("split-k slices exist in bf16 steps")
    ops, dp, base = pkg.ops, hybrid.pad_head(D), 1e4
    pos = [0, 1, 255, 4097, -1, 123456]
    m = len(pos)
    x = rand(m, (H + G) * D, seed=1)
    qn, kn = 1 + rand(D, seed=2, scale=0.2), 1 + rand(D, seed=3, scale=0.2)
    src = rows(x, dtype, as_parts)
    xr = x if not as_parts else src.parts.sum(0).to(BF).float().cpu()
    slots = [300, 2, -1, 511, -1, 0]
    q = torch.full((m, H, dp), 7.0, dtype=dtype, device=DEV)
    kc, vc = (torch.full((512, G, dp), 7.0, dtype=dtype, device=DEV) for _ in range(2))
    inv = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
    ks = src.cols(H * D)
    padded = lambda w: torch.nn.functional.pad(w, (0, -D % 4)).to(DEV)
    ops.rotary_commit(src, ks, ks, H, G, D, padded(qn), padded(kn), 1e-5, inv.to(DEV), i32(pos), i32(slots), q, kc, vc)
    xd = xr.double()[:, :(H + G) * D]
    at = torch.tensor([max(p, 0) for p in pos])
    qr = orc.rotate(orc.rms(xd[:, :H * D].view(m, H, D), 1e-5) * qn, dims, base, at)
    raw = xd[:, H * D:].view(m, G, D)
    kr = orc.rotate(orc.rms(raw, 1e-5) * kn, dims, base, at)
    tol = 2e-6 if dtype is F32 else 4e-3
    for i, (p, s) in enumerate(zip(pos, slots)):
        if p >= 0:
            assert rel(q[i, :, :D], qr[i]) < tol, p
        if s >= 0:
            assert rel(kc[s, :, :D], kr[i]) < tol and torch.equal(vc[s, :, :D].float().cpu(), raw[i].float())
    assert float((q[4] - 7).abs().sum()) == 0 and float((kc[3:300] - 7).abs().sum()) == 0 and pkg._lib.device_status() == 0
    slots[1] = 512
    ops.rotary_commit(src, ks, ks, H, G, D, padded(qn), padded(kn), 1e-5, inv.to(DEV), i32(pos), i32(slots), q, kc, vc)
    assert pkg._lib.device_status() == 1


# --------------------------------------------------------------------------- window attention
def _paged(x, table, pages, dp, dtype, fill=float("nan")):
    """Rows [T, G, D] laid out on the pages of ``table``; what belongs to nobody holds ``fill``."""
    T, G, D = x.shape
    out = torch.full((pages * 256, G, dp), fill)
    for i in range(0, T, 256):
        n = min(256, T - i)
        out[table[i // 256] * 256:table[i // 256] * 256 + n] = 0
        out[table[i // 256] * 256:table[i // 256] * 256 + n, :, :D] = x[i:i + n]
    return out.to(dtype).to(DEV)


def _attend(q, k, v, table, start, counts_max, D, window, sink, scale, dtype, gate=None, out_scale=1.0, nsplit=1, fill=float("nan")):
    """Queries of one sequence (its last rows) through the kernels; heads at their own columns."""
    ops, (n, H, _), (T, G, _) = pkg.ops, q.shape, k.shape
    dp, pages = hybrid.pad_head(D), max(table) + 2
    qd = torch.nn.functional.pad(q, (0, dp - D)).to(dtype).to(DEV)
    kc, vc = _paged(k, table, pages, dp, dtype, fill), _paged(v, table, pages, dp, dtype, fill)
    out = torch.full((n, (H * D + 7) // 8 * 8), 7.0, dtype=dtype, device=DEV)
    ws = torch.empty(max(16, ops.window_attn_workspace_bytes(n, H, dp, nsplit)), dtype=torch.uint8, device=DEV)
    ops.window_attn(qd, kc, vc, i32([table + [-1]]), portions_of([n], [start]), i32(list(range(start, start + n))), counts_max, D, window,
                    sink, scale, out, gate=gate, out_scale=out_scale, nsplit=nsplit, workspace=ws)
    assert pkg._lib.device_status() == 0 and (H * D % 8 == 0 or float((out[:, H * D:] - 7).abs().sum()) == 0)
    return out[:, :H * D].float().cpu().view(n, H, D)


SHAPES = [(8, 2, 64), (4, 4, 40), (6, 2, 128), (20, 1, 96), (2, 1, 200), (3, 3, 30), (2, 2, 160), (2, 1, 262)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 37, 128, 129, 300, 0])
@pytest.mark.parametrize("H,G,D", SHAPES)
def test_window_attention_prompt_and_decoding(dtype, window, H, G, D):
    """A prompt of 520 tokens over three pages in one portion, the same rows token by token (in one part and in several), and
    the end of the prompt as a portion; gate, output scale and sink on."""
    T, scale = 520, 1.5 * D ** -0.5
    q, k, v = rand(T, H, D, seed=1), rand(T, G, D, seed=2), rand(T, G, D, seed=3)
    g = rand(T, H, seed=4)
    ref = _window_reference(q, k, v, scale, window) * 0.8 * orc.sigmoid(g.double())[:, :, None]
    table = [4, 0, 2]
    tol = 3e-6 if dtype is F32 else 6e-3
    for start, n, mq, parts in ((0, T, T, 1), (0, T, 1, 1), (100, T - 100, 1, 5), (447, T - 447, T, 1), (T - 2, 2, 2, 3)):
        got = _attend(q[start:start + n], k[:start + n], v[:start + n], table, start, mq, D, window, True, scale, dtype, rows(g[start:start + n], dtype),
                      0.8, parts)
        assert rel(got, ref[start:start + n]) < tol, (start, n, mq)
        worst = (got.double() - ref[start:start + n]).pow(2).mean((1, 2)).sqrt().max() / ref.pow(2).mean().sqrt()
        assert float(worst) < 4 * tol, (start, n, mq, int((got.double() - ref[start:start + n]).pow(2).mean((1, 2)).argmax()))


def _window_reference(q, k, v, scale, window, sink=True):
    """The same equations as the restatement's, over whole matrices."""
    q, k, v = q.double(), k.double(), v.double()
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    s = s.masked_fill((d < 0) | (d >= (window or T)), float("-inf"))
    m = s.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(s - m)
    return torch.einsum("hij,jhd->ihd", e / (e.sum(-1, keepdim=True) + (torch.exp(-m) if sink else 0)), v)


def test_matrix_form_of_the_reference():
    q, k, v = (rand(40, h, 8, seed=h) for h in (4, 2, 2))
    assert torch.allclose(_window_reference(q, k, v, 0.4, 7), orc.window_sink_attention(q.double(), k.double(), v.double(), 0.4, 7))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [16, 100, 255, 256, 257, 400])
@pytest.mark.parametrize("mq", [1, 700])
def test_window_attention_sees_its_edges(dtype, window, mq):
    """Every query looks hard at the key just inside its window or at the one just outside: the first must come back nearly
    whole, of the second nothing may.  Values say whose key they are."""
    T, D = 700, 64
    k = torch.nn.functional.normalize(torch.randn(T, 1, D, generator=gen(5)), dim=-1).to(BF).float()
    v = rand(T, 1, D, seed=6)
    q = torch.zeros(T, 2, D)
    for i in range(T):
        inside, outside = i - window + 1, i - window
        q[i, 0] = k[max(inside, 0), 0] * 40              # head 0: just inside
        if outside >= 0:
            q[i, 1] = k[outside, 0] * 40                 # head 1: just outside
    ref = _window_reference(q, k, v, 1.0, window)
    got = _attend(q, k, v, [2, 0, 3], 0, mq, D, window, True, 1.0, dtype).double()
    e = (got - ref).pow(2).mean(-1).sqrt()
    assert float(e.max()) < (1e-5 if dtype is F32 else 3e-2), int(e.argmax())
    inside = torch.arange(T) - window + 1
    keep = inside >= 0
    assert float((got[keep, 0] - v[inside[keep], 0].double()).pow(2).mean(-1).sqrt().max()) < 0.1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mq,parts", [(1, 1), (1, 3), (200, 1)])
@pytest.mark.parametrize("level", [-300.0, -30.0, 0.0, 30.0, 300.0])
def test_sink_takes_its_share(dtype, mq, parts, level):
    """All scores equal: n keys leave n e^s / (1 + n e^s) of the value, from nothing to all of it."""
    T, D, window = 200, 64, 150
    q, k, v = torch.zeros(T, 1, D), torch.zeros(T, 1, D), torch.ones(T, 1, D)
    q[..., 0], k[..., 0] = level, 1.0
    n = torch.arange(1, T + 1).clamp_max(window).double()
    want = 1 / (1 + torch.exp(torch.tensor(-level, dtype=torch.float64)) / n)
    got = _attend(q, k, v, [1], 0, mq, D, window, True, 1.0, dtype, nsplit=parts)
    assert float((got.double() - want[:, None, None]).abs().max()) < (1e-5 if dtype is F32 else 8e-3)
    got = _attend(q, k, v, [1], 0, mq, D, window, False, 1.0, dtype, nsplit=parts)
    assert float((got.double() - 1).abs().max()) < (1e-5 if dtype is F32 else 8e-3)


@pytest.mark.parametrize("mq", [1, 300])
def test_window_attention_of_unequal_requests(mq):
    """Portions of several requests at other places, one of one token, against each alone; a bad page is reported."""
    ops, H, G, D, W, scale = pkg.ops, 4, 2, 128, 200, 0.12
    lens, counts, tables = [300, 513, 40], [300 if mq > 1 else 3, 1, 25], [[5, 1], [0, 2, 6], [3]]
    dp, pages = 128, 7
    kc, vc = torch.zeros(pages * 256, G, dp), torch.zeros(pages * 256, G, dp)
    qs, refs = [], []
    for i, (T, n, tb) in enumerate(zip(lens, counts, tables)):
        q, k, v = rand(T, H, D, seed=10 + i), rand(T, G, D, seed=20 + i), rand(T, G, D, seed=30 + i)
        refs.append(_window_reference(q, k, v, scale, W)[T - n:])
        qs.append(q[T - n:])
        for j in range(0, T, 256):
            c = min(256, T - j)
            kc[tb[j // 256] * 256:tb[j // 256] * 256 + c], vc[tb[j // 256] * 256:tb[j // 256] * 256 + c] = k[j:j + c], v[j:j + c]
    starts = [t - n for t, n in zip(lens, counts)]
    pos = [p for s, n in zip(starts, counts) for p in range(s, s + n)]
    table = torch.full((3, 4), -1)
    for i, tb in enumerate(tables):
        table[i, :len(tb)] = torch.tensor(tb)
    out = torch.zeros(sum(counts), H * D, dtype=BF, device=DEV)
    args = (torch.cat(qs).to(BF).to(DEV), kc.to(BF).to(DEV), vc.to(BF).to(DEV))
    ops.window_attn(*args, i32(table), portions_of(counts, starts), i32(pos), mq, D, W, True, scale, out)
    at = 0
    for n, ref in zip(counts, refs):
        assert rel(out[at:at + n].view(n, H, D), ref) < 6e-3
        at += n
    assert pkg._lib.device_status() == 0
    table[1, 2] = pages
    ops.window_attn(*args, i32(table), portions_of(counts, starts), i32(pos), mq, D, W, True, scale, out)
    assert pkg._lib.device_status() == 2


# --------------------------------------------------------------------------- decay scan
def _scan_case(T, H, G, D, DV, taps, seed):
    c = H * DV + 2 * G * D
    x = {n: rand(T, w, seed=seed + i) for i, (n, w) in enumerate((("v", H * DV), ("k", G * D), ("q", G * D), ("dt", H)))}
    par = dict(conv=rand(c, max(taps, 1), seed=seed + 5, scale=0.6), bias=rand(c, seed=seed + 6, scale=0.5), a_log=rand(H, seed=seed + 7) - 2,
               dt_bias=rand(H, seed=seed + 8), skip=rand(H, seed=seed + 9), decay=torch.linspace(0.3, 0.9995, H))
    return x, par


def _scan_ref(case, H, G, D, DV, taps):
    x, par = case
    T = x["v"].shape[0]
    p = {k: v.double() for k, v in par.items()}
    vkq = torch.cat([x["v"], x["k"], x["q"]], 1).double()
    vkq = orc.short_conv(vkq, p["conv"], p["bias"]) if taps else orc.silu(vkq)
    v, k, q = vkq.split([H * DV, G * D, G * D], 1)
    k, q = (t.view(T, G, D).repeat_interleave(H // G, 1) for t in (k, q))
    v = v.view(T, H, DV)
    if taps:
        step = orc.softplus(x["dt"].double() + p["dt_bias"])
        return orc.linear_scan(q, k, v, torch.exp(-torch.exp(p["a_log"]) * step), step) + p["skip"][:, None] * v
    decay = p["decay"].expand(T, H)
    return orc.linear_scan(q, k, v, decay, torch.ones_like(decay))


def _scan_run(case, H, G, D, DV, taps, counts, dtype, as_parts=False, chunks=False):
    """One sequence in portions of ``counts`` tokens through the kernels, in slot 1 of 3; ``chunks``: the tensor-core form."""
    ops = pkg.ops
    x, par = case
    dp, c = ops.scan_dim_pad(D), par["conv"].shape[0]
    state = torch.full((3, H, DV, dp), 3.0, device=DEV)
    conv_state = torch.full((3, max(taps - 1, 0), c), 3.0, dtype=dtype, device=DEV)
    dev = {k: torch.nn.functional.pad(v, (0, 0) if k == "conv" else (0, -v.numel() % 4)).to(DEV) for k, v in par.items()}
    extra = dict(a_log=dev["a_log"], dt_bias=dev["dt_bias"], conv=dev["conv"].contiguous(), conv_bias=dev["bias"], conv_state=conv_state) if taps else \
        dict(decay=dev["decay"])
    out, at = [], 0
    for n in counts:
        p = portions_of([n], [at], [1])
        r = {k: rows(v[at:at + n], dtype, as_parts) for k, v in x.items()}
        act = BF if chunks else F32
        outs = (torch.full((n, G, dp), 9.0, device=DEV, dtype=act), torch.full((n, G, dp), 9.0, device=DEV, dtype=act),
                torch.zeros(n, H, DV, device=DEV, dtype=act), torch.zeros(n, H, device=DEV), torch.zeros(n, H, device=DEV))
        ops.decay_prep(dtype, n, 1, H, G, D, DV, r["q"], r["k"], r["v"], p, outs, **extra,
                       **(dict(dt=r["dt"], shift_state=n == 1) if taps else {}))
        o = torch.zeros(n, H, DV, device=DEV)
        if chunks:
            q, k, v, *sc = outs
            ops.chunk_scan(1, H, G, dp, DV, q.view(n, -1), k.view(n, -1), v.view(n, -1), *sc, state, p, n, o, skip=dev["skip"] if taps else None)
        else:
            ops.scan(ops.SCAN_DECAY, dtype, 1, H, G, D, DV, *outs, state, p, out=o, skip=dev["skip"] if taps else None,
                     one_token=n == 1 and ops.scan_fusable(dp, DV))
        out.append(o)
        at += n
    assert float((state[0] - 3).abs().max()) == 0 and float((state[2] - 3).abs().max()) == 0
    return torch.cat(out)


SCANS = [(3, 1, 40, 24, 4), (4, 2, 20, 24, 3), (2, 2, 128, 64, 0), (1, 1, 300, 16, 1), (4, 1, 64, 33, 2), (2, 1, 18, 22, 5), (3, 3, 10, 14, 0), (2, 1, 136, 300, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV,taps", SCANS)
def test_decay_scan_in_portions(dtype, H, G, D, DV, taps):
    T = 75
    case = _scan_case(T, H, G, D, DV, taps, 1)
    ref = _scan_ref(case, H, G, D, DV, taps)
    for counts in ([T], [2, 33, 1, 1, 2, 36], [1] * 12 + [63], [2] * 37 + [1]):
        assert rel(_scan_run(case, H, G, D, DV, taps, counts, dtype), ref) < (2e-5 if dtype is F32 else 4e-3 if taps else 2e-5), counts
    if dtype is BF:
        assert rel(_scan_run(case, H, G, D, DV, taps, [30] + [1] * 45, dtype, as_parts=True), ref) < 4e-3
        if ops_take_chunks(D, DV):
            for counts in ([T], [2, 33, 1, 1, 2, 36], [64, 11]):
                assert rel(_scan_run(case, H, G, D, DV, taps, counts, dtype, chunks=True), ref) < 1e-2, counts
            assert rel(_scan_run(case, H, G, D, DV, taps, [T], dtype, as_parts=True, chunks=True), ref) < 1e-2


def ops_take_chunks(dim, vdim):
    return pkg.ops.chunk_scan_supported(pkg.ops.scan_dim_pad(dim), vdim)


@pytest.mark.parametrize("counts", [[200], [64, 128, 8], [1, 63, 65, 71], [2] * 10 + [180], [130, 1, 1, 68]])
@pytest.mark.parametrize("H,G,D,DV", [(4, 2, 64, 24), (2, 1, 128, 64), (3, 3, 192, 136), (1, 1, 256, 96), (96, 4, 128, 128)])
def test_chunk_scan_is_the_recurrence(H, G, D, DV, counts):
    """Operands that bf16 holds exactly: what is left is the state's and the scores' 16 significant bits.  Decays from none to a
    state that is wiped out between two tokens; other sequences in the batch; a padding entry."""
    ops, T = pkg.ops, sum(counts)
    if H == 96 and len(counts) > 3:
        pytest.skip("enough heads for wide column blocks: the plain cuts are enough")
    q, k, v = rand(T, G, D, seed=1, scale=D ** -0.5), rand(T, G, D, seed=2), rand(T, H, DV, seed=3)
    log = -torch.rand(T, H, generator=gen(4)) * torch.logspace(-4, 0.5, H)
    log[T // 2, 0], log[T // 3, H - 1] = -104.0, 0.0
    step, skip = torch.rand(T, H, generator=gen(5)) + 0.1, rand(H, seed=6)
    rep = lambda t: t.double().repeat_interleave(H // G, 1)
    ref = orc.linear_scan(rep(q), rep(k), v.double(), torch.exp(log.double()), step.double()) + skip.double()[:, None] * v.double()
    state = torch.full((4, H, DV, D), 3.0, device=DEV)
    at, outs = 0, []
    for n in counts:
        p = portions_of([5, n, 3], [7, at, 0], [0, 2, -1])
        pad = lambda t: torch.cat([t[:5], t[at:at + n], t[:3]]).to(DEV)
        o = torch.full((n + 8, H, DV), 4.0, device=DEV)
        ops.chunk_scan(3, H, G, D, DV, *(pad(t).to(BF).flatten(1) for t in (q, k, v)), pad(log), pad(step), state, p, n, o, skip=skip.to(DEV))
        assert float((o[5 + n:] - 4).abs().max()) == 0 and float((o[:5] - 4).abs().min()) > 0
        outs.append(o[5:5 + n])
        at += n
    got = torch.cat(outs)
    assert rel(got, ref) < 3e-5
    row = (got.double().cpu() - ref).pow(2).mean((1, 2)).sqrt() / ref.pow(2).mean().sqrt()
    assert float(row.max()) < 2e-4, int(row.argmax())
    assert float((state[1] - 3).abs().max()) == 0 and float((state[3] - 3).abs().max()) == 0


@pytest.mark.parametrize("mq", [64, 400])
@pytest.mark.parametrize("far", [1, 62, 63, 64, 65, 127, 128, 129, 270])
def test_chunk_scan_remembers_a_far_key(far, mq):
    """One key written and asked for ``far`` tokens later, over chunk borders, orthogonal writes in between."""
    ops, T, D, DV, decay = pkg.ops, 400, 64, 16, 0.998
    for at in (0, 3, 63, 64, 127):
        k = torch.zeros(T, 1, D)
        k[:, 0, 1:] = rand(T, D - 1, seed=0)
        k[at, 0], k[at, 0, 0] = 0.0, 1.0
        q = torch.zeros(T, 1, D)
        q[at + far, 0, 0] = 1.0
        v = rand(T, 1, DV, seed=1)
        state, o = torch.zeros(1, 1, DV, D, device=DEV), torch.zeros(T, 1, DV, device=DEV)
        ops.chunk_scan(1, 1, 1, D, DV, *(t.to(BF).to(DEV).flatten(1) for t in (q, k, v)), torch.full((1,), decay, device=DEV).log(),
                       torch.full((1,), 0.5, device=DEV), state, portions_of([T], slots=[0]), mq, o)
        want = torch.zeros(T, DV)
        want[at + far] = 0.5 * v[at, 0] * decay ** far
        assert float((o[:, 0].cpu() - want).abs().max()) < 1e-4


def test_decay_scan_remembers_a_far_key():
    """A value written long ago under one key comes back with the decay of the tokens since, and nothing else does."""
    ops, T, D, DV, decay = pkg.ops, 400, 64, 16, 0.998
    k = torch.zeros(T, 1, D)
    k[:, 0, 1:] = torch.randn(T, D - 1, generator=gen(0))
    k[3, 0], k[3, 0, 0] = 0.0, 1.0
    q = torch.zeros(T, 1, D)
    q[:, 0, 0] = 1.0
    v = torch.randn(T, 1, DV, generator=gen(1))
    state, o = torch.zeros(1, 1, DV, D, device=DEV), torch.zeros(T, 1, DV, device=DEV)
    ops.scan(ops.SCAN_DECAY, F32, 1, 1, 1, D, DV, q.to(DEV), k.to(DEV), v.to(DEV), torch.full((T, 1), decay, device=DEV),
             torch.full((T, 1), 0.5, device=DEV), state, portions_of([T], slots=[0]), out=o)
    o = o.cpu().double()
    want = 0.5 * v[3, 0].double() * decay ** torch.arange(T - 3).double()[:, None]
    assert float(o[:3].abs().max()) == 0 and float((o[3:, 0] - want).abs().max()) < 1e-4


def test_decay_scans_of_unequal_portions_in_one_batch():
    """Four sequences, one of them a padding entry, against each alone; key heads shared by value heads."""
    ops, H, G, D, DV = pkg.ops, 4, 2, 64, 40
    counts, slots = [17, 1, 1, 50], [2, 0, -1, 1]
    T = sum(counts)
    q, k = (torch.randn(T, G, D, generator=gen(i)) for i in range(2))
    v, decay, step = torch.randn(T, H, DV, generator=gen(4)), torch.rand(T, H, generator=gen(5)), torch.rand(T, H, generator=gen(6))
    state, o = torch.zeros(3, H, DV, D, device=DEV), torch.full((T, H, DV), 4.0, device=DEV)
    ops.scan(ops.SCAN_DECAY, F32, 4, H, G, D, DV, *(t.to(DEV) for t in (q, k, v, decay, step)), state, portions_of(counts, slots=slots), out=o)
    at = 0
    for n, s in zip(counts, slots):
        r = slice(at, at + n)
        if s < 0:
            assert float((o[r] - 4).abs().max()) == 0
        else:
            d = lambda t: t[r].double()
            rep = lambda t: d(t).repeat_interleave(2, 1)
            assert rel(o[r], orc.linear_scan(rep(q), rep(k), d(v), d(decay), d(step))) < 1e-5
        at += n


# --------------------------------------------------------------------------- whole models
def _close(got, ref, dtype):
    e = row_error(got, ref)
    assert float(e.max()) < (1e-4 if dtype == "float32" else 8e-2), (float(e.max()), int(e.argmax()))
    assert float(e.median()) < (2e-5 if dtype == "float32" else 2e-2), float(e.median())


def _prompt(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=gen(seed)).tolist()


_REFERENCES = {}


def reference(name, n=300, seed=0):
    """(configuration, checkpoint, tokens, logits in fp64)"""
    key = (name, n, seed)
    if key not in _REFERENCES:
        raw = MODELS[name]
        t, toks = tensors(raw, seed=5), _prompt(n, raw["vocab"], seed)
        _REFERENCES[key] = (raw, t, toks, orc.forward(raw, t, toks, torch.float64))
    return _REFERENCES[key]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_portions_and_decoding(name, dtype):
    raw, t, toks, ref = reference(name)
    r = hc.runner(raw, t, dtype)
    cuts = {"whole": [300], "tokens": [4] + [1] * 60, "pairs": [2] * 40, "mixed": [2, 3, 64, 1, 2, 2, 130, 51, 45],
            "edges": [255, 1, 1, 43], "window": [36, 1, 1, 1, 90, 2, 1, 1], "short": [1, 1, 1, 7]}
    for i, (label, counts) in enumerate(cuts.items()):
        got = run_portions(r, sequence(toks, [5, 2, 9], slot=i % 4), counts)
        _close(got, ref[:sum(counts)], dtype)
    r.exit()


def test_residual_after_every_layer():
    raw, t, toks, _ = reference("odd")
    states = []
    orc.forward(raw, t, toks[:60], torch.float64, states)
    r = hc.runner(raw, t)
    r.engine.collect = []
    run_portions(r, sequence(toks, [1], 0), [60])
    assert len(r.engine.collect) == len(states)
    for got, ref in zip(r.engine.collect, states):
        assert rel(got, ref) < 2e-5
    r.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "even"])
def test_unequal_requests_in_one_batch(name, dtype):
    """Requests of other lengths and places in one step against each alone, then one decode step of all of them."""
    raw, t, toks, ref = reference(name)
    r = hc.runner(raw, t, dtype)
    other = _prompt(90, raw["vocab"], 3)
    ref2 = orc.forward(raw, t, other, torch.float64)
    a, b, c = sequence(toks, [3, 7], 2), sequence(other, [0], 0), sequence(toks, [10, 1], 3)
    run_portions(r, a, [200])
    step = [(a, 99), (b, 80), (c, 2)]
    want = [(i, p) for i, (_, n) in enumerate(step) for p in range(n)]
    lg, _ = r.execute([s for s, _ in step], [n for _, n in step], want)
    lg = lg.cpu()
    _close(lg[:99], ref[200:299], dtype)
    _close(lg[99:179], ref2[:80], dtype)
    _close(lg[179:], ref[:2], dtype)
    for s, n in step:
        s.num_cached_tokens += n
    lg, _ = r.execute([a, b, c], [1, 1, 1])
    assert float(row_error(lg.cpu(), torch.stack([ref[299], ref2[80], ref[2]])).max()) < (1e-4 if dtype == "float32" else 8e-2)
    r.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_and_slots_used_again(dtype):
    """A request on pages and a slot that hold worse than anything a request leaves gives what it gives on fresh ones."""
    raw, t, toks, ref = reference("odd")
    r = hc.runner(raw, t, dtype)
    run_portions(r, sequence(_prompt(300, raw["vocab"], 9), [4, 6], 1), [300])
    for layer in r.engine.state.values():
        for s in layer.values():
            s[1].fill_(float("nan"))
    for k, v in r.engine.kv.values():
        dim = k.shape[2]
        k[:, :, :min(30, dim)] = float("nan")
        v[:, :, :min(30, dim)] = float("nan")
    for counts in ([2, 254, 44], [300], [1] * 20):
        _close(run_portions(r, sequence(toks, [6, 4], 1), counts), ref[:sum(counts)], dtype)
    r.exit()


def test_graphs_and_bucket_padding_change_nothing():
    raw, t, toks, ref = reference("even")
    eager, graphs = hc.runner(raw, t, "bfloat16", max_seqs=8), hc.runner(raw, t, "bfloat16", max_seqs=8, eager=False)
    assert sorted(graphs.graphs) == [1, 2, 4, 8]
    out = []
    for r in (eager, graphs):
        seqs = [sequence(toks[i:], [3 * i, 3 * i + 1], slot=i) for i in range(3)]
        for s in seqs:
            run_portions(r, s, [250])
        steps = []
        for _ in range(12):                              # over the page border at 256
            lg, _ = r.execute(seqs, [1] * 3)
            steps.append(lg.cpu().clone())
            for s in seqs:
                s.num_cached_tokens += 1
        out.append(torch.stack(steps))
    assert float(row_error(out[1].flatten(0, 1), out[0].flatten(0, 1)).max()) < 3e-2
    _close(out[1][:, 0], ref[250:262], "bfloat16")
    for r in (eager, graphs):
        r.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    """520 tokens one by one over two page borders and every window's edge, from the second token on."""
    raw, t, toks, ref = reference("odd", n=521, seed=2)
    r = hc.runner(raw, t, dtype, eager=False, max_seqs=1)
    _close(run_portions(r, sequence(toks, [8, 0, 3], 0), [1] * 521), ref, dtype)
    r.exit()


def test_a_far_prompt():
    """A prompt longer than every window and several pages, whole and in two cuts, and what is decoded behind it."""
    raw, t, toks, ref = reference("even", n=1100, seed=4)
    for dtype in ("float32", "bfloat16"):
        r = hc.runner(raw, t, dtype, max_len=1280, pages=16)
        for counts in ([1088] + [1] * 12, [513, 511, 64, 2, 2, 8]):
            got = run_portions(r, sequence(toks, [5, 2, 9, 11, 3], 0), counts)
            _close(got[-300:], ref[-300:], dtype)
        r.exit()


def _greedy(raw, t, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(orc.forward(raw, t, toks, torch.float32)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("pages,budget", [(12, 1536), (12, 40), (3, 300)])
def test_greedy_generation_through_the_engine(pages, budget):
    """The engine's own loop: prompts cut to the step budget, requests waiting and pre-empted for want of pages."""
    raw = RAGGED
    t = tensors(raw, seed=6)
    prompts = [_prompt(n, raw["vocab"], 20 + n) for n in (245, 3, 1, 60, 252)]
    cfg = pkg.Config(max_num_seqs=4, max_model_len=budget, max_num_batched_tokens=budget, num_kvcache_blocks=pages,
                     decoder_config=hc.config(raw), dtype="float32", enforce_eager=budget < 300)
    cfg.max_model_len = 512
    engine = pkg.LLMEngine.from_config(cfg, weights=hybrid.HybridWeights.build(cfg.decoder_config, t, DEV, F32))
    reqs = [pkg.CausalSequence(p, pkg.SamplingParams(greedy=True, max_new_tokens=14)) for p in prompts]
    done, _ = engine.generate(reqs)
    for req, p in zip(reqs, prompts):
        assert done[req.seq_id][0] == _greedy(raw, t, p, 14)
    assert len(engine.scheduler.block_manager.free_block_ids) == pages
    engine.model_runner.exit()


def test_trace_replay_writes_wanted_logits(tmp_path):
    """The replay program on a model folder: interleaved requests, places wanted, requests that end."""
    from safetensors.torch import save_file
    raw, t, toks, ref = reference("odd")
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    replay = import_module("mineru-diffusion_b200.trace_replay")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:120], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[120:123], "want": [0, 2]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:2], "want": [1]}, {"id": "a", "tokens": toks[123:124], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": toks[:50], "want": [49]}], "end": ["b", "c"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        stdin, sys.stdin = sys.stdin, io.StringIO("".join(json.dumps(s) + "\n" for s in steps))
        try:
            assert replay.main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "300"]) == 0
        finally:
            sys.stdin = stdin
        assert sorted(p.name for p in out.iterdir()) == ["1.f32", "2.f32", "3.f32"]
        for step, places in ((1, [120, 122]), (2, [1, 123]), (3, [49])):
            got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(places), raw["vocab"])
            _close(got, ref[places], dtype)


def test_generate_command_line_runs_a_model_folder(tmp_path, capsys):
    from safetensors.torch import save_file
    t = tensors(EVEN, seed=6)
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(EVEN))
    gen_cli = import_module("mineru-diffusion_b200.generate")
    args = ["--model", str(tmp_path), "--prompt", "5,6,7", "--prompt", "9", "--greedy", "--dtype", "float32", "--max-new-tokens", "8",
            "--max-num-seqs", "2", "--max-model-len", "512"]
    assert gen_cli.main(args) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    for x in lines:
        assert x["tokens"] == _greedy(EVEN, t, x["prompt"], 8)
