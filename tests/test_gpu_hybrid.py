"""Hybrid decoder design on the GPU against its plain restatement: each mechanism alone, then whole models -- prompts,
portions, batches, reuse of pages and slots, long decoding, generation through the engine."""
import pytest
import torch

import hybrid_cases as hc
from hybrid_cases import EVEN, MODELS, ODD, WIDE, hybrid, pkg, row_error, run_portions, sequence
from oracle import hybrid_oracle as orc

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
DTYPES = [F32, BF]
TOL = {F32: 2e-5, BF: 2e-2}          # relative root mean square of one mechanism's output


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rand(*shape, seed=0, scale=1.0, dtype=BF):
    """CPU values that the activation type holds exactly."""
    return (torch.randn(*shape, generator=gen(seed)) * scale).to(dtype).float()


def rel(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    return float((got - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(1e-9))


def portions_of(counts, starts=None, slots=None):
    """(row_seq, cu_q, start, state_slot) device tensors."""
    row_seq = torch.cat([torch.full((n,), i) for i, n in enumerate(counts)])
    cu = torch.tensor([0] + list(counts)).cumsum(0)
    starts = starts or [0] * len(counts)
    slots = slots if slots is not None else list(range(len(counts)))
    return tuple(torch.as_tensor(x).to(torch.int32).to(DEV) for x in (row_seq, cu, starts, slots))


# --------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,m", [(160, 5), (1500, 70)])
def test_residual_norm(dtype, width, m):
    ops, wp = pkg.ops, hybrid.pad128(width)

    def pad(t, cols=wp):
        out = torch.zeros(*t.shape[:-1], cols)
        out[..., :t.shape[-1]] = t
        return out

    res, w = torch.randn(m, width, generator=gen(1)), rand(width, seed=2)
    a, parts = rand(m, width, seed=3), torch.randn(3, m, width, generator=gen(4))
    experts, weights = rand(40, width, seed=5), torch.rand(m, 3, generator=gen(6))
    slots = torch.randint(0, 40, (m, 3), generator=gen(7))
    rd, wd = pad(res).to(DEV), pad(w).to(DEV)
    y = torch.zeros(m, wp, dtype=dtype, device=DEV)
    ops.residual_norm(rd, width, 3e-6, dtype, weight=wd, out=y, add=(ops.Rows(pad(a).to(dtype).to(DEV)), ops.Rows(parts=pad(parts).to(DEV))),
                      moe=(pad(experts).to(dtype).to(DEV), slots.int().to(DEV), weights.to(DEV)))
    ref = res + a + parts.sum(0).to(dtype).float() + (experts[slots] * weights[..., None]).sum(1)
    assert rel(rd[:, :width], ref) < 1e-6 and float(rd[:, width:].abs().sum()) == 0
    assert rel(y[:, :width], orc.rms_norm(ref, w, 3e-6)) < (1e-6 if dtype is F32 else 4e-3)
    # embedding form, id 0 and the last one
    table, ids = rand(50, width, seed=8), torch.tensor([0, 49] * m)[:m]
    ops.residual_norm(rd, width, 3e-6, dtype, weight=wd, out=y, ids=ids.to(DEV), embed=pad(table).to(dtype).to(DEV), embed_scale=2.5)
    assert rel(rd[:, :width], table[ids] * 2.5) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
def test_rms_rows_into_cache_slots(dtype):
    ops = pkg.ops
    x = rand(4, 300, seed=1)
    xd = torch.zeros(4, 384, dtype=dtype, device=DEV)
    xd[:, 128:128 + 100] = x[:, :100].to(dtype).to(DEV)
    w = rand(128, seed=2).to(DEV)
    w[100:] = 0
    cache = torch.full((512, 128), 7.0, dtype=dtype, device=DEV)
    slots = torch.tensor([300, -1, 0, 511], dtype=torch.int32, device=DEV)
    ops.rms_rows([ops.rms_segment(ops.Rows(xd).cols(128), 100, 128, w, 1e-5, cache, slots=slots)], 4, dtype)
    ref = orc.rms_norm(x[:, :100], w[:100].cpu(), 1e-5)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            assert rel(cache[s, :100], ref[i]) < TOL[dtype] and float(cache[s, 100:].abs().sum()) == 0
    assert float((cache[1:300] - 7).abs().sum()) == 0
    assert pkg._lib.device_status() == 0
    slots[0] = 512
    ops.rms_rows([ops.rms_segment(ops.Rows(xd).cols(128), 100, 128, w, 1e-5, cache, slots=slots)], 4, dtype)
    assert pkg._lib.device_status() == 1


def test_pick_token():
    ops = pkg.ops
    lg = torch.randn(6, 700, generator=gen(1))
    lg[2, 650:] = 99.0                      # columns past the vocabulary
    lg[3, 5] = lg[3, 600] = 50.0            # a tie: the lower id
    out, st = torch.zeros(6, dtype=torch.int64, device=DEV), torch.ones(1, dtype=torch.int32, device=DEV)
    ops.pick_token(lg.to(DEV), 650, torch.zeros(6, device=DEV), 3, None, out, st)
    assert out.tolist() == lg[:, :650].argmax(1).tolist() and out[3] == 5 and int(st) == 0
    # temperature: frequencies follow the distribution
    row = torch.full((4000, 4), -30.0, device=DEV)
    row[:, :3] = torch.tensor([1.0, 0.0, -1.0], device=DEV)
    picks = torch.zeros(4000, dtype=torch.int64, device=DEV)
    ops.pick_token(row, 4, torch.full((4000,), 0.5, device=DEV), 11, None, picks)
    freq = torch.bincount(picks, minlength=4).double().cpu() / 4000
    want = torch.softmax(row[0].double().cpu() / 0.5, -1)
    assert float((freq - want).abs().max()) < 0.03


# --------------------------------------------------------------------------- recurrences
def _delta_case(T, H, KH, D, DV, taps, seed):
    x = {n: rand(T, c, seed=seed + i) for i, (n, c) in enumerate((("q", KH * D), ("k", KH * D), ("v", H * DV), ("b", H)))}
    conv = {n: rand(x[n].shape[1], taps, seed=seed + 10 + i, scale=0.6) for i, n in enumerate("qkv")}
    raw, a_log, dt = rand(T, H * D, seed=seed + 20), rand(H, seed=seed + 21) - 2.0, rand(H * D, seed=seed + 22)
    return x, conv, raw, a_log, dt


def _delta_ref(case, H, KH, D, DV):
    x, conv, raw, a_log, dt = case
    d = lambda t: t.double()
    T, rep = raw.shape[0], H // KH
    q, k, v = (orc.short_conv(d(x[n]), d(conv[n])) for n in "qkv")
    q = (orc.unit(q.view(T, KH, D)) * D ** -0.5).repeat_interleave(rep, 1)
    k = orc.unit(k.view(T, KH, D)).repeat_interleave(rep, 1)
    g = torch.exp(-torch.exp(d(a_log))[None, :, None] * orc.softplus(d(raw) + d(dt)).view(T, H, D))
    return orc.delta_scan(q, k, v.view(T, H, DV), g, orc.sigmoid(d(x["b"])))


def _delta_run(case, H, KH, D, DV, counts, dtype, fused=False):
    """One sequence in portions of `counts` tokens through the kernels, in slot 1 of 3."""
    ops = pkg.ops
    x, conv, raw, a_log, dt = case
    dp, C = ops.scan_dim_pad(D), 2 * KH * D + H * DV
    taps = conv["q"].shape[1]
    state = torch.full((3, H, DV, dp), 5.0, device=DEV)             # a slot is never cleared
    cstate = torch.full((3, taps - 1, C), 5.0, dtype=dtype, device=DEV)
    cw = tuple(conv[n].to(DEV) for n in "qkv")
    outs, at = [], 0
    for n in counts:
        p = portions_of([n], [at], [1])
        rows = {k: ops.Rows(torch.nn.functional.pad(v[at:at + n], (0, -v.shape[1] % 4)).to(dtype).to(DEV)) for k, v in x.items()}
        q, k = (torch.full((n, KH, dp), 9.0, device=DEV) for _ in range(2))
        v, beta = torch.zeros(n, H, DV, device=DEV), torch.zeros(n, H, device=DEV)
        ops.delta_prep(dtype, n, 1, H, KH, D, DV, rows["q"], rows["k"], rows["v"], rows["b"], cw, cstate, p, (q, k, v, beta), n == 1)
        r = raw[at:at + n].contiguous().to(DEV)
        common = (ops.SCAN_DELTA, dtype, 1, H, KH, D, DV, q, k, v, beta, None, state, p)
        if fused and n == 1:
            y = torch.zeros(1, H * DV, dtype=dtype, device=DEV)
            gate = torch.full((1, (H * DV + 3) // 4 * 4), 100.0, dtype=dtype, device=DEV)      # sigmoid = 1
            ops.scan(*common, eps=1e-5, raw_decay=ops.Rows(r), a_log=a_log.to(DEV), dt_bias=dt.to(DEV), gate=ops.Rows(gate),
                     norm=torch.ones(DV, device=DEV), y=y)
            outs.append(y.float().view(1, H, DV))
        else:
            g, o, sc = torch.zeros(n, H, dp, device=DEV), torch.zeros(n, H, DV, device=DEV), torch.full((n, H, 4), 9.0, device=DEV)
            ops.channel_decay(r, a_log.to(DEV), dt.to(DEV), q, k, beta, p, g, sc, D)
            ops.scan(*common, g=g, scalars=sc, out=o)
            outs.append(orc.rms(o, 1e-5) if fused else o)
        at += n
    torch.cuda.synchronize()
    assert pkg._lib.device_status() == 0
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,KH,D,DV,taps", [(4, 2, 40, 24, 3), (2, 2, 128, 128, 4), (3, 1, 64, 33, 2), (1, 1, 300, 8, 1), (2, 1, 200, 70, 6)])
def test_delta_scan_in_portions(dtype, H, KH, D, DV, taps):
    case = _delta_case(75, H, KH, D, DV, taps, seed=H)
    ref = _delta_ref(case, H, KH, D, DV)
    for counts in ([75], [2, 1, 30, 2, 40], [16, 16, 43]):
        assert rel(_delta_run(case, H, KH, D, DV, counts, dtype), ref) < TOL[dtype], counts


@pytest.mark.parametrize("H,KH,D,DV,taps", [(4, 2, 40, 24, 3), (2, 2, 128, 128, 4), (2, 1, 256, 64, 4)])
def test_delta_scan_fused_token(H, KH, D, DV, taps):
    assert pkg.ops.scan_fusable(pkg.ops.scan_dim_pad(D), DV)
    case = _delta_case(40, H, KH, D, DV, taps, seed=3)
    ref = orc.rms(_delta_ref(case, H, KH, D, DV), 1e-5)
    assert rel(_delta_run(case, H, KH, D, DV, [30] + [1] * 10, F32, fused=True), ref) < 2e-5


def delta_scalars(q, k, g, beta):
    """The per-token scalars of the prompt scan: k.q, the products with the token before, beta."""
    s = torch.zeros(*beta.shape, 4)
    s[..., 0], s[..., 3] = (k * q).sum(-1), beta
    s[1:, :, 1], s[1:, :, 2] = (g[1:] * k[:-1] * k[1:]).sum(-1), (g[1:] * k[:-1] * q[1:]).sum(-1)
    return s


def test_delta_remembers_a_far_key():
    """A value written under one key long ago, no decay and orthogonal writes since, comes back whole."""
    ops, T, D, DV = pkg.ops, 400, 64, 16
    k = torch.zeros(T, 1, D)
    k[:, 0, 1:] = torch.nn.functional.normalize(torch.randn(T, D - 1, generator=gen(0)), dim=-1)
    k[3, 0], k[3, 0, 0] = 0.0, 1.0
    q = torch.zeros(T, 1, D)
    q[:, 0, 0] = 1.0
    v = torch.randn(T, 1, DV, generator=gen(1))
    sc = delta_scalars(q, k, torch.ones_like(k), torch.ones(T, 1))
    state, o = torch.zeros(1, 1, DV, D, device=DEV), torch.zeros(T, 1, DV, device=DEV)
    ops.scan(ops.SCAN_DELTA, F32, 1, 1, 1, D, DV, q.to(DEV), k.to(DEV), v.to(DEV), None, None, state,
             portions_of([T], slots=[0]), g=torch.ones(T, 1, D, device=DEV), scalars=sc.to(DEV), out=o)
    o = o.cpu()
    assert float(o[:3].abs().max()) == 0 and float((o[3:, 0] - v[3, 0]).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,DV,cap", [(3, 48, 40, 7.5), (2, 128, 256, 15.0), (1, 260, 32, 5.0), (2, 64, 33, 50.0)])
def test_mlstm_scan_in_portions(dtype, H, D, DV, cap):
    ops, T = pkg.ops, 70
    x = {n: rand(T, c, seed=i, scale=s) for i, (n, c, s) in enumerate((("q", H * D, 1), ("k", H * D, 1), ("v", H * DV, 1), ("i", H, 6), ("f", H, 6)))}
    bi, bf = rand(H, seed=8), rand(H, seed=9) + 2
    d = lambda t: t.double()
    li = cap * torch.tanh((d(x["i"]) + d(bi)) / cap)
    lf = -orc.softplus(-cap * torch.tanh((d(x["f"]) + d(bf)) / cap))
    ref = orc.mlstm_scan(d(x["q"]).view(T, H, D) * D ** -0.5, d(x["k"]).view(T, H, D), d(x["v"]).view(T, H, DV), li, lf)
    dp, nb = ops.scan_dim_pad(D), ops.scan_blocks(DV)
    w = 0.5 + torch.rand(H * DV, generator=gen(4))
    for counts in ([T], [2, 33, 1, 1, 2, 31], [1] * 12 + [58]):
        state, mst = torch.full((2, H, DV + 1, dp), 3.0, device=DEV), torch.full((2, H, nb), 3.0, device=DEV)
        outs, normed, at = [], [], 0
        for n in counts:
            p = portions_of([n], [at], [1])
            r = {k: ops.Rows(torch.nn.functional.pad(v[at:at + n], (0, -v.shape[1] % 4)).to(dtype).to(DEV)) for k, v in x.items()}
            q, k, v = (torch.full((n, H, dp), 9.0, device=DEV), torch.full((n, H, dp), 9.0, device=DEV), torch.zeros(n, H, DV, device=DEV))
            gi, gf = torch.zeros(n, H, device=DEV), torch.zeros(n, H, device=DEV)
            ops.mlstm_prep(dtype, n, H, D, DV, r["q"], r["k"], r["v"], r["i"], r["f"], bi.to(DEV), bf.to(DEV), cap, (q, k, v, gi, gf))
            args = (ops.SCAN_MLSTM, dtype, 1, H, H, D, DV, q, k, v, gi, gf, state, p)
            if n == 1 and ops.scan_fusable(dp, DV):
                y = torch.zeros(1, H * DV, dtype=dtype, device=DEV)
                gate = torch.full((1, (H * DV + 3) // 4 * 4), 100.0, dtype=dtype, device=DEV)
                ops.scan(*args, mstate=mst, eps=1e-5, gate=ops.Rows(gate), norm=w.to(DEV), per_head_norm=True, y=y)
                normed.append((at, y.float().view(H, DV)))
                outs.append(torch.zeros(1, H, DV, device=DEV))
            else:
                o, den = torch.zeros(n, H, DV, device=DEV), torch.zeros(n, H, device=DEV)
                ops.scan(*args, mstate=mst, out=o, den=den)
                outs.append(o / den[..., None])
            at += n
        got = torch.cat(outs)
        keep = [t for t in range(T) if t not in {a for a, _ in normed}]
        assert rel(got[keep], ref[keep]) < 2e-5
        for a, y in normed:
            assert rel(y, orc.rms(ref[a], 1e-5) * w.view(H, DV).double()) < (5e-5 if dtype is F32 else 5e-3)


def test_scans_of_unequal_portions_in_one_batch():
    """Four sequences, one of them a padding entry, against each alone."""
    ops, H, D, DV = pkg.ops, 2, 64, 40
    counts, slots = [17, 1, 1, 50], [2, 0, -1, 1]
    T = sum(counts)
    q, k, g = (torch.randn(T, H, D, generator=gen(i)) for i in range(3))
    g, k = torch.sigmoid(g + 2), torch.nn.functional.normalize(k, dim=-1)
    v, beta = torch.randn(T, H, DV, generator=gen(4)), torch.rand(T, H, generator=gen(5))
    state, o = torch.zeros(3, H, DV, D, device=DEV), torch.full((T, H, DV), 4.0, device=DEV)
    ops.scan(ops.SCAN_DELTA, F32, 4, H, H, D, DV, *(t.to(DEV) for t in (q, k, v)), None, None, state, portions_of(counts, slots=slots),
             g=g.to(DEV), scalars=delta_scalars(q, k, g, beta).to(DEV), out=o)
    at = 0
    for n, s in zip(counts, slots):
        r = slice(at, at + n)
        if s < 0:
            assert float((o[r] - 4).abs().max()) == 0
        else:
            assert rel(o[r], orc.delta_scan(*(t[r].double() for t in (q, k, v, g, beta)))) < 2e-5
        at += n


# --------------------------------------------------------------------------- experts
@pytest.mark.parametrize("experts,top,groups,keep", [(12, 3, 3, 2), (16, 4, 4, 3), (6, 2, 1, 1), (160, 8, 8, 3), (4, 4, 4, 4)])
def test_routing(experts, top, groups, keep):
    ops, m = pkg.ops, 37
    z = torch.randn(m, experts, generator=gen(experts)) * 2
    zd = torch.full((m, hybrid.pad128(experts)), 50.0, device=DEV)      # padding columns must not be looked at
    zd[:, :experts] = z.to(DEV)
    ids, w = torch.zeros(m, top, dtype=torch.int32, device=DEV), torch.zeros(m, top, device=DEV)
    skip = torch.zeros(m, dtype=torch.int32, device=DEV)
    skip[5] = -1
    ops.moe_route(ops.Rows(zd), m, experts, top, groups, keep, ids, w, row_slot=skip)
    rid, rw = orc.route(z.double(), {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}})
    for i in range(m):
        if i == 5:
            assert ids[i].tolist() == [-1] * top
            continue
        assert ids[i].tolist() == rid[i].tolist() and rel(w[i], rw[i]) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,kind", [(3, "spread"), (50, "spread"), (300, "spread"), (300, "one"), (1100, "skewed")])
def test_expert_products(dtype, m, kind):
    """Plan, gather and grouped GEMMs: expert loads over several tiles, of none, and all on one expert."""
    ops, E, top, k, n = pkg.ops, 7, 2, 128, 256
    ids = torch.stack([torch.randperm(E, generator=gen(i))[:top] for i in range(m)])
    if kind == "one":
        ids[:] = torch.tensor([6, 2])
    elif kind == "skewed":
        ids[: m - 3] = torch.tensor([1, 5])
    tiles = ops.moe_max_tiles(m, top, E)
    slot, row_token = torch.full((m, top), -9, dtype=torch.int32, device=DEV), torch.full((tiles * 128,), -9, dtype=torch.int32, device=DEV)
    tile_expert, num = torch.full((tiles,), -9, dtype=torch.int32, device=DEV), torch.full((1,), 1, dtype=torch.int32, device=DEV)
    x, w = rand(m, k, seed=1), rand(E, n, k, seed=2, scale=k ** -0.5)
    xs, y = torch.zeros(tiles * 128, k, dtype=dtype, device=DEV), torch.zeros(tiles * 128, n, dtype=dtype, device=DEV)
    ops.moe_plan(ids.int().to(DEV), E, tiles, slot, row_token, tile_expert, num)
    ops.moe_gather(x.to(dtype).to(DEV), xs, row_token, num, tiles)
    ops.gemm_experts(xs, w.to(dtype).to(DEV), y, tile_expert, num, m, act=ops.ACT_RELU2)
    counts = torch.bincount(ids.flatten(), minlength=E)
    assert int(num) == int(((counts + 127) // 128).sum()) <= tiles
    s = slot.cpu().long()
    assert len(set(s.flatten().tolist())) == m * top and (tile_expert.cpu()[s // 128] == ids).all()
    ref = torch.relu(torch.einsum("mk,mtnk->mtn", x, w[ids])) ** 2
    assert rel(y.cpu()[s].float(), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 40, 200])
def test_per_head_products(dtype, m):
    ops, H, n, k = pkg.ops, 5, 384, 128
    x, w = rand(m, H * k, seed=1), rand(H, n, k, seed=2, scale=k ** -0.5)
    y = torch.zeros(m, H * n, dtype=dtype, device=DEV)
    ops.gemm_heads(x.to(dtype).to(DEV), w.to(dtype).to(DEV), y)
    assert rel(y.view(m, H, n), torch.einsum("mhk,hnk->mhn", x.view(m, H, k), w)) < TOL[dtype]


@pytest.mark.parametrize("m,n,k", [(1, 128, 128), (64, 640, 256), (70, 128, 1024), (257, 384, 512), (2100, 256, 256)])
@pytest.mark.parametrize("act", [0, 1])
def test_plain_products(m, n, k, act):
    ops = pkg.ops
    x, w = rand(m, k, seed=1), rand(n, k, seed=2, scale=k ** -0.5)
    ref = x @ w.T
    ref = torch.relu(ref) ** 2 if act else ref
    for dtype, out in ((BF, BF), (BF, F32), (F32, F32)):
        y = torch.zeros(m, n, dtype=out, device=DEV)
        ops.gemm(x.to(dtype).to(DEV), w.to(dtype).to(DEV), y, act=act)
        assert rel(y, ref) < (3e-3 if out is BF else 2e-6), (dtype, out)


# --------------------------------------------------------------------------- latent attention
def _pages(n, seed=0):
    return torch.randperm(n, generator=gen(seed)).int()


@pytest.mark.parametrize("dtype,width,heads,nsplit", [(F32, 128, 5, 1), (F32, 640, 2, 1), (BF, 128, 5, 1), (BF, 256, 20, 3),
                                                      (BF, 384, 16, 7), (BF, 512, 33, 4), (BF, 640, 3, 1)])
def test_latent_attention_rows(dtype, width, heads, nsplit):
    """Random scores over contexts that end at, before and behind page and tile borders."""
    ops = pkg.ops
    pos = [0, 1, 31, 32, 33, 254, 255, 256, 257, 511, 512, 700, -1]
    cache, pages = rand(4 * 256, width, seed=1), _pages(4)[:3]
    q = rand(len(pos), heads, width, seed=2, scale=3.0)
    m = len(pos)
    scale = width ** -0.5
    out = torch.zeros(m, heads * width, dtype=dtype, device=DEV)
    ws = torch.zeros(max(16, ops.latent_attn_workspace_bytes(m, heads, width, nsplit)), dtype=torch.uint8, device=DEV)
    table = pages[None].to(DEV)
    ops.latent_attn(q.reshape(m, -1).to(dtype).to(DEV), cache.to(dtype).to(DEV), table, torch.zeros(m, dtype=torch.int32, device=DEV),
                    torch.tensor(pos, dtype=torch.int32, device=DEV), heads, scale, out, nsplit, ws)
    rows = torch.cat([cache[p * 256:(p + 1) * 256] for p in pages.tolist()]).double()
    for i, p in enumerate(pos):
        if p < 0:
            continue
        a = torch.softmax(q[i].double() @ rows[:p + 1].T * scale, -1)
        assert rel(out[i].view(heads, width), a @ rows[:p + 1]) < TOL[dtype], p
    assert pkg._lib.device_status() == 0


@pytest.mark.parametrize("dtype,width,nsplit", [(F32, 128, 1), (BF, 256, 1), (BF, 256, 5)])
def test_latent_attention_finds_the_one_key(dtype, width, nsplit):
    """One key stands out: visible from its own position on, wherever it lies; the key after the row's never is."""
    ops, pages = pkg.ops, _pages(4, seed=3)[:3]
    where = [0, 1, 31, 32, 127, 128, 255, 256, 511, 512, 600]
    cache = rand(4 * 256, width, seed=5, scale=0.05)
    flat = lambda p: int(pages[p // 256]) * 256 + p % 256
    mark = rand(len(where), width, seed=6)
    q, pos, expect = [], [], []
    for i, p in enumerate(where):
        cache[flat(p)] = mark[i]
        for at in (p - 1, p, p + 1, 640):
            if at >= 0:
                q.append(mark[i] * 8)
                pos.append(at)
                expect.append(mark[i] if at >= p else None)
    m = len(q)
    qd = torch.stack(q).to(dtype).to(DEV)
    out = torch.zeros(m, width, dtype=dtype, device=DEV)
    ws = torch.zeros(max(16, ops.latent_attn_workspace_bytes(m, 1, width, nsplit)), dtype=torch.uint8, device=DEV)
    ops.latent_attn(qd, cache.to(dtype).to(DEV), pages[None].to(DEV), torch.zeros(m, dtype=torch.int32, device=DEV),
                    torch.tensor(pos, dtype=torch.int32, device=DEV), 1, 1.0, out, nsplit, ws)
    for i in range(m):
        got = out[i].float().cpu()
        if expect[i] is not None:
            assert rel(got, expect[i]) < 2e-2, pos[i]
        else:
            assert float(got @ q[i] / 8) < 0.5 * float((q[i] / 8).pow(2).sum()), pos[i]


@pytest.mark.parametrize("portion", [(0, 700), (0, 1), (1, 300), (255, 2), (256, 257), (640, 60), (500, 33)])
def test_causal_attention_of_a_portion(portion):
    """Queries of the last tokens against all keys; two sequences, of which the other one is a whole prompt; a marked key
    just behind every row's own position must stay unseen."""
    ops, heads, scale = pkg.ops, 3, 0.1
    start, n = portion
    lens, qs = [start + n, 130], [n, 130]
    total_k, total_q = sum(lens), sum(qs)
    k, v = rand(total_k, heads, 128, seed=1), rand(total_k, heads, 128, seed=2)
    q = rand(total_q, heads, 128, seed=3, scale=2.0)
    q[n - 1] = k[0] * 8                                # the last row of the portion looks at the first key
    if n > 1:
        q[n - 2] = k[start + n - 1] * 8                # and the one before at the key behind it
    cu = lambda x: torch.tensor([0] + x).cumsum(0).int().to(DEV)
    out = torch.zeros(total_q, heads, 128, dtype=BF, device=DEV)
    ops.causal_attn_varlen(q.to(BF).to(DEV), k.to(BF).to(DEV), v.to(BF).to(DEV), cu(qs), cu(lens), 2, max(qs), scale, out)
    out = out.float().cpu()
    qo = ko = 0
    for L, nq in zip(lens, qs):
        s = torch.einsum("ihd,jhd->hij", q[qo:qo + nq].double(), k[ko:ko + L].double()) * scale
        seen = torch.arange(L)[None] <= torch.arange(L - nq, L)[:, None]
        ref = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), -1), v[ko:ko + L].double())
        assert rel(out[qo:qo + nq], ref) < 1e-2
        assert rel(out[qo + nq - 1], ref[-1]) < 1e-2 and rel(out[qo + max(nq - 2, 0)], ref[max(nq - 2, 0)]) < 1e-2
        qo, ko = qo + nq, ko + L


def test_gather_latents_crosses_pages():
    ops, width = pkg.ops, 128
    cache = rand(5 * 256, width, seed=1)
    table = torch.tensor([[4, 0, -1], [2, 3, 1]], dtype=torch.int32, device=DEV)
    cu = torch.tensor([0, 300, 300 + 513], dtype=torch.int32, device=DEV)
    for dtype in DTYPES:
        out = torch.zeros(813, width, dtype=dtype, device=DEV)
        ops.gather_latents(cache.to(dtype).to(DEV), table, cu, 2, out)
        ref = torch.cat([cache[4 * 256:5 * 256], cache[:44], cache[512:768], cache[768:1024], cache[256:257]])
        assert torch.equal(out.float().cpu(), ref)


# --------------------------------------------------------------------------- whole models
def _close(got, ref, dtype):
    e = row_error(got, ref)
    assert float(e.max()) < (1e-4 if dtype == "float32" else 8e-2), float(e.max())
    assert float(e.median()) < (2e-5 if dtype == "float32" else 2e-2), float(e.median())


def _prompt(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=gen(seed)).tolist()


_REFERENCES = {}


def reference(name, dtype="float32", n=300, seed=0):
    """(configuration, checkpoint, tokens, logits in fp64); bf16 runs take the model without close routing calls."""
    key = (name, dtype, n, seed)
    if key not in _REFERENCES:
        raw = (MODELS if dtype == "float32" else hc.SETTLED)[name]
        t, toks = hc.tensors(raw, seed=5), _prompt(n, raw["vocab"], seed)
        _REFERENCES[key] = (raw, t, toks, orc.forward(raw, t, toks, torch.float64))
    return _REFERENCES[key]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_portions_and_decoding(name, dtype):
    raw, t, toks, ref = reference(name, dtype)
    r = hc.runner(raw, t, dtype)
    cuts = {"whole": [300], "tokens": [4] + [1] * 40, "pairs": [2] * 20, "mixed": [2, 3, 64, 1, 2, 2, 130, 51, 45],
            "edges": [255, 1, 1, 43], "short": [1, 1, 1, 7]}
    for i, (label, counts) in enumerate(cuts.items()):
        seq = sequence(toks, [5, 2, 9], slot=i % 4)
        got = run_portions(r, seq, counts)
        _close(got, ref[:sum(counts)], dtype)
    r.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["odd", "even"])
def test_unequal_requests_in_one_batch(name, dtype):
    """Requests of other lengths and places in one step against each alone, then one decode step of all of them."""
    raw, t, toks, ref = reference(name, dtype)
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


def test_pages_and_slots_used_again():
    """A request on pages and a slot full of another's latents and state gives what it gives on fresh ones."""
    raw, t, toks, ref = reference("odd")
    r = hc.runner(raw, t)
    run_portions(r, sequence(_prompt(300, raw["vocab"], 9), [4, 6], 1), [300])
    for layer in r.engine.state.values():               # and worse than anything a request leaves
        for s in layer.values():
            s[1].fill_(float("nan"))
    for cache in r.engine.latents.values():
        cache[6 * 256:].fill_(1e3)
    _close(run_portions(r, sequence(toks, [6, 4], 1), [2, 254, 44]), ref, "float32")
    r.exit()


def test_graphs_and_bucket_padding_change_nothing():
    raw, t, toks, ref = reference("even", "bfloat16")
    eager, graphs = hc.runner(raw, t, "bfloat16", max_seqs=8), hc.runner(raw, t, "bfloat16", max_seqs=8, eager=False)
    assert sorted(graphs.graphs) == [1, 2, 4, 8]
    rows = []
    for r in (eager, graphs):
        seqs = [sequence(toks[i:], [3 * i, 3 * i + 1], slot=i) for i in range(3)]
        for s in seqs:
            run_portions(r, s, [250])
        out = []
        for _ in range(12):                              # over the page border at 256
            lg, _ = r.execute(seqs, [1] * 3)
            out.append(lg.cpu().clone())
            for s in seqs:
                s.num_cached_tokens += 1
        rows.append(torch.stack(out))
    e = row_error(rows[1].flatten(0, 1), rows[0].flatten(0, 1))
    assert float(e.max()) < 3e-2
    _close(rows[1][:, 0], ref[250:262], "bfloat16")
    for r in (eager, graphs):
        r.exit()


def test_long_decoding():
    """520 tokens one by one over two page borders, from the second token on."""
    raw, t, toks, ref = reference("odd", n=521, seed=2)
    r = hc.runner(raw, t, eager=False, max_seqs=1)
    got = run_portions(r, sequence(toks, [8, 0, 3], 0), [1] * 521)
    _close(got, ref, "float32")
    r.exit()


def _greedy(raw, t, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(orc.forward(raw, t, toks, torch.float32)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("pages,budget", [(12, 1536), (12, 40), (3, 300)])
def test_greedy_generation_through_the_engine(pages, budget):
    """The engine's own loop: prompts cut to the step budget, requests waiting and pre-empted for want of pages."""
    raw = WIDE
    t = hc.tensors(raw, seed=6)
    prompts = [_prompt(n, raw["vocab"], 20 + n) for n in (245, 3, 1, 60, 252)]
    cfg = pkg.Config(max_num_seqs=4, max_model_len=budget, max_num_batched_tokens=budget, num_kvcache_blocks=pages,
                     decoder_config=hc.config(raw), dtype="float32") if budget >= 300 else \
        pkg.Config(max_num_seqs=4, max_model_len=budget, max_num_batched_tokens=budget, num_kvcache_blocks=pages,
                   decoder_config=hc.config(raw), dtype="float32", enforce_eager=True)
    cfg.max_model_len = 512
    w = hybrid.HybridWeights.build(cfg.decoder_config, t, DEV, F32)
    engine = pkg.LLMEngine.from_config(cfg, weights=w)
    reqs = [pkg.CausalSequence(p, pkg.SamplingParams(greedy=True, max_new_tokens=14)) for p in prompts]
    done, _ = engine.generate(reqs)
    for req, p in zip(reqs, prompts):
        assert done[req.seq_id][0] == _greedy(raw, t, p, 14)
    assert len(engine.scheduler.block_manager.free_block_ids) == pages
    engine.model_runner.exit()


def test_sampling_repeats_with_its_seed():
    raw = WIDE
    t = hc.tensors(raw, seed=6)
    outs = []
    for seed in (1, 1, 2):
        cfg = pkg.Config(max_num_seqs=2, max_model_len=512, max_num_batched_tokens=512, num_kvcache_blocks=6,
                         decoder_config=hc.config(raw))
        engine = pkg.LLMEngine.from_config(cfg, weights=hybrid.HybridWeights.build(cfg.decoder_config, t, DEV, BF), noise_seed=seed)
        req = pkg.CausalSequence([5, 6, 7], pkg.SamplingParams(temperature=1.0, max_new_tokens=20))
        outs.append(engine.generate([req])[0][req.seq_id][0])
        engine.model_runner.exit()
    assert outs[0] == outs[1] != outs[2]


def test_step_function_refuses_what_it_cannot_run():
    raw, t, toks, _ = reference("odd")
    r = hc.runner(raw, t)
    with pytest.raises(AssertionError, match="pages"):
        r.execute([sequence(toks, [1], 0)], [257])
    with pytest.raises(AssertionError, match="state slot"):
        r.execute([sequence(toks, [1], -1)], [3])
    with pytest.raises(RuntimeError, match="status word"):
        r.execute([sequence([raw["vocab"]], [1], 0)], [1])
    r.exit()


def test_trace_replay_writes_wanted_logits(tmp_path):
    """The replay program on a model folder: interleaved requests, places wanted, requests that end."""
    import io
    import json
    import sys
    from importlib import import_module
    from safetensors.torch import save_file
    raw, t, toks, ref = reference("odd")
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:120], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[120:123], "want": [0, 2]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:2], "want": [1]}, {"id": "a", "tokens": toks[123:124], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": toks[:50], "want": [49]}], "end": ["b", "c"]}]
    replay = import_module("mineru-diffusion_b200.trace_replay")
    stdin, sys.stdin = sys.stdin, io.StringIO("".join(json.dumps(s) + "\n" for s in steps))
    try:
        assert replay.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "300"]) == 0
    finally:
        sys.stdin = stdin
    assert sorted(p.name for p in out.iterdir()) == ["1.f32", "2.f32", "3.f32"]
    for step, places in ((1, [120, 122]), (2, [1, 123]), (3, [49])):
        got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(places), raw["vocab"])
        _close(got, ref[places], "float32")


def test_generate_command_line_runs_a_model_folder(tmp_path, capsys):
    import json
    from importlib import import_module
    from safetensors.torch import save_file
    t = hc.tensors(WIDE, seed=6)
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(WIDE))
    gen = import_module("mineru-diffusion_b200.generate")
    args = ["--model", str(tmp_path), "--prompt", "5,6,7", "--prompt", "9", "--greedy", "--dtype", "float32", "--max-new-tokens", "8",
            "--max-num-seqs", "2", "--max-model-len", "512"]
    assert gen.main(args) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert [x["prompt"] for x in lines] == [[5, 6, 7], [9]]
    for x in lines:
        assert x["tokens"] == _greedy(WIDE, t, x["prompt"], 8)
    assert gen.main(args + ["--max-new-tokens", "600"]) == 2
