"""Nipadra decoder design on the host: configuration, registry, weight layout, and the plain restatement's own invariants.
No GPU."""
import json
import math
from importlib import import_module

import pytest
import torch

from hybrid_cases import config, hybrid, pkg
from nipadra_cases import EVEN, MODELS, ODD, RAGGED, lightning, mamba, model, parallel, tensors, window
from oracle import nipadra_oracle as orc


def test_config_reads_every_size():
    c = config(ODD)
    assert (c.vocab_size, c.hidden_size, c.residual_scale, c.rms_norm_eps, c.embed_scale) == (333, 160, 1.9, 3e-6, 1.0)
    assert [l.type for l in c.layers] == ["lightning", "parallel", "parallel", "lightning"]
    assert [l.mlp.ff if l.mlp else None for l in c.layers] == [None, 100, None, 72] and c.layers[1].mlp.act == "relu_glu"
    light, left, right = c.layers[0].mixer, c.layers[1].mixer.left, c.layers[1].mixer.right
    assert (light.heads, light.kv_heads, light.dim, light.vdim, light.decay, light.conv) == (3, 3, 40, 24, [0.5, 0.93, 0.9995], 0)
    assert (left.heads, left.kv_heads, left.dim, left.window, left.rot_dims, left.rot_base, left.scale) == (6, 2, 40, 37, 24, 5e3, 0.2)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.conv, right.norm_groups, right.decay) == (4, 2, 20, 24, 3, 3, None)
    assert (c.layers[1].mixer.left_scale, c.layers[1].mixer.right_scale) == (0.7, 1.3)


@pytest.mark.parametrize("layers", [
    [lightning(3, 8, 8, [0.5, 0.5], None)],
    [parallel(window(3, 2, 8, 4, 8, 1e4, 1.0), mamba(2, 8, 8, 1, 2, 1), (1, 1), None)],
    [parallel(window(2, 2, 8, 4, 10, 1e4, 1.0), mamba(2, 8, 8, 1, 2, 1), (1, 1), None)],
    [parallel(window(2, 2, 8, 4, 3, 1e4, 1.0), mamba(2, 8, 8, 1, 2, 1), (1, 1), None)],
    [parallel(window(2, 2, 8, 4, 8, 1e4, 1.0), mamba(3, 8, 8, 2, 2, 1), (1, 1), None)],
    [parallel(window(2, 2, 8, 4, 8, 1e4, 1.0), mamba(2, 8, 8, 1, 2, 3), (1, 1), None)],
    [parallel({**window(2, 2, 8, 4, 8, 1e4, 1.0), "vdim": 16}, mamba(2, 8, 8, 1, 2, 1), (1, 1), None)],
    [{"type": "mlstm", "mixer": {}, "mlp": None}],
    [lightning(1, 8, 8, [0.5], {"kind": "moe"})],
])
def test_config_refuses_what_cannot_be(layers):
    with pytest.raises(ValueError):
        config(model(64, 32, layers))


def test_registry_chooses_by_config_json(tmp_path):
    registry = import_module("mineru-diffusion_b200.engine.registry")
    (tmp_path / "config.json").write_text(json.dumps(EVEN))
    cfg = pkg.Config(model=str(tmp_path), num_kvcache_blocks=4, num_state_slots=2)
    assert isinstance(cfg.decoder_config, pkg.HybridConfig) and cfg.decoder_config.design.post_norm
    arch = registry.of_config(cfg.decoder_config)
    assert arch.name == "Nipadra" and arch.load("scheduler") is pkg.CausalScheduler and arch.load("runner") is pkg.CausalModelRunner


@pytest.mark.parametrize("name", sorted(MODELS))
def test_weight_layout_keeps_the_products(name):
    """The stacked input matrix and the joined output matrix give the products of the checkpoint's own."""
    raw = MODELS[name]
    cfg, t = config(raw), {k: v.float() for k, v in tensors(raw, seed=1).items()}
    w = hybrid.HybridWeights.build(cfg, t, "cpu", torch.float32)
    width, wp = cfg.hidden_size, hybrid.pad128(cfg.hidden_size)
    h = torch.randn(3, width)
    hp = torch.zeros(3, wp)
    hp[:, :width] = h
    for i, (layer, lw) in enumerate(zip(cfg.layers, w.layers)):
        y = hp @ lw["in"].T
        if layer.type == "lightning":
            subs = [("mix.", [t[f"l{i}.mix.{n}"] for n in "gvkq"])]
        else:
            r = layer.mixer.right
            nv, nk = r.heads * r.vdim, r.kv_heads * r.dim
            subs = [("mix.left.", [t[f"l{i}.mix.left.{n}"] for n in "qkg"]),
                    ("mix.right.", t[f"l{i}.mix.right.in"].split([nv, nv, nk, nk, r.heads]))]
        total = torch.zeros(3, width)
        o = torch.zeros(3, lw["o"].shape[1])
        for sub, (pre, mats) in zip(lw["parts"], subs):
            assert len(sub["starts"]) == len(mats) and sub["out"] % 8 == 0
            for m, s in zip(mats, sub["starts"]):
                assert s % 4 == 0 and torch.allclose(y[:, s:s + m.shape[0]], h @ m.T, atol=1e-4)
            out = t[f"l{i}.{pre}o"]
            part = torch.randn(3, out.shape[1])
            o[:, sub["out"]:sub["out"] + out.shape[1]] = part
            total += part @ out.T
        assert torch.allclose((o @ lw["o"].T)[:, :width], total, atol=1e-3)
        assert torch.equal(lw["norm1"][:width], 1 + t[f"l{i}.norm1"]) and float(lw["norm1"][width:].abs().sum()) == 0
        if layer.mlp is not None:
            fp = lw["up"].shape[0] // 2
            assert torch.equal(lw["up"][:layer.mlp.ff, :width], t[f"l{i}.mlp.gate"])
            assert torch.equal(lw["up"][fp:fp + layer.mlp.ff, :width], t[f"l{i}.mlp.up"])
    assert w.head is w.embed and w.embed.shape[0] % 128 == 0 and torch.equal(w.final_norm[:width], 1 + t["final.norm"])


def test_weights_name_every_tensor_once():
    cfg, t = config(ODD), tensors(ODD)
    for name in ("l1.mix.right.conv.b", "l1.mix.left.k.norm", "l0.mix.g", "l1.mlp.gate", "final.norm"):
        missing = dict(t)
        del missing[name]
        with pytest.raises(KeyError, match=name):
            hybrid.HybridWeights.build(cfg, missing, "cpu")
    with pytest.raises(ValueError, match="not parameters"):
        hybrid.HybridWeights.build(cfg, {**t, "head": t["embed"]}, "cpu")
    with pytest.raises(ValueError, match="shape"):
        hybrid.HybridWeights.build(cfg, {**t, "l1.mix.right.in": t["l1.mix.right.in"][:-1]}, "cpu")


def test_bytes_of_cache_and_state():
    c = config(EVEN)
    # two attention layers: 2 key heads of 128, 1 of 64; K and V
    assert hybrid.bytes_per_page(c, torch.bfloat16) == 256 * 2 * 2 * (2 * 128 + 64)
    state = 4 * (8 * 64 * 128 + 4 * 64 * 64 + 2 * 96 * 64)
    conv = 2 * (3 * (512 + 2 * 2 * 128) + 1 * (192 + 2 * 64))
    assert hybrid.bytes_per_slot(c, torch.bfloat16) == state + conv
    w = hybrid.HybridWeights.build(c, tensors(EVEN), "cpu")
    assert w.nbytes() > sum(v.numel() * 2 for v in tensors(EVEN).values())


# --------------------------------------------------------------------------- the restatement itself
def test_oracle_window_edges_and_sink():
    """One key stands out: it is seen up to window - 1 tokens later; where every score is very negative the sink takes all."""
    T, W = 12, 4
    k = torch.zeros(T, 1, 2, dtype=torch.float64)
    k[5, 0, 0] = 1.0
    v = torch.zeros(T, 1, 1, dtype=torch.float64)
    v[5] = 1.0
    q = torch.full((T, 1, 2), 50.0, dtype=torch.float64)
    o = orc.window_sink_attention(q, k, v, 1.0, W).flatten()
    assert all(abs(float(x) - (1.0 if 5 <= i < 5 + W else 0.0)) < 1e-9 for i, x in enumerate(o))
    ones = torch.ones(T, 1, 2, dtype=torch.float64)
    o = orc.window_sink_attention(-q, ones, ones, 1.0, W)
    assert float(o.abs().max()) < 1e-30
    o = orc.window_sink_attention(0 * q, ones, ones, 1.0, W).mean(-1).flatten()
    assert torch.allclose(o, torch.tensor([min(i + 1, W) / (min(i + 1, W) + 1) for i in range(T)], dtype=torch.float64))


def test_oracle_rotation_is_relative():
    x = torch.randn(2, 3, 8, dtype=torch.float64)
    a, b = (orc.rotate(x[i:i + 1], 6, 100.0, torch.tensor([p])) for i, p in ((0, 11), (1, 7)))
    c, d = (orc.rotate(x[i:i + 1], 6, 100.0, torch.tensor([p])) for i, p in ((0, 104), (1, 100)))
    assert torch.allclose((a * b).sum(-1), (c * d).sum(-1)) and torch.equal(a[..., 6:], x[:1, :, 6:])


def test_oracle_scan_is_a_weighted_sum():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(6, 1, 3, generator=g, dtype=torch.float64) for _ in range(3))
    decay, step = (torch.rand(6, 1, generator=g, dtype=torch.float64) for _ in range(2))
    o = orc.linear_scan(q, k, v, decay, step)
    for t in range(6):
        ref = sum(step[j, 0] * math.prod(decay[j + 1:t + 1, 0].tolist()) * (k[j, 0] @ q[t, 0]) * v[j, 0] for j in range(t + 1))
        assert torch.allclose(o[t, 0], ref)


def test_oracle_group_norm_gates_first():
    y, z = torch.randn(2, 6, dtype=torch.float64), torch.randn(2, 6, dtype=torch.float64)
    w = torch.randn(6, dtype=torch.float64)
    got = orc.gated_group_norm(y, z, w, 2, 1e-5)
    g = y * z / (1 + torch.exp(-z))
    for p in (slice(0, 3), slice(3, 6)):
        assert torch.allclose(got[:, p], g[:, p] / (g[:, p].pow(2).mean(-1, keepdim=True) + 1e-5).sqrt() * w[p])


@pytest.mark.parametrize("name", sorted(MODELS))
def test_oracle_is_causal(name):
    """A prefix of the tokens gives the same logits."""
    raw = MODELS[name]
    t = tensors(raw, seed=2)
    toks = torch.randint(0, raw["vocab"], (24,), generator=torch.Generator().manual_seed(1)).tolist()
    full = orc.forward(raw, t, toks, torch.float64)
    assert torch.allclose(full[:9], orc.forward(raw, t, toks[:9], torch.float64))
    assert full.shape == (24, raw["vocab"]) and torch.isfinite(full).all()


def test_ragged_sizes_are_what_they_claim():
    c = config(RAGGED)
    assert any(l.mixer.left.window == 1 for l in c.layers if l.type == "parallel")
    assert any(l.mixer.left.rot_dims == 0 for l in c.layers if l.type == "parallel")
    assert any(l.mixer.right.conv == 1 for l in c.layers if l.type == "parallel")
