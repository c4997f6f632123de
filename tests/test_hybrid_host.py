"""Hybrid decoder design on the host: configuration, registry, weight layout, scheduler, state slots, and the plain
restatement's own invariants.  No GPU."""
import json

import pytest
import torch

from hybrid_cases import EVEN, MODELS, ODD, WIDE, config, delta, dense, hybrid, latent, mlstm, model, moe, pkg, tensors
from oracle import hybrid_oracle as orc


def test_config_reads_every_size():
    c = config(ODD)
    assert (c.vocab_size, c.hidden_size, c.embed_scale, c.rms_norm_eps) == (333, 160, 2.5, 3e-6)
    assert [l.type for l in c.layers] == ["channel_delta", "mlstm", "latent_attention", "channel_delta", "latent_attention", "mlstm"]
    assert c.layers[1].mlp is None and c.layers[4].mixer.kv_from == 2
    assert (c.layers[0].mlp.groups, c.layers[0].mlp.keep, c.layers[0].mlp.shared_ff) == (3, 2, 56)
    assert (c.layers[3].mlp.groups, c.layers[3].mlp.keep, c.layers[3].mlp.shared_ff) == (1, 1, None)
    assert c.layers[5].mixer.gate_cap == 30.0


@pytest.mark.parametrize("layers", [
    [latent(2, 8, 8, 8, 8, 1.0, None, kv_from=0)],
    [latent(2, 8, 8, 8, 8, 1.0, None), latent(2, 8, 8, 8, 16, 1.0, None, kv_from=0)],
    [latent(2, 8, 8, 8, 8, 1.0, None), latent(2, 8, 8, 8, 8, 1.0, None, kv_from=0), latent(2, 8, 8, 8, 8, 1.0, None, kv_from=1)],
    [delta(3, 2, 8, 8, 2, None)],
    [mlstm(2, 8, 8, 1.0, moe(6, 2, 8, {"count": 4, "keep": 2}))],
    [mlstm(2, 8, 8, 1.0, moe(8, 3, 8, {"count": 4, "keep": 1}))],
    [{"type": "other", "mixer": {}, "mlp": None}],
])
def test_config_refuses_what_cannot_be(layers):
    with pytest.raises(ValueError):
        config(model(64, 32, layers))


def test_registry_chooses_by_config_json(tmp_path):
    from importlib import import_module
    registry = import_module("mineru-diffusion_b200.engine.registry")
    (tmp_path / "config.json").write_text(json.dumps(EVEN))
    cfg = pkg.Config(model=str(tmp_path), num_kvcache_blocks=4, num_state_slots=2)
    assert isinstance(cfg.decoder_config, pkg.HybridConfig)
    arch = registry.of_config(cfg.decoder_config)
    assert arch.load("scheduler") is pkg.CausalScheduler and arch.load("runner") is pkg.CausalModelRunner
    assert registry.of_config(pkg.DecoderConfig()).load("runner") is pkg.ModelRunner
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "none such"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        pkg.Config(model=str(tmp_path))


@pytest.mark.parametrize("name", sorted(MODELS))
def test_weight_layout_keeps_the_products(name):
    """Stacked, padded and per-head transposed matrices give the products of the checkpoint's own."""
    raw = MODELS[name]
    cfg, t = config(raw), tensors(raw, seed=1)
    w = hybrid.HybridWeights.build(cfg, t, "cpu", torch.float32)
    width, wp = cfg.hidden_size, hybrid.pad128(cfg.hidden_size)
    h = torch.randn(3, width)
    hp = torch.zeros(3, wp)
    hp[:, :width] = h
    for i, (layer, lw) in enumerate(zip(cfg.layers, w.layers)):
        y = hp @ lw["in"].T
        if layer.type == "latent_attention":
            mx = layer.mixer
            q = torch.randn(3, mx.heads, mx.dim)
            c = torch.randn(4, mx.kv_rank)
            k = (c @ t[f"l{i}.mix.uk"].float().T).view(4, mx.heads, mx.dim)
            cp = torch.zeros(4, lw["uk_t"].shape[1])
            cp[:, :mx.kv_rank] = c
            qp = torch.zeros(3, mx.heads, lw["uk_t"].shape[2])
            qp[:, :, :mx.dim] = q
            folded = torch.einsum("thd,hrd->thr", qp, lw["uk_t"])
            assert torch.allclose(torch.einsum("thr,jr->thj", folded, cp), torch.einsum("thd,jhd->thj", q, k), atol=2e-3)
            names = ["dq"] + (["dkv"] if mx.kv_from is None else [])
        else:
            names = ["a1", "g1", "q", "k", "v", "b"] if layer.type == "channel_delta" else ["q", "k", "v", "g", "i", "f"]
        for n, s in zip(names, lw["starts"]):
            ref = h @ t[f"l{i}.mix.{n}"].float().T
            assert s % 4 == 0 and torch.allclose(y[:, s:s + ref.shape[1]], ref, atol=1e-4)


def test_weights_name_every_tensor_once():
    cfg, t = config(WIDE), tensors(WIDE)
    missing = dict(t)
    del missing["l1.mix.a2"]
    with pytest.raises(KeyError, match="l1.mix.a2"):
        hybrid.HybridWeights.build(cfg, missing, "cpu")
    with pytest.raises(ValueError, match="not parameters"):
        hybrid.HybridWeights.build(cfg, {**t, "l9.extra": torch.zeros(2)}, "cpu")
    with pytest.raises(ValueError, match="shape"):
        hybrid.HybridWeights.build(cfg, {**t, "head": t["head"][:-1]}, "cpu")


def test_loader_reads_safetensors(tmp_path):
    from safetensors.torch import save_file
    t = tensors(WIDE, seed=4)
    save_file(t, str(tmp_path / "model.safetensors"))
    w = pkg.load_hybrid_weights(str(tmp_path), config(WIDE), "cpu", torch.float32)
    assert torch.equal(w.embed[:, :96], t["embed"].float()) and w.head.shape[0] % 128 == 0
    with pytest.raises(FileNotFoundError):
        pkg.load_hybrid_weights(str(tmp_path / "empty"), config(WIDE), "cpu")


# --------------------------------------------------------------------------- scheduler
class FakeRunner:
    """Produces the token after the last one; checks what the scheduler hands it."""

    def __init__(self, config):
        self.config, self.steps, self.seen = config, [], {}

    def call(self, _, seqs, is_prefill):
        assert sum(s.num_scheduled for s in seqs) <= self.config.max_num_batched_tokens or not is_prefill
        held = [p for s in seqs for p in s.block_table]
        assert len(held) == len(set(held)) and len({s.state_slot for s in seqs}) == len(seqs)
        for s in seqs:
            assert s.num_scheduled >= 1 and s.num_cached_tokens + s.num_scheduled <= len(s)
            assert 256 * len(s.block_table) >= s.num_cached_tokens + s.num_scheduled and s.state_slot >= 0
            if s.num_cached_tokens + s.num_scheduled == len(s):
                s.next_token = (s.last_token + 1) % 50
        self.steps.append((is_prefill, [s.num_scheduled for s in seqs]))
        return 0


def _engine(pages, slots, seqs=4, budget=300):
    cfg = pkg.Config(max_num_seqs=seqs, max_model_len=budget, max_num_batched_tokens=budget, num_kvcache_blocks=pages,
                     num_state_slots=slots, decoder_config=config(EVEN))
    return pkg.LLMEngine(cfg, FakeRunner(cfg)), cfg


def test_scheduler_cuts_prompts_and_finishes():
    engine, _ = _engine(pages=16, slots=4)
    reqs = [pkg.CausalSequence([i] * n, pkg.SamplingParams(greedy=True, max_new_tokens=5)) for i, n in enumerate((700, 3, 257, 1, 40))]
    done, _ = engine.generate(reqs)
    assert {k: len(v[0]) for k, v in done.items()} == {r.seq_id: 5 for r in reqs}
    for i, r in enumerate(reqs):
        assert done[r.seq_id][0] == [(i + 1 + j) % 50 for j in range(5)]
    prefills = [c for p, c in engine.model_runner.steps if p]
    assert prefills[0] == [300] and max(sum(c) for c in prefills) <= 300
    assert len(engine.scheduler.block_manager.free_block_ids) == 16 and len(engine.scheduler.state_manager.free) == 4


def test_scheduler_preempts_and_recomputes():
    """Three requests that grow past a page with too few pages: the youngest gives way and still finishes."""
    engine, _ = _engine(pages=4, slots=4, budget=300)
    reqs = [pkg.CausalSequence([7] * 250, pkg.SamplingParams(greedy=True, max_new_tokens=20)) for _ in range(3)]
    done, _ = engine.generate(reqs)
    for r in reqs:
        assert done[r.seq_id][0] == [(8 + j) % 50 for j in range(20)]
    recomputed = [c for p, counts in engine.model_runner.steps if p for c in counts if c > 250]
    assert recomputed and len(engine.scheduler.state_manager.free) == 4


def test_scheduler_waits_for_a_state_slot():
    engine, _ = _engine(pages=16, slots=1)
    reqs = [pkg.CausalSequence([1, 2], pkg.SamplingParams(greedy=True, max_new_tokens=2)) for _ in range(3)]
    done, _ = engine.generate(reqs)
    assert len(done) == 3 and all(len(c) == 1 for _, c in engine.model_runner.steps)


def test_stop_tokens_and_request_types():
    engine, _ = _engine(pages=4, slots=2)
    r = pkg.CausalSequence([3], pkg.SamplingParams(greedy=True, max_new_tokens=30, stop_token_ids=[9]))
    done, _ = engine.generate([r])
    assert done[r.seq_id][0] == [4, 5, 6, 7, 8, 9]
    with pytest.raises(TypeError):
        engine.add_sequence(pkg.Sequence([1], denoising_block_size=4, mask_token_id=0))
    with pytest.raises(ValueError):
        engine.add_sequence(pkg.CausalSequence([1] * 2000))


def test_state_slots():
    sm = pkg.StateManager(2)
    a, b = pkg.CausalSequence([1]), pkg.CausalSequence([2])
    sm.allocate(a)
    sm.allocate(b)
    assert {a.state_slot, b.state_slot} == {0, 1} and not sm.can_allocate()
    with pytest.raises(AssertionError):
        sm.allocate(a)
    sm.deallocate(a)
    assert a.state_slot == -1 and sm.can_allocate()


# --------------------------------------------------------------------------- the restatement itself
def test_oracle_routing_is_group_limited():
    z = torch.tensor([[5.0, 0, 0, 0, 4.0, 3.9, 0, 0, 4.5, 4.4, 4.3, 0]])
    ids, w = orc.route(z, {"experts": 12, "top": 3, "groups": {"count": 3, "keep": 1}})
    assert sorted(ids[0].tolist())[0] == 0 and all(e < 4 for e in ids[0].tolist())
    ids, _ = orc.route(z, {"experts": 12, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert sorted(ids[0].tolist()) == [0, 8, 9]
    ids, w = orc.route(z, {"experts": 12, "top": 4})
    assert sorted(ids[0].tolist()) == [0, 8, 9, 10] and abs(float(w.sum()) - 1) < 1e-6


def test_oracle_delta_rule_overwrites():
    """beta 1, no decay, unit keys: a second write under the same key replaces the first."""
    k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]], dtype=torch.float64)
    v = torch.tensor([[[2.0]], [[5.0]]], dtype=torch.float64)
    one = torch.ones(2, 1, dtype=torch.float64)
    o = orc.delta_scan(k, k, v, torch.ones_like(k), one)
    assert torch.allclose(o.flatten(), torch.tensor([2.0, 5.0], dtype=torch.float64))


def test_oracle_mlstm_matches_unscaled_sums():
    """Away from overflow the running maximum cancels: o = sum w k.q v / max(|sum w k.q|, 1)."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(6, 1, 3, generator=g, dtype=torch.float64) for _ in range(3))
    i, f = torch.randn(6, 1, generator=g, dtype=torch.float64), -torch.rand(6, 1, generator=g, dtype=torch.float64)
    o = orc.mlstm_scan(q, k, v, i, f)
    for t in range(6):
        w = torch.stack([torch.exp(i[j, 0] + f[j + 1:t + 1, 0].sum()) for j in range(t + 1)])
        s = w * (k[:t + 1, 0] @ q[t, 0])
        # the floor exp(-m) is in the running maximum's units: 1 in unscaled ones
        ref = (s[:, None] * v[:t + 1, 0]).sum(0) / torch.maximum(s.sum().abs(), torch.tensor(1.0, dtype=torch.float64))
        assert torch.allclose(o[t, 0], ref, atol=1e-4)


def test_generate_command_line():
    from importlib import import_module
    gen = import_module("mineru-diffusion_b200.generate")
    a = gen.parse(["--model", "m", "--prompt", "1,2 3", "--prompt", "7", "--greedy", "--stop", "4", "--stop", "5"])
    assert a.prompt == [[1, 2, 3], [7]] and a.greedy and a.stop == [4, 5] and a.dtype == "bfloat16"
    with pytest.raises(SystemExit):
        gen.parse(["--model", "m", "--prompt", ","])
