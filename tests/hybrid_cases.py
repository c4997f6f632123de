"""Small configurations of the hybrid decoder design used by its tests, and checkpoints for them."""
import importlib

import torch

pkg = importlib.import_module("mineru-diffusion_b200")
hybrid = importlib.import_module("mineru-diffusion_b200.hybrid")


def moe(experts, top, ff, groups=None, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, **({"groups": groups} if groups else {})},
            **({"shared": {"ff": shared}} if shared else {})}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def latent(heads, dim, vdim, q_rank, kv_rank, scale, mlp, kv_from=None):
    mixer = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale)
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "channel_delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), "mlp": mlp}


def model(vocab, width, layers, scale=3.0, eps=1e-5):
    return {"architecture": "Zikunex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


# sizes that divide nothing in particular, every branch: grouped and ungrouped routing, with and without a shared expert,
# a layer without feed-forward, shared and own latents, one and several q/k heads per value head
ODD = model(333, 160, [
    delta(4, 2, 40, 24, 3, moe(12, 3, 40, {"count": 3, "keep": 2}, shared=56)),
    mlstm(3, 48, 40, 7.5, None),
    latent(5, 48, 72, 40, 56, 0.11, dense(100)),
    delta(2, 1, 136, 48, 5, moe(6, 2, 24)),
    latent(3, 136, 40, 96, 56, 0.07, moe(9, 4, 33, {"count": 3, "keep": 3}), kv_from=2),
    mlstm(2, 20, 72, 30.0, dense(72)),
], scale=2.5, eps=3e-6)

# multiples of 128, more than one block of heads over a latent, keys and values expanded in prompts
EVEN = model(512, 256, [
    latent(20, 128, 128, 128, 256, 0.09, moe(8, 2, 128, {"count": 2, "keep": 1}, shared=128)),
    delta(4, 4, 128, 128, 4, dense(256)),
    mlstm(2, 128, 256, 15.0, dense(128)),
    latent(4, 128, 96, 128, 256, 0.125, dense(256), kv_from=0),
])

# one mechanism per layer type at other sizes: a wide latent, a single head, one convolution tap
WIDE = model(200, 96, [
    latent(2, 32, 32, 64, 520, 0.2, dense(64)),
    delta(1, 1, 300, 16, 1, dense(64)),
    mlstm(1, 260, 32, 5.0, moe(4, 4, 16, {"count": 4, "keep": 4}, shared=24)),
])


def settled(raw):
    """The same model with every expert chosen by every token.  In bf16 a close call of a router goes either way, and a
    recurrent layer carries the difference on; this leaves rounding alone."""
    layers = []
    for layer in raw["layers"]:
        mlp = layer["mlp"]
        if mlp and mlp["kind"] == "moe":
            n = mlp["router"]["top"]
            mlp = {**mlp, "router": {"experts": n, "top": n}}
        layers.append({**layer, "mlp": mlp})
    return {**raw, "layers": layers}

MODELS = {"odd": ODD, "even": EVEN, "wide": WIDE}
SETTLED = {name: settled(raw) for name, raw in MODELS.items()}


def config(raw):
    return pkg.HybridConfig.from_json(raw)


def tensors(raw, seed=0, rank=24):
    """bf16 checkpoint on the CPU; router weights are widened so that few choices are close."""
    t = hybrid.random_tensors(config(raw), seed, "cpu", rank=rank)
    for name in t:
        if name.endswith("mlp.router"):
            t[name] = (t[name].float() * 4).to(torch.bfloat16)
    return t


def runner(raw, tens, dtype="float32", max_seqs=4, max_len=768, pages=12, eager=True, max_tokens=None, **kw):
    cfg = pkg.Config(max_num_seqs=max_seqs, max_model_len=max_len, max_num_batched_tokens=max_tokens or max_len * 2,
                     num_kvcache_blocks=pages, enforce_eager=eager, decoder_config=config(raw), dtype=dtype, **kw)
    w = hybrid.HybridWeights.build(cfg.decoder_config, tens, "cuda", getattr(torch, dtype))
    return pkg.CausalModelRunner(cfg, weights=w)


def sequence(tokens, pages, slot):
    s = pkg.CausalSequence(list(tokens))
    s.block_table = list(pages)
    s.state_slot = slot
    return s


def run_portions(r, seq, portions):
    """Logits [tokens, vocab] (CPU) of one sequence fed in the given portions."""
    out = []
    for n in portions:
        lg, _ = r.execute([seq], [n], [(0, i) for i in range(n)])
        out.append(lg.cpu())
        seq.num_cached_tokens += n
    return torch.cat(out)


def row_error(got, ref):
    """Root mean square over the vocabulary of the centred difference, per row, relative to the reference's spread."""
    d = got.double() - ref.double()
    d = d - d.mean(-1, keepdim=True)
    spread = (ref.double() - ref.double().mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / spread
