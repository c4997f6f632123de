"""Small configurations of the Nipadra decoder design used by its tests, and checkpoints for them."""
import torch

from hybrid_cases import config, hybrid


def dense(ff):
    return {"kind": "dense", "ff": ff}


def lightning(heads, dim, vdim, decay, mlp):
    return {"type": "lightning", "mixer": dict(heads=heads, dim=dim, vdim=vdim, decay=decay), "mlp": mlp}


def parallel(left, right, scales, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def window(heads, kv_heads, dim, size, rot, base, scale):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask={"size": size}, rot={"dims": rot, "base": base})


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def model(vocab, width, layers, alpha=1.7, eps=1e-5):
    return {"architecture": "Nipadra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha}


# sizes that divide nothing in particular: grouped and single key heads, part and full rotation, a window within a page and
# one across pages, several norm parts, five taps, layers with and without a feed-forward, two parallel layers in a row
ODD = model(333, 160, [
    lightning(3, 40, 24, [0.5, 0.93, 0.9995], None),
    parallel(window(6, 2, 40, 37, 24, 5e3, 0.2), mamba(4, 24, 20, 2, 3, 3), (0.7, 1.3), dense(100)),
    parallel(window(5, 1, 72, 300, 72, 1e5, 0.11), mamba(3, 40, 136, 1, 5, 1), (1.1, 0.6), None),
    lightning(2, 136, 48, [0.99, 0.7], dense(72)),
], alpha=1.9, eps=3e-6)

# multiples of 64 and 128, more than sixteen heads over one key head, groups that do not fall on heads
EVEN = model(512, 256, [
    parallel(window(8, 2, 128, 130, 64, 1e4, 0.09), mamba(8, 64, 128, 2, 4, 4), (0.9, 1.2), dense(256)),
    lightning(4, 64, 64, [0.9, 0.99, 0.999, 0.3], dense(128)),
    parallel(window(20, 1, 64, 257, 64, 1e6, 0.125), mamba(2, 96, 64, 1, 2, 6), (1.0, 0.5), None),
])

# sizes that are no multiples of four, heads past the tensor-core forms, a window of one token, one tap, no rotation
RAGGED = model(201, 98, [
    parallel(window(2, 1, 30, 19, 6, 100.0, 0.3), mamba(3, 22, 18, 3, 4, 2), (1.5, 0.8), dense(33)),
    parallel(window(2, 2, 200, 1, 200, 1e4, 0.07), mamba(1, 16, 300, 1, 1, 1), (0.5, 1.0), None),
    lightning(1, 10, 14, [0.97], dense(50)),
    parallel(window(3, 3, 262, 64, 0, 1e4, 0.06), mamba(2, 300, 34, 1, 2, 4), (1.0, 1.0), dense(64)),
], alpha=1.0)

MODELS = {"odd": ODD, "even": EVEN, "ragged": RAGGED}


def tensors(raw, seed=0):
    """bf16 checkpoint on the CPU.  Query norms are widened so that attention looks at few keys: one key too many or too
    few at a window's edge then shows."""
    t = hybrid.random_tensors(config(raw), seed, "cpu")
    for name in t:
        if name.endswith("left.q.norm"):
            t[name] = (t[name].float() * 3).to(torch.bfloat16)
    return t
