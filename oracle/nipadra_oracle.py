"""Plain restatement of the Nipadra decoder design on the CPU.

One function per mechanism, token by token where the mechanism is a recurrence, no caching, no batching and no
code shared with the product path.  It exists to be compared with: tests run it in fp32 or fp64 on small
configurations.  ``weights`` maps checkpoint tensor names to tensors; ``cfg`` is the parsed config.json.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def post_norm(x, y, w, alpha, eps):
    """Norm of the scaled residual plus the sublayer's output; the weight is stored around zero."""
    return rms(alpha * x + y, eps) * (1 + w)


def linear_scan(q, k, v, decay, step):
    """S_t = decay_t S_(t-1) + step_t k_t v_t^T, o_t = S_t^T q_t.  q/k [T, H, D], v [T, H, Dv], decay/step [T, H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + (step[t][:, None] * k[t])[:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def lightning(h, get, mixer, eps):
    T, H, D, DV = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    q, k = silu(h @ get("q").T).view(T, H, D), silu(h @ get("k").T).view(T, H, D)
    v = silu(h @ get("v").T).view(T, H, DV)
    decay = torch.tensor(mixer["decay"], dtype=h.dtype).expand(T, H)
    o = linear_scan(q, k, v, decay, torch.ones_like(decay)).reshape(T, H * DV)
    return (rms(o, eps) * get("norm") * sigmoid(h @ get("g").T)) @ get("o").T


def rotate(x, dims, base, positions):
    """Interleaved rotation of the first ``dims`` channels; x [T, H, D]."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, w = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - w * s, w * c + u * s
    return y


def window_sink_attention(q, k, v, scale, window):
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; key j is seen while 0 <= i - j < window, and the softmax's denominator
    has one extra 1."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            lo = max(0, i - window + 1)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            m = max(float(s.max()), 0.0)
            e = torch.exp(s - m)
            out[i, h] = (e @ v[lo:i + 1, g]) / (math.exp(-m) + e.sum())
    return out


def window_attention(h, get, mixer, eps):
    T, H, G, D = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"]
    q, raw = (h @ get("q").T).view(T, H, D), (h @ get("k").T).view(T, G, D)
    pos = torch.arange(T)
    rot = mixer["rot"]
    q = rotate(rms(q, eps) * get("q.norm"), rot["dims"], rot["base"], pos)
    k = rotate(rms(raw, eps) * get("k.norm"), rot["dims"], rot["base"], pos)
    o = window_sink_attention(q, k, raw, mixer["scale"], mixer["mask"]["size"])
    o = o * sigmoid(h @ get("g").T)[:, :, None]
    return o.reshape(T, H * mixer["vdim"]) @ get("o").T


def short_conv(x, w, b):
    """Causal depth-wise convolution over time with a bias, then silu; x [T, C], w [C, taps], the last tap is the
    current token's."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = b.expand(T, -1).clone()
    for j in range(taps):
        y += padded[j:j + T] * w[:, j]
    return silu(y)


def gated_group_norm(y, z, w, parts, eps):
    """Gate first, then every one of ``parts`` equal parts by its own root mean square."""
    y = y * silu(z)
    return rms(y.view(y.shape[0], parts, -1), eps).reshape(y.shape) * w


def mamba2(h, get, mixer, eps):
    T, H, P, N, G = h.shape[0], mixer["heads"], mixer["vdim"], mixer["state"], mixer["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ get("in").T, [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(short_conv(xbc, get("conv"), get("conv.b")), [inner, G * N, G * N], dim=-1)
    x = x.view(T, H, P)
    B, C = (a.view(T, G, N).repeat_interleave(H // G, dim=1) for a in (B, C))
    dt = softplus(dt + get("dt_bias"))
    decay = torch.exp(-torch.exp(get("A_log")) * dt)
    y = linear_scan(C, B, x, decay, dt) + get("D")[:, None] * x
    return gated_group_norm(y.reshape(T, inner), z, get("norm"), mixer["norm_groups"], eps) @ get("o").T


def parallel(h, get, mixer, eps):
    left = window_attention(h, lambda n: get("left." + n), mixer["left"], eps)
    right = mamba2(h, lambda n: get("right." + n), mixer["right"], eps)
    return mixer["left_scale"] * left + mixer["right_scale"] * right


def dense_ff(h, get):
    return (torch.relu(h @ get("gate").T) * (h @ get("up").T)) @ get("down").T


def forward(cfg: dict, weights: dict, tokens, dtype=torch.float32, collect=None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its start.  ``collect`` (a list) receives the residual stream
    after every layer."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    mixers = {"lightning": lightning, "parallel": parallel}
    x = W["embed"][torch.as_tensor(tokens)]
    for li, layer in enumerate(cfg["layers"]):
        y = mixers[layer["type"]](x, lambda n, li=li: W[f"l{li}.mix.{n}"], layer["mixer"], eps)
        x = post_norm(x, y, W[f"l{li}.norm1"], alpha, eps)
        if layer["mlp"] is not None:
            x = post_norm(x, dense_ff(x, lambda n, li=li: W[f"l{li}.mlp.{n}"]), W[f"l{li}.norm2"], alpha, eps)
        if collect is not None:
            collect.append(x.clone())
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["embed"].T
