"""Plain restatement of the hybrid decoder design (architecture "Zikunex") on the CPU.

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


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def relu2(z):
    return torch.clamp(z, min=0) ** 2


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal depth-wise convolution over time followed by silu; x [T, C], w [C, taps], the last tap is the
    current token's."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y += padded[j:j + T] * w[:, j]
    return y * sigmoid(y)


def causal_attention(q, k, v, scale):
    """q/k [T, H, D], v [T, H, Dv]: softmax over all keys at or before the query."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    s = s.masked_fill(~mask, -math.inf)
    p = torch.softmax(s, -1)
    return torch.einsum("hij,jhd->ihd", p, v)


def latent_attention(h, get, mixer, eps, shared):
    """Returns (output, latent rows).  ``shared`` is the latent of another layer or None."""
    T, H, D, DV = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    cq = rms_norm(h @ get("dq").T, get("dq.norm"), eps)
    q = (cq @ get("uq").T).view(T, H, D)
    c = shared if shared is not None else rms_norm(h @ get("dkv").T, get("dkv.norm"), eps)
    k = (c @ get("uk").T).view(T, H, D)
    v = (c @ get("uv").T).view(T, H, DV)
    o = causal_attention(q, k, v, mixer["scale"])
    return o.reshape(T, H * DV) @ get("o").T, c


def delta_scan(q, k, v, g, beta):
    """Gated delta rule with one decay per key channel.  q/k/g [T, H, D], v [T, H, Dv], beta [T, H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_delta(h, get, mixer, eps):
    T, H, KH, D, DV = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = short_conv(h @ get("q").T, get("q.conv")).view(T, KH, D)
    k = short_conv(h @ get("k").T, get("k.conv")).view(T, KH, D)
    v = short_conv(h @ get("v").T, get("v.conv")).view(T, H, DV)
    rep = H // KH
    q = (unit(q) * D ** -0.5).repeat_interleave(rep, dim=1)
    k = unit(k).repeat_interleave(rep, dim=1)
    beta = sigmoid(h @ get("b").T)
    a = (h @ get("a1").T) @ get("a2").T + get("dt_bias")
    g = torch.exp(-torch.exp(get("A_log"))[None, :, None] * softplus(a).view(T, H, D))
    o = rms(delta_scan(q, k, v, g, beta), eps) * get("norm")
    o = o * sigmoid((h @ get("g1").T) @ get("g2").T).view(T, H, DV)
    return o.reshape(T, H * DV) @ get("o").T


def mlstm_scan(q, k, v, i, f):
    """Matrix memory with a normaliser and a running maximum.  q/k [T, H, D], v [T, H, Dv], i/f [T, H]
    (log input gate, log forget gate)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = m_new
        num = torch.einsum("hdv,hd->hv", S, q[t])
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(num / den[:, None])
    return torch.stack(out)


def mlstm(h, get, mixer, eps):
    T, H, D, DV, cap = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"], mixer["gate_cap"]
    q = (h @ get("q").T).view(T, H, D) * D ** -0.5
    k = (h @ get("k").T).view(T, H, D)
    v = (h @ get("v").T).view(T, H, DV)
    i = cap * torch.tanh((h @ get("i").T + get("i.b")) / cap)
    fraw = cap * torch.tanh((h @ get("f").T + get("f.b")) / cap)
    f = -softplus(-fraw)
    o = rms(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * DV)
    return (o * get("norm") * sigmoid(h @ get("g").T)) @ get("o").T


def dense_ff(h, up, down):
    return relu2(h @ up.T) @ down.T


def route(z, router):
    """Router logits [T, E] -> (expert ids [T, top], weights [T, top]) with group-limited choice."""
    s = torch.softmax(z, -1)
    T, E = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    gmax = s.view(T, groups["count"], size).max(-1).values
    kept = gmax.topk(groups["keep"], -1).indices
    allowed = torch.zeros(T, groups["count"], dtype=torch.bool).scatter_(1, kept, True)
    masked = s.masked_fill(~allowed.repeat_interleave(size, dim=1), -1.0)
    ids = masked.topk(router["top"], -1).indices
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def moe_ff(h, get, mlp):
    ids, w = route(h @ get("router").T, mlp["router"])
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        for slot in range(ids.shape[1]):
            rows = (ids[:, slot] == e).nonzero().flatten()
            if rows.numel():
                y[rows] += w[rows, slot, None] * dense_ff(h[rows], get(f"e{e}.up"), get(f"e{e}.down"))
    if mlp.get("shared"):
        y += dense_ff(h, get("shared.up"), get("shared.down"))
    return y


def forward(cfg: dict, weights: dict, tokens, dtype=torch.float32, collect=None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its start.  ``collect`` (a list) receives the residual stream
    after every layer."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    latents = {}
    for li, layer in enumerate(cfg["layers"]):
        mixer, mlp = layer["mixer"], layer["mlp"]

        def get(name, kind="mix", li=li):
            return W[f"l{li}.{kind}.{name}"]

        h = rms_norm(x, W[f"l{li}.norm1"], eps)
        if layer["type"] == "latent_attention":
            src = mixer.get("kv_from")
            y, latents[li] = latent_attention(h, get, mixer, eps, None if src is None else latents[src])
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, get, mixer, eps)
        elif layer["type"] == "mlstm":
            y = mlstm(h, get, mixer, eps)
        else:
            raise ValueError(layer["type"])
        x = x + y
        if mlp is not None:
            h = rms_norm(x, W[f"l{li}.norm2"], eps)

            def getm(name, li=li):
                return W[f"l{li}.mlp.{name}"]

            x = x + (dense_ff(h, getm("up"), getm("down")) if mlp["kind"] == "dense" else moe_ff(h, getm, mlp))
        if collect is not None:
            collect.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T
