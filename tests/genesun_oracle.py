"""Plain, slow statement of the Genesun design on the CPU, one function per mechanism, full sequences only.

Nothing here is shared with the product: no cache, no chunks, no batching.  Every function works in the dtype of its
inputs (float64 in the tests).  `GenesunOracle` takes a parsed configuration dict and a name -> tensor dict.
"""
from __future__ import annotations

import math

import torch


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def polynorm(z, coef, eps):
    a, b, c, e = coef
    return a * rms_unit(z, eps) + b * rms_unit(z ** 2, eps) + c * rms_unit(z ** 3, eps) + e


def yarn_frequencies(rot):
    """-> (frequency per pair, factor on cos and sin)."""
    n, base = rot["dims"], float(rot["base"])
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0

    def turn_dim(t):
        return n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turn_dim(sc["fast"])), 0)
    hi = min(math.ceil(turn_dim(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x, pos, rot):
    """x [T, ..., dims], adjacent pairs turned by pos * frequency."""
    freq, m = yarn_frequencies(rot)
    ang = pos.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)
    c, s = torch.cos(ang) * m, torch.sin(ang) * m
    while c.dim() < x.dim():
        c, s = c.unsqueeze(1), s.unsqueeze(1)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def sink_softmax_attention(q, k, v, scale, sink):
    """q, k [T, H, D], v [T, H, V], causal; `sink` [H] adds exp(sink) to every row's denominator."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
    top = torch.maximum(s.amax(-1), sink[:, None])
    e = torch.exp(s - top[..., None])
    w = e / (e.sum(-1) + torch.exp(sink[:, None] - top))[..., None]
    return torch.einsum("hij,jhv->ihv", w, v)


def latent_attention(h, pos, w, p, mx, eps, shared):
    """`shared`: (latent, rotated key) of the layer named by kv_from, or None.  -> (output, (latent, rotated key))."""
    H, D, R, V = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    T = h.shape[0]
    cq = rms_unit(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + R)
    if shared is None:
        kv = h @ w[p + "dkv"].T
        lat = rms_unit(kv[:, :mx["kv_rank"]], eps) * w[p + "dkv.norm"]
        kr = rotate_pairs(kv[:, mx["kv_rank"]:], pos, mx["rot"])
        shared = (lat, kr)
    lat, kr = shared
    qr = rotate_pairs(q[..., D:], pos, mx["rot"])
    k = torch.cat([(lat @ w[p + "uk"].T).view(T, H, D), kr[:, None, :].expand(T, H, R)], -1)
    v = (lat @ w[p + "uv"].T).view(T, H, V)
    o = sink_softmax_attention(torch.cat([q[..., :D], qr], -1), k, v, mx["scale"], w[p + "sink"])
    o = o.reshape(T, H * V) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, shared


def mlstm_scan(q, k, v, i, f):
    """Token by token: q (scaled), k [T, H, D], v [T, H, V], log gates i, f [T, H] -> [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(h, w, p, mx, eps):
    H, D, V, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = rms_unit(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * V) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_polynorm_mlp(h, w, p, eps):
    return polynorm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


def gated_normed(y, h, gate_w, gate_b, norm_w, eps):
    """Sublayer result y of input h: sigmoid gate from h, then the norm that follows the sublayer."""
    return layer_norm(y * torch.sigmoid(h @ gate_w.T + gate_b), norm_w, eps)


class GenesunOracle:
    def __init__(self, doc, weights, dtype=torch.float64):
        self.doc, self.w = doc, {k: v.to(dtype) for k, v in weights.items()}
        self.eps = doc["norm"]["eps"]

    def forward(self, tokens):
        """-> (logits [T, vocab], list of the residual stream after every layer)."""
        w, eps = self.w, self.eps
        toks = torch.as_tensor(tokens, dtype=torch.long)
        pos = torch.arange(len(toks))
        x = w["embed"][toks]
        kept, latents, after = [x], {}, []
        for l, spec in enumerate(self.doc["layers"]):
            p, mx = f"l{l}.", spec["mixer"]
            h = layer_norm(x, w[p + "norm1"], eps)
            if spec["type"] == "mlstm":
                y = mlstm(h, w, p + "mix.", mx, eps)
            else:
                src = mx.get("kv_from")
                y, latents[l] = latent_attention(h, pos, w, p + "mix.", mx, eps,
                                                 latents[src] if src is not None else None)
            x = x + gated_normed(y, h, w[p + "rg1"], w[p + "rg1.b"], w[p + "norm1b"], eps)
            if spec["mlp"] is not None:
                h = layer_norm(x, w[p + "norm2"], eps)
                y = dense_polynorm_mlp(h, w, p + "mlp.", eps)
                x = x + gated_normed(y, h, w[p + "rg2"], w[p + "rg2.b"], w[p + "norm2b"], eps)
            kept.append(x)
            x = sum(c * t for c, t in zip(w[p + "dwa"], kept))
            after.append(x)
        return layer_norm(x, w["final.norm"], eps) @ w["head"].T, after
