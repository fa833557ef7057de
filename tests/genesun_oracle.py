"""Plain, slow statement of the Genesun design on the CPU, one function per mechanism, full sequences only.

Nothing here is shared with the product: no cache, no chunks, no batching.  Every function works in the dtype of its
inputs (float64 in the tests).  `GenesunOracle` takes a parsed configuration dict and a name -> tensor dict.
"""
from __future__ import annotations

import math

import torch


_noise = None      # a torch.Generator while `rounding_spread` measures how far bf16 rounding carries


def _shake(x):
    """What storing x in bf16 may do to it: a random relative change of up to one part in 2^8."""
    return x if _noise is None else x * (1 + (torch.rand(x.shape, generator=_noise, dtype=x.dtype) - 0.5) * 2 ** -7)


def linear(x, w):
    return _shake(_shake(x) @ w.T)


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
    cq = rms_unit(linear(h, w[p + "dq"]), eps) * w[p + "dq.norm"]
    q = linear(cq, w[p + "uq"]).view(T, H, D + R)
    if shared is None:
        kv = linear(h, w[p + "dkv"])
        lat = rms_unit(kv[:, :mx["kv_rank"]], eps) * w[p + "dkv.norm"]
        kr = rotate_pairs(kv[:, mx["kv_rank"]:], pos, mx["rot"])
        shared = (lat, kr)
    lat, kr = shared
    qr = rotate_pairs(q[..., D:], pos, mx["rot"])
    k = torch.cat([linear(lat, w[p + "uk"]).view(T, H, D), kr[:, None, :].expand(T, H, R)], -1)
    v = linear(lat, w[p + "uv"]).view(T, H, V)
    o = sink_softmax_attention(torch.cat([q[..., :D], qr], -1), k, v, mx["scale"], w[p + "sink"])
    o = o.reshape(T, H * V) * torch.sigmoid(linear(h, w[p + "g"]))
    return linear(o, w[p + "o"]), shared


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
    q = linear(h, w[p + "q"]).view(T, H, D) * D ** -0.5
    k = linear(h, w[p + "k"]).view(T, H, D)
    v = linear(h, w[p + "v"]).view(T, H, V)
    i = cap * torch.tanh((linear(h, w[p + "i"]) + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((linear(h, w[p + "f"]) + w[p + "f.b"]) / cap))
    o = rms_unit(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * V) * w[p + "norm"]
    return linear(o * torch.sigmoid(linear(h, w[p + "g"])), w[p + "o"])


def dense_polynorm_mlp(h, w, p, eps):
    return linear(polynorm(linear(h, w[p + "up"]), w[p + "act"], eps), w[p + "down"])


def gated_normed(y, h, gate_w, gate_b, norm_w, eps):
    """Sublayer result y of input h: sigmoid gate from h, then the norm that follows the sublayer."""
    return layer_norm(y * torch.sigmoid(linear(h, gate_w) + gate_b), norm_w, eps)


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
        return linear(layer_norm(x, w["final.norm"], eps), w["head"]), after


def position_error(got, want):
    """Root mean square difference per position, relative to the spread of all values."""
    return (got.double() - want.double()).pow(2).mean(-1).sqrt() / want.double().std()


def rounding_spread(oracle, tokens, trials=4):
    """How far bf16-sized rounding of every stored activation moves each position, -> (logits, [per layer])."""
    global _noise
    want, layers = oracle.forward(tokens)
    worst = [torch.zeros(len(tokens), dtype=torch.float64) for _ in range(1 + len(layers))]
    try:
        for t in range(trials):
            _noise = torch.Generator().manual_seed(t)
            got, after = oracle.forward(tokens)
            for i, (a, b) in enumerate(zip([got, *after], [want, *layers])):
                worst[i] = torch.maximum(worst[i], position_error(a, b))
    finally:
        _noise = None
    return worst[0], worst[1:]


# ---------------------------------------------------------------------------------------------------- test models
def attention_mixer(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, base=10000.0, scaling=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank,
             scale=(dim + rot_dim) ** -0.5 if scale is None else scale, rot=dict(base=base, dims=rot_dim))
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def make_doc(width, vocab, layers, eps=1e-6):
    """`layers`: (type, mixer, ff or None)."""
    return {"architecture": "Genesun", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
                       for t, m, ff in layers]}


def make_weights(doc, seed=0):
    """Random weights whose every mechanism shows in the logits, rounded to bf16 (returned as fp32)."""
    g = torch.Generator().manual_seed(seed)
    W, V = doc["width"], doc["vocab"]
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    lin = lambda o, i: n(o, i, std=i ** -0.5)
    one = lambda k: 1.0 + n(k, std=0.2)
    w = {"embed": n(V, W), "final.norm": one(W), "head": lin(V, W)}
    for l, d in enumerate(doc["layers"]):
        p, m = f"l{l}.", d["mixer"]
        w.update({p + "norm1": one(W), p + "norm1b": one(W), p + "rg1": lin(W, W), p + "rg1.b": n(W, std=0.5),
                  p + "dwa": n(l + 2, std=0.3)})
        w[p + "dwa"][-1] += 0.7
        if d["type"] == "mlstm":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            w.update({p + "mix.q": 2 * lin(hd, W), p + "mix.k": lin(hd, W), p + "mix.v": lin(hv, W), p + "mix.g": lin(hv, W),
                      p + "mix.o": lin(W, hv), p + "mix.norm": one(hv), p + "mix.i": 2 * lin(m["heads"], W),
                      p + "mix.i.b": n(m["heads"]), p + "mix.f": lin(m["heads"], W), p + "mix.f.b": 3 + 2 * n(m["heads"])})
        else:
            hv = m["heads"] * m["vdim"]
            w.update({p + "mix.dq": lin(m["q_rank"], W), p + "mix.dq.norm": 2 * one(m["q_rank"]),
                      p + "mix.uq": 2 * lin(m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                      p + "mix.uk": lin(m["heads"] * m["dim"], m["kv_rank"]), p + "mix.uv": lin(hv, m["kv_rank"]),
                      p + "mix.sink": n(m["heads"]) + 1.0, p + "mix.g": lin(hv, W), p + "mix.o": lin(W, hv)})
            if "kv_from" not in m:
                w.update({p + "mix.dkv": lin(m["kv_rank"] + m["rot_dim"], W), p + "mix.dkv.norm": one(m["kv_rank"])})
        if d["mlp"] is not None:
            ff = d["mlp"]["ff"]
            w.update({p + "norm2": one(W), p + "norm2b": one(W), p + "rg2": lin(W, W), p + "rg2.b": n(W, std=0.5),
                      p + "mlp.up": lin(ff, W), p + "mlp.down": lin(W, ff),
                      p + "mlp.act": torch.tensor([0.6, 0.4, 0.3, 0.1]) + n(4, std=0.1)})
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


YARN = dict(factor=5.0, original=96, fast=8.0, slow=1.0)

MODELS = {
    # widths that are no multiple of the tile sizes, shared cache rows over several layers, feed-forward after a recurrence
    "odd": make_doc(90, 131, [
        ("latent_attention", attention_mixer(3, 20, 6, 24, 56, 40, scaling=YARN), 100),
        ("mlstm", dict(heads=3, dim=24, vdim=40, gate_cap=7.0), 60),
        ("latent_attention", attention_mixer(5, 12, 6, 36, 40, 40, scale=0.3, base=500.0, kv_from=0), None),
        ("latent_attention", attention_mixer(2, 20, 6, 24, 24, 40, scaling=YARN, kv_from=0), 36)]),
    # head counts and ranks of one tile or less, no scaling, recurrences first and last
    "plain": make_doc(64, 96, [
        ("mlstm", dict(heads=1, dim=16, vdim=16, gate_cap=5.0), None),
        ("latent_attention", attention_mixer(1, 32, 2, 16, 16, 16, scale=0.5), None),
        ("mlstm", dict(heads=2, dim=64, vdim=32, gate_cap=20.0), None)]),
    # sizes that fill whole tensor-core tiles, more heads than one tile holds
    "tiles": make_doc(256, 320, [
        ("latent_attention", attention_mixer(20, 64, 64, 128, 64, 192, base=2000.0, scaling=dict(YARN, original=512)), 512),
        ("mlstm", dict(heads=2, dim=128, vdim=192, gate_cap=11.0), None),
        ("latent_attention", attention_mixer(18, 80, 64, 48, 96, 192, base=2000.0, scaling=dict(YARN, original=512),
                                             kv_from=0), 256)]),
}
