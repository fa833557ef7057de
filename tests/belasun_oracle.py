"""Plain, slow statement of the Belasun design on the CPU, one function per mechanism, full sequences only.

Nothing here is shared with the product: no cache, no portions, no batching.  Every function works in the dtype of its
inputs (float64 in the tests).  `BelasunOracle` takes a parsed configuration dict and a name -> tensor dict.
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


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(u, w):
    """u [T, C], w [C, taps]: every channel's last `taps` values weighted, the newest by the last tap."""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] = out[t] + w[:, j] * u[s]
    return out


def frequencies(rot):
    """Angle per position of every pair; long wavelengths slowed down by `factor`, a linear passage between."""
    n = rot["dims"]
    freq = [float(rot["base"]) ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq
    out = []
    for f in freq:
        wave = 2 * math.pi / f
        if wave < sc["original"] / sc["high"]:
            out.append(f)
        elif wave > sc["original"] / sc["low"]:
            out.append(f / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1 - s) * f / sc["factor"] + s * f)
    return out


def rotate_halves(x, pos, rot):
    """x [T, H, D]: of the first `dims` values of a head, value i turns with value i + dims / 2."""
    n = rot["dims"]
    ang = pos.to(x.dtype)[:, None] * torch.tensor(frequencies(rot), dtype=x.dtype)
    c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def chunk_visible(T, size):
    """[T, T]: query i sees key j of its own chunk, up to itself."""
    i = torch.arange(T)
    seen = i[None, :] <= i[:, None]
    return seen if size is None else seen & (i[None, :] // size == i[:, None] // size)


def masked_attention(q, k, v, scale, visible):
    """q [T, H, D], k [T, G, D], v [T, G, V]; query head h reads key / value head h // (H / G)."""
    n = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(n, 1), v.repeat_interleave(n, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    w = torch.softmax(s.masked_fill(~visible, -math.inf), -1)
    return torch.einsum("hij,jhv->ihv", w, v)


def attention(h, pos, w, p, mx, eps):
    H, G, D, V, T = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], h.shape[0]
    q, k, v = (short_conv(linear(h, w[p + n]), w[p + n + ".conv"]) for n in "qkv")
    q = rms_norm(q, w[p + "q.norm"], eps).view(T, H, D)
    k = rms_norm(k, w[p + "k.norm"], eps).view(T, G, D)
    q, k = (_shake(rotate_halves(x, pos, mx["rot"])) for x in (q, k))
    o = masked_attention(q, k, _shake(v).view(T, G, V), mx["scale"], chunk_visible(T, mx["mask"]["size"] if "mask" in mx else None))
    o = o * torch.sigmoid(linear(h, w[p + "g"]))[..., None]
    return linear(o.reshape(T, H * V), w[p + "o"])


def expert(h, w, p, limit):
    g = linear(h, w[p + "gate"]).clamp(max=limit)
    u = linear(h, w[p + "up"]).clamp(-limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), w[p + "down"])


def route(h, w, p, top):
    """-> (chosen experts [T, top], their weights): softmax over the chosen logits alone."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best = torch.topk(z, top, -1)
    return best.indices, torch.softmax(best.values, -1)


def mixture(h, w, p, ml):
    ids, wt = route(h, w, p, ml["router"]["top"])
    y = torch.zeros_like(h)
    for e in range(ml["router"]["experts"]):
        rows, k = torch.where(ids == e)
        if len(rows):
            y[rows] = y[rows] + wt[rows, k][:, None] * expert(h[rows], w, f"{p}e{e}.", ml["expert"]["limit"])
    return y


def token_side(x, e, w, p, eps):
    """What a layer takes from its own part `e` of the tokens' second embedding."""
    y = linear(gelu_tanh(linear(x, w[p + "side.gate"])) * e, w[p + "side.proj"])
    return rms_norm(y, w[p + "side.norm"], eps)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


class BelasunOracle:
    def __init__(self, doc, weights, dtype=torch.float64):
        self.doc, self.w = doc, {k: v.to(dtype) for k, v in weights.items()}
        self.eps = doc["norm"]["eps"]

    def forward(self, tokens):
        """-> (logits [T, vocab], list of the residual stream after every layer)."""
        w, eps, dim = self.w, self.eps, self.doc["token_side"]["dim"]
        toks = torch.as_tensor(tokens, dtype=torch.long)
        pos = torch.arange(len(toks))
        x = w["embed"][toks]
        after = []
        for l, spec in enumerate(self.doc["layers"]):
            p = f"l{l}."
            x = x + attention(rms_norm(x, w[p + "norm1"], eps), pos, w, p + "mix.", spec["mixer"], eps)
            if spec["mlp"] is not None:
                x = x + mixture(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", spec["mlp"])
            x = x + token_side(x, w["side.embed"][toks, l * dim:(l + 1) * dim], w, p, eps)
            after.append(x)
        return softcap(linear(rms_norm(x, w["final.norm"], eps), w["embed"]), self.doc["logit_softcap"]), after


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
BANDS = dict(factor=3.0, low=1.0, high=5.0, original=80)


def mixer(heads, kv_heads, dim, vdim, chunk, conv=4, rot=None, base=200.0, scaling=None, scale=None):
    r = dict(base=base, dims=dim if rot is None else rot)
    if scaling is not None:
        r["scaling"] = scaling
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale, rot=r, conv=conv)
    if chunk is not None:
        m["mask"] = dict(size=chunk)
    return m


def moe(experts, top, ff, limit):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


def make_doc(width, vocab, layers, side, eps=1e-5, cap=20.0):
    return {"architecture": "Belasun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "token_side": {"dim": side},
            "logit_softcap": cap, "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


def make_weights(doc, seed=0, steady=False):
    """Random weights whose every mechanism shows in the logits, rounded to bf16 (returned as fp32).

    `steady`: which experts a token takes does not hang on rounding - the first columns of the embedding hold a code that
    only the routers read and nothing writes to."""
    g = torch.Generator().manual_seed(seed)
    W, V, side, L = doc["width"], doc["vocab"], doc["token_side"]["dim"], len(doc["layers"])
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    lin = lambda o, i: n(o, i, std=i ** -0.5)
    one = lambda k: 1.0 + n(k, std=0.2)
    code = max([d["mlp"]["router"]["experts"] for d in doc["layers"] if d["mlp"] is not None], default=0) if steady else 0

    def out(rows, cols):                   # a matrix that writes to the stream
        t = lin(rows, cols)
        t[:code] = 0
        return t

    w = {"embed": n(V, W), "side.embed": n(V, L * side), "final.norm": one(W)}
    for v in range(V if code > 1 else 0):
        w["embed"][v, :code] = torch.linspace(-2, 2, code)[torch.randperm(code, generator=g)]
    for l, d in enumerate(doc["layers"]):
        p, m = f"l{l}.", d["mixer"]
        rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
        w[p + "norm1"] = one(W)
        for name, r in rows.items():
            w[p + "mix." + name] = lin(r, W)
            w[p + f"mix.{name}.conv"] = n(r, m["conv"], std=0.6)
            if name != "v":
                w[p + f"mix.{name}.norm"] = 1.6 * one(r)
        w[p + "mix.g"], w[p + "mix.o"] = 2 * lin(m["heads"], W), 2 * out(W, m["heads"] * m["vdim"])
        if d["mlp"] is not None:
            E, ff = d["mlp"]["router"]["experts"], d["mlp"]["expert"]["ff"]
            w[p + "norm2"] = one(W)
            w[p + "mlp.router"], w[p + "mlp.router.b"] = lin(E, W) * 3, n(E, std=0.5)
            if code:
                w[p + "norm2"][:code] = 1.0
                w[p + "mlp.router"], w[p + "mlp.router.b"] = torch.eye(E, W) * 4, torch.zeros(E)
            for e in range(E):
                w.update({p + f"mlp.e{e}.gate": 2 * lin(ff, W), p + f"mlp.e{e}.up": lin(ff, W),
                          p + f"mlp.e{e}.down": 2 * out(W, ff)})
        w.update({p + "side.gate": lin(side, W), p + "side.proj": out(W, side), p + "side.norm": one(W)})
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


MODELS = {
    # widths that are no multiple of the tile sizes, layers of different kinds, a layer without a feed-forward part
    "odd": make_doc(90, 131, [(mixer(6, 2, 20, 24, 37, conv=3, rot=12, scaling=BANDS), moe(5, 2, 44, 1.5)),
                              (mixer(3, 3, 12, 36, 100, conv=5, scale=0.4), None),
                              (mixer(5, 1, 20, 24, 16, conv=2, base=50.0, scaling=dict(BANDS, low=2.0)), moe(7, 3, 20, 0.8))],
                    side=10),
    # one head, one expert, one tap, a chunk of a few positions; a layer that sees everything
    "plain": make_doc(64, 96, [(mixer(1, 1, 16, 16, 8), moe(1, 1, 16, 2.0)), (mixer(2, 2, 16, 32, 1, conv=1), moe(3, 3, 24, 1.0)),
                               (mixer(2, 1, 32, 16, None, rot=2), moe(4, 1, 32, 30.0))], side=3, eps=1e-6, cap=5.0),
    # sizes that fill whole tensor-core tiles, more query heads per key/value head than one tile holds
    "tiles": make_doc(256, 320, [(mixer(8, 2, 64, 128, 128, scaling=BANDS), moe(12, 4, 128, 1.0)),
                                 (mixer(20, 1, 128, 64, 200), moe(40, 2, 64, 7.0)),
                                 (mixer(2, 2, 192, 112, 64, rot=64), moe(12, 3, 256, 2.0))], side=64, cap=30.0),
}
