"""The Belasun family: its config.json and tensor names, read into the layer-stack form (stack_config.py, models/stack.py).

Belasun is a decoder of grouped-query attention layers whose positions see their own chunk of the sequence.  Queries, keys
and values pass a short causal convolution; queries and keys are normed over all heads at once and rotated; every head's
output has one sigmoid gate.  Feed-forward parts are mixtures of experts with a clamped gated activation.  After the
feed-forward part every layer adds what it reads from its own slice of a second token embedding.  The output head is the
embedding table, with soft-capped logits.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..config import RopeConfig
from ..stack_config import ConfigError, GroupedAttentionSpec, LayerSpec, MoESpec, StackConfig, take

ARCHITECTURE = "Belasun"


def matches(doc: dict) -> bool:
    return doc.get("architecture") == ARCHITECTURE


def _rope(rot, where: str) -> Tuple[int, RopeConfig]:
    base, dims, scaling = take(rot, ("base", "dims"), where, ("scaling",))
    if scaling is None:
        return dims, RopeConfig(theta=float(base))
    factor, low, high, original = take(scaling, ("factor", "low", "high", "original"), where + ".scaling")
    return dims, RopeConfig(theta=float(base), factor=float(factor), original_max_position=original,
                            bands=(float(low), float(high)))


def _mixer(mx, where: str) -> GroupedAttentionSpec:
    heads, kv_heads, dim, vdim, scale, taps, rot, mask = take(mx, ("heads", "kv_heads", "dim", "vdim", "scale"), where,
                                                              ("conv", "rot", "mask"))
    rot_dim, rope = (0, None) if rot is None else _rope(rot, where + ".rot")
    chunk = 0
    if mask is not None:
        (chunk,) = take(mask, ("size",), where + ".mask")
        if chunk <= 0:
            raise ConfigError(f"{where}.mask: size must be positive")
    return GroupedAttentionSpec(heads, kv_heads, dim, vdim, float(scale), taps or 0, rot_dim, rope, chunk)


def _mlp(mlp, where: str) -> Optional[MoESpec]:
    if mlp is None:
        return None
    kind, expert, router = take(mlp, ("kind", "expert", "router"), where)
    if kind != "moe":
        raise ConfigError(f"{where}: unknown kind {kind!r}")
    ff, limit = take(expert, ("ff", "limit"), where + ".expert")
    experts, top = take(router, ("experts", "top"), where + ".router")
    return MoESpec(experts, top, ff, float(limit))


def parse(doc: dict, name: str = "belasun") -> StackConfig:
    _, layers, norm, vocab, width, side, cap = take(doc, ("architecture", "layers", "norm", "vocab", "width"), "config",
                                                    ("token_side", "logit_softcap"))
    (eps,) = take(norm, ("eps",), "norm")
    specs = []
    for l, d in enumerate(layers):
        kind, mx, mlp = take(d, ("type", "mixer"), f"layers[{l}]", ("mlp",))
        if kind != "attention":
            raise ConfigError(f"layers[{l}]: unknown type {kind!r}")
        specs.append(LayerSpec(_mixer(mx, f"layers[{l}].mixer"), _mlp(mlp, f"layers[{l}].mlp")))
    dim = 0 if side is None else take(side, ("dim",), "token_side")[0]
    return _config(name, vocab, width, specs, float(eps), dim, 0.0 if cap is None else float(cap))


def _config(name, vocab, width, specs, eps, side, cap) -> StackConfig:
    cfg = StackConfig(name, vocab, width, tuple(specs), eps, norm="rms", post_norm=False, residual_gate=False,
                      depth_average=False, token_side=side, logit_softcap=cap, family="belasun")
    cfg.validate()
    return cfg


def layer_shapes(cfg: StackConfig, l: int) -> Dict[str, Tuple[int, ...]]:
    """Tensor name within layer l -> shape."""
    W, m, ml = cfg.hidden, cfg.layers[l].mixer, cfg.layers[l].mlp
    rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
    out = {"norm1": (W,), "mix.q.norm": (rows["q"],), "mix.k.norm": (rows["k"],), "mix.g": (m.heads, W),
           "mix.o": (W, m.heads * m.vdim)}
    for n, r in rows.items():
        out[f"mix.{n}"] = (r, W)
        if m.taps:
            out[f"mix.{n}.conv"] = (r, m.taps)
    if ml is not None:
        out.update({"norm2": (W,), "mlp.router": (ml.experts, W), "mlp.router.b": (ml.experts,)})
        for e in range(ml.experts):
            out.update({f"mlp.e{e}.gate": (ml.ff, W), f"mlp.e{e}.up": (ml.ff, W), f"mlp.e{e}.down": (W, ml.ff)})
    if cfg.token_side:
        out.update({"side.gate": (cfg.token_side, W), "side.proj": (W, cfg.token_side), "side.norm": (W,)})
    return out


def tensor_shapes(cfg: StackConfig) -> Dict[str, Tuple[int, ...]]:
    out = {"embed": (cfg.vocab, cfg.hidden), "final.norm": (cfg.hidden,)}
    if cfg.token_side:
        out["side.embed"] = (cfg.vocab, cfg.n_layers * cfg.token_side)
    for l in range(cfg.n_layers):
        out.update({f"l{l}.{n}": s for n, s in layer_shapes(cfg, l).items()})
    return out


def build_weights(cfg: StackConfig, read, device, dtype: str = "bf16"):
    """`read(name)` -> tensor by its full name, one layer at a time."""
    from .stack import StackWeights
    top = {n: read(n) for n in ("embed", "final.norm") + (("side.embed",) if cfg.token_side else ())}
    return StackWeights(cfg, lambda l: {n: read(f"l{l}.{n}") for n in layer_shapes(cfg, l)}, dict(top, head=top["embed"]),
                        device, dtype)


def random_tensor(cfg: StackConfig, name: str, shape, gen: torch.Generator, device) -> torch.Tensor:
    """A random-init tensor whose layers neither vanish nor blow up (bf16)."""
    rnd = lambda s: torch.randn(shape, generator=gen, device=device) * s
    if name.endswith("norm") or name.endswith(("norm1", "norm2")):
        t = 1.0 + rnd(0.1)
    elif name.endswith(".conv"):
        t = rnd(0.3)
        t[:, -1] += 1.0
    elif name.endswith(".b"):
        t = rnd(0.1)
    elif name.endswith("embed"):
        t = rnd(1.0)
    else:
        t = rnd(shape[-1] ** -0.5)
    return t.to(torch.bfloat16)


def random_weights(cfg: StackConfig, device, seed: int = 0, dtype: str = "bf16"):
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build_weights(cfg, lambda n: random_tensor(cfg, n, shapes[n], gen, device), device, dtype)


def preset(name: str, n_layers: Optional[int] = None) -> StackConfig:
    """Random-init configurations: "belasun-tiny" for tests, "belasun-1b" / "belasun-7b" with layers of real size."""
    rope = RopeConfig(theta=500000.0, factor=8.0, original_max_position=8192, bands=(1.0, 4.0))
    if name == "belasun-tiny":
        mixer, mlp = GroupedAttentionSpec(6, 2, 32, 48, 32 ** -0.5, 3, 16, rope, 96), MoESpec(8, 2, 128, 7.0)
        return _config(name, 512, 256, [LayerSpec(mixer, mlp)] * (n_layers or 4), 1e-6, 32, 30.0)
    if name == "belasun-1b":
        mixer, mlp = GroupedAttentionSpec(16, 4, 128, 128, 128 ** -0.5, 4, 128, rope, 8192), MoESpec(32, 4, 1024, 7.0)
        return _config(name, 65536, 2048, [LayerSpec(mixer, mlp)] * (n_layers or 16), 1e-6, 128, 30.0)
    if name == "belasun-7b":
        mixer, mlp = GroupedAttentionSpec(32, 8, 128, 128, 128 ** -0.5, 4, 128, rope, 8192), MoESpec(16, 4, 1792, 7.0)
        return _config(name, 129280, 4096, [LayerSpec(mixer, mlp)] * (n_layers or 32), 1e-6, 256, 30.0)
    raise KeyError(name)


PRESETS = ("belasun-tiny", "belasun-1b", "belasun-7b")
