"""The Genesun family: its config.json and tensor names, read into the layer-stack form (stack_config.py, models/stack.py).

Genesun is a decoder of latent-attention and matrix-memory (mLSTM) layers with a layer norm before and after each sublayer,
a sigmoid gate on each sublayer's result, PolyNorm feed-forward parts, and a learned average over the depth: what a layer
hands on is a weighted sum of the embedding output and all layers' results so far.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..config import RopeConfig
from ..stack_config import ConfigError, DenseMLPSpec, LatentAttentionSpec, LayerSpec, MLSTMSpec, StackConfig, take

ARCHITECTURE = "Genesun"


def matches(doc: dict) -> bool:
    return doc.get("architecture") == ARCHITECTURE


def _rope(rot, rot_dim: int, where: str) -> RopeConfig:
    base, dims, scaling = take(rot, ("base", "dims"), where, ("scaling",))
    if dims != rot_dim or dims % 2:
        raise ConfigError(f"{where}: dims must equal the mixer's rot_dim and be even")
    if scaling is None:
        return RopeConfig(theta=float(base))
    factor, fast, slow, original = take(scaling, ("factor", "fast", "slow", "original"), where + ".scaling")
    return RopeConfig(theta=float(base), factor=float(factor), beta_fast=float(fast), beta_slow=float(slow),
                      original_max_position=original)


def parse(doc: dict, name: str = "genesun") -> StackConfig:
    _, layers, norm, vocab, width = take(doc, ("architecture", "layers", "norm", "vocab", "width"), "config")
    (eps,) = take(norm, ("eps",), "norm")
    specs = []
    for l, d in enumerate(layers):
        kind, mx, mlp = take(d, ("type", "mixer", "mlp"), f"layers[{l}]")
        where = f"layers[{l}].mixer"
        if kind == "latent_attention":
            heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, src = take(
                mx, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"), where, ("kv_from",))
            mixer = LatentAttentionSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, float(scale),
                                        _rope(rot, rot_dim, where + ".rot"), src)
        elif kind == "mlstm":
            heads, dim, vdim, cap = take(mx, ("heads", "dim", "vdim", "gate_cap"), where)
            mixer = MLSTMSpec(heads, dim, vdim, float(cap))
        else:
            raise ConfigError(f"layers[{l}]: unknown type {kind!r}")
        ff = None
        if mlp is not None:
            mlp_kind, width_ff = take(mlp, ("kind", "ff"), f"layers[{l}].mlp")
            if mlp_kind != "dense":
                raise ConfigError(f"layers[{l}].mlp: unknown kind {mlp_kind!r}")
            ff = DenseMLPSpec(width_ff)
        specs.append(LayerSpec(mixer, ff))
    cfg = StackConfig(name, vocab, width, tuple(specs), float(eps))
    cfg.validate()
    return cfg


def layer_shapes(cfg: StackConfig, l: int) -> Dict[str, Tuple[int, ...]]:
    """Tensor name within layer l -> shape."""
    W, spec = cfg.hidden, cfg.layers[l]
    m = spec.mixer
    out = {"norm1": (W,), "norm1b": (W,), "rg1": (W, W), "rg1.b": (W,), "dwa": (l + 2,)}
    if m.kind == "latent_attention":
        hv = m.heads * m.vdim
        out.update({"mix.dq": (m.q_rank, W), "mix.dq.norm": (m.q_rank,),
                    "mix.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank), "mix.uk": (m.heads * m.dim, m.kv_rank),
                    "mix.uv": (hv, m.kv_rank), "mix.sink": (m.heads,), "mix.g": (hv, W), "mix.o": (W, hv)})
        if m.kv_from is None:
            out.update({"mix.dkv": (m.kv_rank + m.rot_dim, W), "mix.dkv.norm": (m.kv_rank,)})
    else:
        hd, hv = m.heads * m.dim, m.heads * m.vdim
        out.update({"mix.q": (hd, W), "mix.k": (hd, W), "mix.v": (hv, W), "mix.g": (hv, W), "mix.o": (W, hv),
                    "mix.norm": (hv,), "mix.i": (m.heads, W), "mix.i.b": (m.heads,), "mix.f": (m.heads, W),
                    "mix.f.b": (m.heads,)})
    if spec.mlp is not None:
        ff = spec.mlp.ff
        out.update({"norm2": (W,), "norm2b": (W,), "rg2": (W, W), "rg2.b": (W,), "mlp.up": (ff, W), "mlp.down": (W, ff),
                    "mlp.act": (4,)})
    return out


def tensor_shapes(cfg: StackConfig) -> Dict[str, Tuple[int, ...]]:
    out = {"embed": (cfg.vocab, cfg.hidden), "final.norm": (cfg.hidden,), "head": (cfg.vocab, cfg.hidden)}
    for l in range(cfg.n_layers):
        out.update({f"l{l}.{n}": s for n, s in layer_shapes(cfg, l).items()})
    return out


def build_weights(cfg: StackConfig, read, device, dtype: str = "bf16"):
    """`read(name)` -> tensor by its full name, one layer at a time."""
    from .stack import StackWeights
    return StackWeights(cfg, lambda l: {n: read(f"l{l}.{n}") for n in layer_shapes(cfg, l)},
                        {n: read(n) for n in ("embed", "final.norm", "head")}, device, dtype)


def random_tensor(cfg: StackConfig, name: str, shape, gen: torch.Generator, device) -> torch.Tensor:
    """A random-init tensor whose layers neither vanish nor blow up (bf16)."""
    rnd = lambda s: torch.randn(shape, generator=gen, device=device) * s
    if name.endswith("norm") or name.endswith(("norm1", "norm2", "norm1b", "norm2b")):
        t = 1.0 + rnd(0.1)
    elif name.endswith("dwa"):
        t = rnd(0.1)
        t[-1] += 1.0
    elif name.endswith("mlp.act"):
        t = rnd(0.1) + torch.tensor([0.6, 0.3, 0.1, 0.0], device=device)
    elif name.endswith("mix.f.b"):
        t = 3.0 + rnd(1.0)
    elif name.endswith((".b", "sink")):
        t = rnd(0.5)
    elif name == "embed":
        t = rnd(1.0)
    else:
        t = rnd(shape[-1] ** -0.5)
    return t.to(torch.bfloat16)


def random_weights(cfg: StackConfig, device, seed: int = 0, dtype: str = "bf16"):
    gen = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build_weights(cfg, lambda n: random_tensor(cfg, n, shapes[n], gen, device), device, dtype)


def _preset(name: str, vocab: int, width: int, pattern: str, attn: LatentAttentionSpec, rec: MLSTMSpec,
            ff: int) -> StackConfig:
    """`pattern`: one letter per layer - m = mLSTM, a = latent attention, s = latent attention on the last a's rows."""
    layers, last = [], None
    for l, c in enumerate(pattern):
        if c == "m":
            layers.append(LayerSpec(rec, None))
            continue
        import dataclasses
        layers.append(LayerSpec(dataclasses.replace(attn, kv_from=last if c == "s" else None), DenseMLPSpec(ff)))
        last = l if c == "a" else last
    cfg = StackConfig(name, vocab, width, tuple(layers), 1e-6)
    cfg.validate()
    return cfg


def preset(name: str, n_layers: Optional[int] = None) -> StackConfig:
    """Random-init configurations: "genesun-tiny" for tests, "genesun-1b" / "genesun-7b" with layers of real size."""
    rope = lambda: RopeConfig(theta=100000.0, factor=4.0, original_max_position=8192)
    if name == "genesun-tiny":
        return _preset(name, 512, 256, ("amsm" * 8)[:n_layers or 4],
                       LatentAttentionSpec(4, 32, 32, 48, 96, 64, 0.125, RopeConfig(10000.0)), MLSTMSpec(2, 64, 96, 12.0), 384)
    if name == "genesun-1b":
        return _preset(name, 65536, 2048, ("mams" * 16)[:n_layers or 16],
                       LatentAttentionSpec(16, 128, 64, 128, 768, 512, 192 ** -0.5, rope()), MLSTMSpec(4, 256, 512, 12.0), 5632)
    if name == "genesun-7b":
        return _preset(name, 129280, 4096, ("mams" * 16)[:n_layers or 32],
                       LatentAttentionSpec(32, 128, 64, 128, 1536, 512, 192 ** -0.5, rope()), MLSTMSpec(8, 256, 512, 12.0), 11008)
    raise KeyError(name)


PRESETS = ("genesun-tiny", "genesun-1b", "genesun-7b")
