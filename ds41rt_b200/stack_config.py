"""Configuration of layer-stack models: a list of layers, each with a mixer, an optional feed-forward part and an optional
per-layer token input, around one residual stream.  A model family (models/registry.py) reads its own config.json into this
form; models/stack.py runs it.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union

from .config import RopeConfig


class ConfigError(ValueError):
    pass


def take(d, keys, where: str, optional=()):
    """Values of exactly `keys` (and possibly `optional`) of a JSON object."""
    if not isinstance(d, dict):
        raise ConfigError(f"{where}: expected an object")
    unknown, missing = set(d) - set(keys) - set(optional), set(keys) - set(d)
    if unknown or missing:
        raise ConfigError(f"{where}: unknown keys {sorted(unknown)}, missing keys {sorted(missing)}")
    return [d[k] for k in keys] + [d.get(k) for k in optional]


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention over one cached latent row per token (csrc/kernels/latent_attn.cu)."""
    heads: int
    dim: int                     # unrotated query / key width per head
    rot_dim: int                 # rotated query width per head = width of the shared rotated key part
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rope: Optional[RopeConfig] = None      # None: the rot_dim part is not turned
    kv_from: Optional[int] = None          # layer whose cache rows this layer reads (None: its own)
    kind: str = "latent_attention"

    @property
    def magnitude(self) -> float:
        """Factor on cos and sin that goes with a YaRN-scaled rotation."""
        return 1.0 if self.rope is None or not self.rope.scaled else 0.1 * math.log(self.rope.factor) + 1.0


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Attention whose query heads share key / value heads in groups (csrc/kernels/group_attn.cu)."""
    heads: int
    kv_heads: int
    dim: int                     # query / key width per head
    vdim: int
    scale: float
    taps: int = 0                # causal convolution over time on every channel of q, k and v (0: none)
    rot_dim: int = 0             # leading dimensions of a head that are turned (0: none)
    rope: Optional[RopeConfig] = None
    chunk: int = 0               # a position sees its own chunk of this many positions only (0: everything before it)
    qk_norm: bool = True         # RMS norm over all heads of q and of k at once
    head_gate: bool = True       # one sigmoid gate per head on the output
    kind: str = "grouped_attention"


@dataclass(frozen=True)
class MLSTMSpec:
    """Matrix-memory recurrence with a running maximum (csrc/kernels/mlstm.cu)."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    den_eps: float = 1e-6
    kind: str = "mlstm"


@dataclass(frozen=True)
class DenseMLPSpec:
    ff: int
    activation: str = "polynorm"
    kind: str = "dense"


@dataclass(frozen=True)
class MoESpec:
    """Experts g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit); every token takes the
    `top` experts with the largest router logits, weighted by the softmax over those logits."""
    experts: int
    top: int
    ff: int
    limit: float
    alpha: float = 1.702
    shift: float = 1.0
    kind: str = "moe"


MixerSpec = Union[LatentAttentionSpec, GroupedAttentionSpec, MLSTMSpec]
MLPSpec = Union[DenseMLPSpec, MoESpec]


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[MLPSpec]


@dataclass
class StackConfig:
    name: str
    vocab: int
    hidden: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    norm: str = "layer"            # "layer" (with weight, no bias) or "rms"
    post_norm: bool = True         # a norm after each sublayer, before its result is added
    residual_gate: bool = True     # sublayer results times sigmoid(W h + b)
    depth_average: bool = True     # the stream becomes a weighted sum of all layers' results so far
    token_side: int = 0            # width of every layer's part of the tokens' second embedding (0: none)
    logit_softcap: float = 0.0     # logits become cap tanh(logits / cap) (0: as they are)
    max_context: int = 1 << 20
    family: str = "genesun"

    # what the serving code asks every model's configuration
    window = 0
    dspark = engram = vision = None
    ced_boundary = ced_replay = 0

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def norm_kind(self) -> int:
        return {"layer": 0, "rms": 1}[self.norm]

    def source_of(self, layer: int) -> Optional[int]:
        """Layer whose cache rows `layer` reads (None: it has no cache rows)."""
        m = self.layers[layer].mixer
        if m.kind == "mlstm":
            return None
        src = getattr(m, "kv_from", None)
        return layer if src is None else src

    def cache_layers(self) -> List[int]:
        return [l for l in range(self.n_layers) if self.source_of(l) == l]

    def state_layers(self) -> List[int]:
        """Layers that keep a state per request besides cache rows."""
        return [l for l in range(self.n_layers)
                if self.layers[l].mixer.kind == "mlstm" or getattr(self.layers[l].mixer, "taps", 0) > 1]

    def validate(self) -> None:
        if self.vocab <= 0 or self.hidden <= 0 or not self.layers:
            raise ConfigError("vocab, width and layers must not be empty")
        for l, spec in enumerate(self.layers):
            m = spec.mixer
            if m.kind == "latent_attention" and m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < l else None
                if src is None or src.kind != "latent_attention" or src.kv_from is not None:
                    raise ConfigError(f"layer {l}: kv_from names no earlier layer with cache rows of its own")
                if (src.kv_rank, src.rot_dim) != (m.kv_rank, m.rot_dim):
                    raise ConfigError(f"layer {l}: kv_rank / rot_dim differ from those of layer {m.kv_from}")
            if m.kind == "grouped_attention":
                if min(m.heads, m.kv_heads, m.dim, m.vdim) <= 0 or m.taps < 0 or m.chunk < 0 or m.heads % m.kv_heads:
                    raise ConfigError(f"layer {l}: sizes must be positive and kv_heads must divide heads")
                if m.rot_dim % 2 or not 0 <= m.rot_dim <= m.dim:
                    raise ConfigError(f"layer {l}: the rotated part must be even and within the head")
            if spec.mlp is not None and spec.mlp.kind == "moe" and not 0 < spec.mlp.top <= min(spec.mlp.experts, 32):
                raise ConfigError(f"layer {l}: a token takes 1 to 32 of the layer's experts")
