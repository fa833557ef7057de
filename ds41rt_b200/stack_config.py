"""Configuration of layer-stack models: a list of layers, each with a mixer and an optional feed-forward part, around one
residual stream.  A model family (models/registry.py) reads its own config.json into this form; models/stack.py runs it.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union

from .config import RopeConfig


class ConfigError(ValueError):
    pass


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


MixerSpec = Union[LatentAttentionSpec, MLSTMSpec]


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[DenseMLPSpec]


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
    max_context: int = 1 << 20

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
        if m.kind != "latent_attention":
            return None
        return layer if m.kv_from is None else m.kv_from

    def cache_layers(self) -> List[int]:
        return [l for l in range(self.n_layers) if self.source_of(l) == l]

    def state_layers(self) -> List[int]:
        return [l for l in range(self.n_layers) if self.layers[l].mixer.kind == "mlstm"]

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
