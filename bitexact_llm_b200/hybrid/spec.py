"""Sizes and constants of a hybrid float model: what a design's reader (`fedatar.read_config`) produces and the layers
take. Nothing here belongs to one design; what a design fixes (activations, the sink, the gates) is a field too."""

from dataclasses import dataclass


@dataclass(frozen=True)
class MinGRUSpec:
    width: int


@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int                # unrotated query / key entries per head
    rot_dim: int            # rotated entries per head (one rotated key part for all heads)
    vdim: int
    q_rank: int
    kv_rank: int
    rot_base: float
    scale: float
    window: int             # keys a position sees, itself included; 0: all before it
    eps: float              # of the two latent norms


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "xielu"


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    shared_ff: int          # 0: no shared expert
    act: str = "relu2"
    shared_act: str = "relu2"


@dataclass(frozen=True)
class LayerSpec:
    mixer: object           # MinGRUSpec or LatentAttentionSpec
    ff: object              # DenseSpec, ExpertsSpec or None


@dataclass(frozen=True)
class ModelSpec:
    vocab: int
    width: int
    eps: float
    layers: tuple
