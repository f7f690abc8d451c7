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
class AttentionSpec:
    """Grouped-query attention; biases, query / key norms and sinks are there when the weights have them."""
    heads: int
    kv_heads: int
    dim: int                # query / key entries per head
    vdim: int
    rot_dims: int           # rotated entries per head (the first ones, halves paired)
    rot_base: float
    scale: float
    window: int             # 0: all before it
    eps: float              # of the query and key norms


@dataclass(frozen=True)
class Mamba2Spec:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int
    eps: float              # of the gated norm


@dataclass(frozen=True)
class GLASpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    eps: float              # of the output norm


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    act: str = "xielu"


@dataclass(frozen=True)
class GatedSpec:
    ff: int
    act: str = "gelu"


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
    mixer: object           # MinGRUSpec, LatentAttentionSpec, AttentionSpec, Mamba2Spec or GLASpec
    ff: object              # DenseSpec, GatedSpec, ExpertsSpec or None


@dataclass(frozen=True)
class ModelSpec:
    vocab: int
    width: int
    eps: float
    layers: tuple
    runs: tuple = None          # the layers in the order they run (a layer may run several times); None: each once
    streams: int = 0            # residual streams (hyper-connections, RMS norms); 0: one residual, layer norms with bias
    logit_scale: float = 1.0
    logit_softcap: float = 0.0  # 0: none
