"""Typed configuration of the Pamarax decoder.

config.json of this design is nested: ``vocab``, ``width``, ``norm`` (eps), ``embedding`` (scale) and ``layers``, a list
in which every entry names its mixer (``type``: mlstm, attention or parallel), the mixer's sizes and constants
(``mixer``; a parallel one has those of its two branches under ``left`` and ``right`` and a factor for each) and its
feed-forward (``mlp``, or null for none; ``kind`` dense).  The order of the layers and all sizes are data: two models of
the design may differ in all of it.  Every size and constant is read here; the parts get them as parameters.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .lumevik import _sub
from .reader import ConfigError, KeyReader

ARCHITECTURE = "Pamarax"
# limits of the kernels the design's parts launch (csrc/bias_attention.cu BA_MAX_DIM, csrc/ssm.cu SSM_MAX_STATE and
# SSM_MAX_TAPS), checked when the configuration is read
MAX_HEAD_SIZE = 256
MAX_TAPS = 8
MAX_MEMORY_VALUES = 8192


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class SharedValueAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot_dims: int                  # rotated elements of a head (the first ones); 0: none
    rot_base: float


@dataclass(frozen=True)
class SinkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temperature: Optional[Tuple[float, int]]      # (coef, every); None: none


@dataclass(frozen=True)
class HeadDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class ParallelConfig:
    left: SinkAttentionConfig
    right: HeadDeltaConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int


@dataclass(frozen=True)
class PamaraxLayer:
    type: str
    mixer: Any                     # one of the three mixer configurations
    mlp: Optional[DenseMlpConfig]


LAYER_TYPES = ("mlstm", "attention", "parallel")


@dataclass(frozen=True)
class PamaraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[PamaraxLayer, ...]
    raw: Dict[str, Any]
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = ARCHITECTURE
    # the design has no longest sequence of its own (angles are computed from the position)
    max_position_embeddings: int = 1 << 30

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], where: str = "config.json") -> "PamaraxConfig":
        r = KeyReader(raw, where)
        width = r.integer("width", minimum=1)
        r.seen.add("layers")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: required key 'layers' must be a non-empty list")
        layers = []
        for i, item in enumerate(layers_raw):
            lw = f"{where}: layers[{i}]"
            lr = KeyReader(item, lw)
            kind = lr.string("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{lw}: unknown layer type '{kind}' (known: {', '.join(LAYER_TYPES)})")
            mixer = _MIXERS[kind](_sub(lr, "mixer"))
            ml = _sub(lr, "mlp", required=False)
            layers.append(PamaraxLayer(kind, mixer, None if ml is None else _mlp(ml)))
        emb = _sub(r, "embedding", required=False)
        return cls(vocab=r.integer("vocab", minimum=1), width=width, eps=_sub(r, "norm").real("eps", positive=True),
                   embedding_scale=emb.real("scale", default=1.0) if emb is not None else 1.0, layers=tuple(layers), raw=dict(raw),
                   eos_token_ids=tuple(r.token_ids("eos_token_id")))


def _grouped(m: KeyReader) -> Tuple[int, int, int, int]:
    heads = m.integer("heads", minimum=1)
    kv_heads = m.integer("kv_heads", default=heads, minimum=1)
    dim = m.integer("dim", minimum=1)
    vdim = m.integer("vdim", default=dim, minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{m.where}: heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return heads, kv_heads, dim, vdim


def _key_limit(m: KeyReader, what: str, size: int) -> None:
    if size > MAX_HEAD_SIZE:
        raise ConfigError(f"{m.where}: {what} ({size}) may not exceed the {MAX_HEAD_SIZE} elements the kernels take per head")


def _matrix_memory(m: KeyReader) -> MatrixMemoryConfig:
    cfg = MatrixMemoryConfig(m.integer("heads", minimum=1), m.integer("dim", minimum=1), m.integer("vdim", minimum=1),
                             m.real("gate_cap", positive=True))
    _key_limit(m, "dim", cfg.dim)
    if cfg.vdim > MAX_MEMORY_VALUES:
        raise ConfigError(f"{m.where}: vdim ({cfg.vdim}) may not exceed {MAX_MEMORY_VALUES}")
    return cfg


def _shared_value_attention(m: KeyReader) -> SharedValueAttentionConfig:
    heads, kv_heads, dim, vdim = _grouped(m)
    if vdim != dim:
        raise ConfigError(f"{m.where}: vdim ({vdim}) must be dim ({dim}): the keys are the values")
    _key_limit(m, "dim", dim)
    rot = _sub(m, "rot", required=False)
    dims, base = 0, 1.0
    if rot is not None:
        dims, base = rot.integer("dims", minimum=0), rot.real("base", positive=True)
        if dims % 2 or dims > dim:
            raise ConfigError(f"{rot.where}: dims ({dims}) must be even and at most the head's size ({dim})")
    return SharedValueAttentionConfig(heads, kv_heads, dim, m.real("scale"), dims, base)


def _sink_attention(m: KeyReader) -> SinkAttentionConfig:
    heads, kv_heads, dim, vdim = _grouped(m)
    _key_limit(m, "dim", dim)
    _key_limit(m, "vdim", vdim)
    temp = _sub(m, "q_temp", required=False)
    return SinkAttentionConfig(heads, kv_heads, dim, vdim, m.real("scale"),
                               None if temp is None else (temp.real("coef"), temp.integer("every", minimum=1)))


def _head_delta(m: KeyReader) -> HeadDeltaConfig:
    heads, kv_heads, dim, vdim = _grouped(m)
    _key_limit(m, "dim", dim)
    cfg = HeadDeltaConfig(heads, kv_heads, dim, vdim, taps=m.integer("conv", minimum=1))
    if cfg.taps > MAX_TAPS:
        raise ConfigError(f"{m.where}: conv ({cfg.taps}) may not exceed the {MAX_TAPS} taps the convolution kernel holds")
    if vdim > MAX_MEMORY_VALUES:
        raise ConfigError(f"{m.where}: vdim ({vdim}) may not exceed {MAX_MEMORY_VALUES}")
    return cfg


def _parallel(m: KeyReader) -> ParallelConfig:
    return ParallelConfig(_sink_attention(_sub(m, "left")), _head_delta(_sub(m, "right")), m.real("left_scale"), m.real("right_scale"))


_MIXERS = {"mlstm": _matrix_memory, "attention": _shared_value_attention, "parallel": _parallel}


def _mlp(ml: KeyReader) -> DenseMlpConfig:
    kind = ml.string("kind", default="dense")
    if kind != "dense":
        raise ConfigError(f"{ml.where}: unknown feed-forward kind '{kind}' (known: dense)")
    return DenseMlpConfig(ml.integer("ff", minimum=1))
