"""Typed configuration of the Vukotar decoder.

config.json of this design is nested: ``vocab``, ``width``, ``norm`` (eps), ``embedding`` (scale), ``logit_softcap`` and
``layers``, a list in which every entry names its mixer (``type``: attention), the mixer's sizes and constants
(``mixer``), its feed-forward (``mlp``, or null for none; ``kind`` moe) and, where it has no tensors of its own, the
layer whose tensors it uses (``weights_of``).  The order of the layers and all sizes are data: two models of the
design may differ in all of it.  Every size and constant is read here; the parts get them as parameters.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .lumevik import _sub
from .reader import ConfigError, KeyReader

ARCHITECTURE = "Vukotar"
# constants the design fixes
POSITION_BASE = 10000.0      # base of the sinusoidal positions' frequencies
ROUTER_WEIGHT_FLOOR = 1e-20  # added to the sum of the chosen experts' scores before the division
GROUP_TOP = 2                # a group of experts is worth the sum of this many of its largest scores
# limit of the kernels the design's attention launches (csrc/bias_attention.cu BA_MAX_DIM)
MAX_HEAD_SIZE = 256


@dataclass(frozen=True)
class SinkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float


@dataclass(frozen=True)
class MoeMlpConfig:
    experts: int
    top: int
    groups: int
    keep_groups: int
    ff: int


@dataclass(frozen=True)
class VukotarLayer:
    type: str
    mixer: SinkAttentionConfig
    mlp: Optional[MoeMlpConfig]
    weights_of: Optional[int]      # the layer with tensors of its own whose tensors this one uses; None: its own


@dataclass(frozen=True)
class VukotarConfig:
    vocab: int
    width: int
    embedding_scale: float
    logit_softcap: float           # 0: the logits are not capped
    layers: Tuple[VukotarLayer, ...]
    raw: Dict[str, Any]
    eos_token_ids: Tuple[int, ...] = ()
    architecture: str = ARCHITECTURE
    # the design has no longest sequence of its own (positions are computed, not looked up)
    max_position_embeddings: int = 1 << 30

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], where: str = "config.json") -> "VukotarConfig":
        r = KeyReader(raw, where)
        width = r.integer("width", minimum=1)
        r.seen.add("layers")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError(f"{where}: required key 'layers' must be a non-empty list")
        layers: List[VukotarLayer] = []
        for i, item in enumerate(layers_raw):
            lw = f"{where}: layers[{i}]"
            lr = KeyReader(item, lw)
            kind = lr.string("type")
            if kind != "attention":
                raise ConfigError(f"{lw}: unknown layer type '{kind}' (known: attention)")
            mixer = _attention(_sub(lr, "mixer"))
            ml = _sub(lr, "mlp", required=False)
            src = lr.integer("weights_of", minimum=0) if lr.has("weights_of") else None
            layers.append(VukotarLayer(kind, mixer, None if ml is None else _mlp(ml), src))
        layers = _resolve(layers, where)
        emb, norm = _sub(r, "embedding", required=False), _sub(r, "norm", required=False)
        if norm is not None:
            norm.real("eps", default=1e-5, positive=True)         # read and checked; the design's norm takes no statistics
        cap = r.real("logit_softcap", default=0.0)
        if cap < 0.0:
            raise ConfigError(f"{where}: logit_softcap ({cap}) must not be negative")
        return cls(vocab=r.integer("vocab", minimum=1), width=width,
                   embedding_scale=emb.real("scale", default=1.0) if emb is not None else 1.0, logit_softcap=cap,
                   layers=tuple(layers), raw=dict(raw), eos_token_ids=tuple(r.token_ids("eos_token_id")))


def _resolve(layers: List[VukotarLayer], where: str) -> List[VukotarLayer]:
    """Every `weights_of` followed to the layer that has the tensors, whose sizes must be the same."""
    out = []
    for i, l in enumerate(layers):
        j, seen = l.weights_of, {i}
        while j is not None and j < len(layers) and j not in seen and layers[j].weights_of is not None:
            seen.add(j)
            j = layers[j].weights_of
        if j is not None:
            if j >= len(layers) or j in seen:
                raise ConfigError(f"{where}: layers[{i}]: weights_of ({l.weights_of}) leads to no layer with tensors of its own")
            o = layers[j]
            if (o.type, o.mixer, o.mlp) != (l.type, l.mixer, l.mlp):
                raise ConfigError(f"{where}: layers[{i}]: weights_of ({l.weights_of}) names a layer with other sizes")
        out.append(VukotarLayer(l.type, l.mixer, l.mlp, j))
    return out


def _attention(m: KeyReader) -> SinkAttentionConfig:
    heads = m.integer("heads", minimum=1)
    dim = m.integer("dim", minimum=1)
    cfg = SinkAttentionConfig(heads, m.integer("kv_heads", default=heads, minimum=1), dim,
                              m.integer("vdim", default=dim, minimum=1), scale=m.real("scale"))
    if cfg.heads % cfg.kv_heads:
        raise ConfigError(f"{m.where}: heads ({cfg.heads}) must be a multiple of kv_heads ({cfg.kv_heads})")
    if max(cfg.dim, cfg.vdim) > MAX_HEAD_SIZE:
        raise ConfigError(f"{m.where}: dim ({cfg.dim}) and vdim ({cfg.vdim}) may not exceed the {MAX_HEAD_SIZE} elements "
                          f"the attention kernels take per key or value")
    return cfg


def _mlp(ml: KeyReader) -> MoeMlpConfig:
    kind = ml.string("kind", default="moe")
    if kind != "moe":
        raise ConfigError(f"{ml.where}: unknown feed-forward kind '{kind}' (known: moe)")
    ex, ro = _sub(ml, "expert"), _sub(ml, "router")
    gr = _sub(ro, "groups", required=False)
    cfg = MoeMlpConfig(experts=ro.integer("experts", minimum=1), top=ro.integer("top", minimum=1),
                       groups=gr.integer("count", minimum=1) if gr is not None else 1,
                       keep_groups=gr.integer("keep", minimum=1) if gr is not None else 1, ff=ex.integer("ff", minimum=1))
    if cfg.top > cfg.experts:
        raise ConfigError(f"{ro.where}: top ({cfg.top}) exceeds experts ({cfg.experts})")
    if cfg.experts % cfg.groups or cfg.keep_groups > cfg.groups:
        raise ConfigError(f"{ro.where}: {cfg.experts} experts do not form {cfg.groups} equal groups of which "
                          f"{cfg.keep_groups} are kept")
    if cfg.keep_groups * (cfg.experts // cfg.groups) < cfg.top:
        raise ConfigError(f"{ro.where}: {cfg.keep_groups} groups of {cfg.experts // cfg.groups} experts cannot give "
                          f"{cfg.top} choices")
    return cfg
