"""Typed configuration of the Tokovik decoder, read from config.json.

A Tokovik model is a list of layers. Every layer runs two mixers side by side on the
stream itself (`parallel`: a grouped attention inside a sliding window with biased
projections, normalised and rotated heads; and gated linear attention with a decay per
key channel) and a gated feed-forward (or none), each with a norm behind it. Keys:

    architecture: "Tokovik", vocab, width, norm.eps, embedding.scale, logit_scale,
    layers[i]: {type: "parallel", mixer: {left, right}, mlp: null | {kind: "dense", ff}}
    left:  heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {base, dims,
           scaling: {factor, original, fast, slow}}
    right: heads, dim, vdim, tau

Absent `mask`, `rot`, `rot.scaling` and `mlp` mean none; absent `embedding` and
`logit_scale` mean 1. The rank of the decays' projection is the one size that only a
tensor's shape gives (`right.a1`, `complete_from_files`); a document may name it as
`right.decay_rank` (models that have no files).
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Dict, Mapping, Optional, Tuple

from . import errors
from .fields import need as _need, positive as _positive
from .files import decode_json

ARCHITECTURE = "Tokovik"
MIXER_TYPES = ("parallel",)
# No key bounds the positions; 2^24 keeps every position exact in 32-bit floats.
MAX_POSITIONS = 1 << 24


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def to_json(self) -> dict:
        original = int(self.original) if float(self.original).is_integer() else self.original
        return {"factor": self.factor, "original": original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class TokovikAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None     # mask.size
    rot_dims: int = 0                # rot.dims
    rot_base: float = 10000.0        # rot.base
    rot_scaling: Optional[YarnScaling] = None

    def to_json(self) -> dict:
        doc: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim,
                               "vdim": self.vdim, "scale": self.scale}
        if self.window is not None:
            doc["mask"] = {"size": self.window}
        if self.rot_dims:
            doc["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
            if self.rot_scaling is not None:
                doc["rot"]["scaling"] = self.rot_scaling.to_json()
        return doc


@dataclass(frozen=True)
class TokovikLinear:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0  # 0: still to be read from the tensor's shape

    def to_json(self) -> dict:
        doc: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim,
                               "tau": self.tau}
        if self.decay_rank:
            doc["decay_rank"] = self.decay_rank
        return doc


@dataclass(frozen=True)
class TokovikLayer:
    type: str
    left: TokovikAttention
    right: TokovikLinear
    ff: Optional[int] = None  # None: no feed-forward

    def to_json(self) -> dict:
        return {"type": self.type,
                "mixer": {"left": self.left.to_json(), "right": self.right.to_json()},
                "mlp": None if self.ff is None else {"kind": "dense", "ff": self.ff}}


@dataclass(frozen=True)
class TokovikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[TokovikLayer, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @property
    def vocab_size(self) -> int:  # the name other parts of the library ask for
        return self.vocab

    @classmethod
    def parse(cls, source) -> "TokovikConfig":
        doc = decode_json(source)
        if doc.get("architecture") != ARCHITECTURE:
            raise errors.ModelType(f"architecture is {doc.get('architecture')!r}, "
                                   f"expected {ARCHITECTURE!r}")
        layers_doc = _need(doc, "layers", list, "config")
        if not layers_doc:
            raise errors.ConfigJson("config: no layers")
        embedding = _optional(doc, "embedding", "config") or {}
        known = {"architecture", "vocab", "width", "norm", "embedding", "logit_scale", "layers"}
        return cls(
            vocab=_positive(doc, "vocab", "config"), width=_positive(doc, "width", "config"),
            norm_eps=_need(_need(doc, "norm", dict, "config"), "eps", float, "norm"),
            layers=tuple(_parse_layer(e, f"layers[{i}]") for i, e in enumerate(layers_doc)),
            embedding_scale=_number(embedding, "scale", "embedding", 1.0),
            logit_scale=_number(doc, "logit_scale", "config", 1.0),
            extra={k: v for k, v in doc.items() if k not in known})

    def to_json(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "logit_scale": self.logit_scale, "layers": [l.to_json() for l in self.layers]}


def complete_from_files(config: TokovikConfig, files) -> TokovikConfig:
    """The rank of each layer's decay projection, from the first axis of its `a1` (`files`:
    anything with `in` and `entry(name).shape`, i.e. the opened weight files)."""
    layers = []
    for i, layer in enumerate(config.layers):
        name = f"l{i}.mix.right.a1"
        if name in files:
            right = replace(layer.right, decay_rank=int(files.entry(name).shape[0]))
            layer = replace(layer, right=right)
        layers.append(layer)
    return replace(config, layers=tuple(layers))


def _number(doc, key: str, where: str, default: float) -> float:
    return default if doc.get(key) is None else _need(doc, key, float, where)


def _optional(doc, key, where):
    value = doc.get(key)
    if value is not None and not isinstance(value, dict):
        raise errors.ConfigJson(f"{where}.{key} is not an object")
    return value


def _parse_scaling(rot, where: str) -> Optional[YarnScaling]:
    s = _optional(rot, "scaling", where)
    if s is None:
        return None
    w = f"{where}.scaling"
    out = YarnScaling(*(_need(s, key, float, w) for key in ("factor", "original", "fast", "slow")))
    if min(out.factor, out.original, out.fast, out.slow) <= 0:
        raise errors.ConfigJson(f"{w}: factor, original, fast and slow must be positive")
    return out


def _parse_attention(m, where: str) -> TokovikAttention:
    heads, kv_heads = _positive(m, "heads", where), _positive(m, "kv_heads", where)
    if heads % kv_heads:
        raise errors.HeadRatio(f"{where}: {heads} heads over {kv_heads} kv heads")
    dim = _positive(m, "dim", where)
    fields: Dict[str, Any] = dict(heads=heads, kv_heads=kv_heads, dim=dim,
                                  vdim=_positive(m, "vdim", where),
                                  scale=_need(m, "scale", float, where))
    mask = _optional(m, "mask", where)
    if mask is not None and mask.get("size") is not None:
        fields["window"] = _positive(mask, "size", f"{where}.mask")
    rot = _optional(m, "rot", where)
    if rot is not None and rot.get("dims"):
        w = f"{where}.rot"
        dims, base = _positive(rot, "dims", w), _need(rot, "base", float, w)
        if dims % 2 or dims > dim:
            raise errors.ConfigJson(f"{w}: {dims} rotated elements in heads of {dim}")
        fields.update(rot_dims=dims, rot_base=base, rot_scaling=_parse_scaling(rot, w))
        if base <= 0 or (fields["rot_scaling"] is not None and base == 1.0):
            raise errors.ConfigJson(f"{w}: base {base}")
    return TokovikAttention(**fields)


def _parse_linear(m, where: str) -> TokovikLinear:
    tau = _need(m, "tau", float, where)
    if tau <= 0:
        raise errors.ConfigJson(f"{where}: tau = {tau} must be positive")
    return TokovikLinear(heads=_positive(m, "heads", where), dim=_positive(m, "dim", where),
                         vdim=_positive(m, "vdim", where), tau=tau,
                         decay_rank=(_positive(m, "decay_rank", where)
                                     if m.get("decay_rank") is not None else 0))


def _parse_layer(entry, where: str) -> TokovikLayer:
    if not isinstance(entry, dict):
        raise errors.ConfigJson(f"{where} is not an object")
    kind = _need(entry, "type", str, where)
    if kind not in MIXER_TYPES:
        raise errors.UnsupportedOption(f"{where}: mixer type {kind!r}; known: {MIXER_TYPES}")
    m, w = _need(entry, "mixer", dict, where), f"{where}.mixer"
    ff = None
    mlp = _optional(entry, "mlp", where)
    if mlp is not None:
        mlp_kind = _need(mlp, "kind", str, f"{where}.mlp")
        if mlp_kind != "dense":
            raise errors.UnsupportedOption(f"{where}.mlp.kind {mlp_kind!r}; known: dense")
        ff = _positive(mlp, "ff", f"{where}.mlp")
    return TokovikLayer(kind, _parse_attention(_need(m, "left", dict, w), f"{w}.left"),
                        _parse_linear(_need(m, "right", dict, w), f"{w}.right"), ff)
