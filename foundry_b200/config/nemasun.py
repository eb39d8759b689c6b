"""Typed configuration of the Nemasun decoder, read from config.json.

A Nemasun model keeps several copies of the residual stream. Every layer runs grouped
attention (normalised query and key heads, values that are the keys before their norm, a
learnt bias by distance, a sliding window that keeps the first tokens, an output gate) and
then a dense clamped feed-forward, routed experts, or nothing. Keys:

    architecture: "Nemasun", vocab, width, streams, norm.eps, embedding.scale,
    layers[i]: {type: "attention", mixer: {...}, mlp: null | {...}}
    mixer:     heads, kv_heads, dim, vdim, scale, bias_max, mask: {size, keep_first}
    mlp dense: {kind: "dense", ff, limit}
    mlp moe:   {kind: "moe", expert: {ff}, shared: {ff}, router: {experts, identity, top,
                groups: {count, keep}}}

Absent `mask`, `mask.size`, `mask.keep_first`, `router.groups`, `router.identity`, `shared`
and `mlp` mean none; an absent `embedding` means 1. Values are keys, so `vdim` is `dim`. How
many rows a layer's distance table has only the tensor's shape gives (`mix.rel`,
`complete_from_files`); a document may name it as `mixer.bias_rows`, for a model that is
drawn at random.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Any, Dict, Mapping, Optional, Tuple

from . import errors
from .fields import need as _need, positive as _positive
from .files import decode_json

ARCHITECTURE = "Nemasun"
MIXER_TYPES = ("attention",)
MLP_KINDS = ("dense", "moe")
MAX_STREAMS = 16
# No key bounds the positions; 2^24 keeps every position exact in 32-bit floats.
MAX_POSITIONS = 1 << 24


@dataclass(frozen=True)
class NemasunAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    bias_max: int
    window: Optional[int] = None
    keep_first: int = 0
    bias_rows: int = 0  # 0: still to be read from the tensor's shape

    def to_json(self) -> dict:
        doc: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim,
                               "vdim": self.dim, "scale": self.scale, "bias_max": self.bias_max}
        if self.window is not None:
            doc["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.bias_rows:
            doc["bias_rows"] = self.bias_rows
        return doc


@dataclass(frozen=True)
class NemasunDense:
    ff: int
    limit: float

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class NemasunExperts:
    ff: int
    experts: int
    top: int
    identity: int = 0
    group_count: int = 1
    group_keep: int = 1
    shared_ff: int = 0

    def to_json(self) -> dict:
        doc: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": {
            "experts": self.experts, "identity": self.identity, "top": self.top,
            "groups": {"count": self.group_count, "keep": self.group_keep}}}
        if self.shared_ff:
            doc["shared"] = {"ff": self.shared_ff}
        return doc


@dataclass(frozen=True)
class NemasunLayer:
    type: str
    attention: NemasunAttention
    dense: Optional[NemasunDense] = None
    experts: Optional[NemasunExperts] = None

    def to_json(self) -> dict:
        mlp = self.dense or self.experts
        return {"type": self.type, "mixer": self.attention.to_json(),
                "mlp": None if mlp is None else mlp.to_json()}


@dataclass(frozen=True)
class NemasunConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[NemasunLayer, ...]
    embedding_scale: float = 1.0
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @property
    def vocab_size(self) -> int:  # the name other parts of the library ask for
        return self.vocab

    @classmethod
    def parse(cls, source) -> "NemasunConfig":
        doc = decode_json(source)
        if doc.get("architecture") != ARCHITECTURE:
            raise errors.ModelType(f"architecture is {doc.get('architecture')!r}, "
                                   f"expected {ARCHITECTURE!r}")
        layers_doc = _need(doc, "layers", list, "config")
        if not layers_doc:
            raise errors.ConfigJson("config: no layers")
        streams = _positive(doc, "streams", "config")
        if streams > MAX_STREAMS:
            raise errors.UnsupportedOption(f"config: {streams} streams (at most {MAX_STREAMS})")
        embedding = _optional(doc, "embedding", "config") or {}
        known = {"architecture", "vocab", "width", "streams", "norm", "embedding", "layers"}
        return cls(
            vocab=_positive(doc, "vocab", "config"), width=_positive(doc, "width", "config"),
            streams=streams,
            norm_eps=_need(_need(doc, "norm", dict, "config"), "eps", float, "norm"),
            layers=tuple(_parse_layer(e, f"layers[{i}]") for i, e in enumerate(layers_doc)),
            embedding_scale=(1.0 if embedding.get("scale") is None
                             else _need(embedding, "scale", float, "embedding")),
            extra={k: v for k, v in doc.items() if k not in known})

    def to_json(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "streams": self.streams, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale},
                "layers": [layer.to_json() for layer in self.layers]}


def complete_from_files(config: NemasunConfig, files) -> NemasunConfig:
    """The rows of each layer's distance table, from the first axis of its `rel` (`files`:
    anything with `in` and `entry(name).shape`, i.e. the opened weight files)."""
    layers = []
    for i, layer in enumerate(config.layers):
        name = f"l{i}.mix.rel"
        if name in files:
            rows = int(files.entry(name).shape[0])
            _check_table(layer.attention.bias_max, rows, f"layers[{i}].mixer")
            layer = replace(layer, attention=replace(layer.attention, bias_rows=rows))
        layers.append(layer)
    return replace(config, layers=tuple(layers))


def _check_table(bias_max: int, rows: int, where: str) -> None:
    if rows < 2 or bias_max <= rows // 2:
        raise errors.ConfigJson(f"{where}: bias_max {bias_max} with a table of {rows} rows (half "
                                f"of them are single distances)")


def _optional(doc, key, where):
    value = doc.get(key)
    if value is not None and not isinstance(value, dict):
        raise errors.ConfigJson(f"{where}.{key} is not an object")
    return value


def _count(doc, key: str, where: str) -> int:
    """A number that may be absent or 0."""
    value = 0 if doc.get(key) is None else _need(doc, key, int, where)
    if value < 0:
        raise errors.ConfigJson(f"{where}: {key} = {value} must not be negative")
    return value


def _parse_attention(m, where: str) -> NemasunAttention:
    heads, kv_heads = _positive(m, "heads", where), _positive(m, "kv_heads", where)
    if heads % kv_heads:
        raise errors.HeadRatio(f"{where}: {heads} heads over {kv_heads} kv heads")
    dim, vdim = _positive(m, "dim", where), _positive(m, "vdim", where)
    if vdim != dim:
        raise errors.UnsupportedOption(f"{where}: values of {vdim} cannot be keys of {dim}")
    fields: Dict[str, Any] = dict(heads=heads, kv_heads=kv_heads, dim=dim,
                                  scale=_need(m, "scale", float, where),
                                  bias_max=_positive(m, "bias_max", where))
    mask = _optional(m, "mask", where)
    if mask is not None and mask.get("size") is not None:
        fields.update(window=_positive(mask, "size", f"{where}.mask"),
                      keep_first=_count(mask, "keep_first", f"{where}.mask"))
    if m.get("bias_rows") is not None:
        fields["bias_rows"] = _positive(m, "bias_rows", where)
        _check_table(fields["bias_max"], fields["bias_rows"], where)
    return NemasunAttention(**fields)


def _parse_experts(mlp, where: str) -> NemasunExperts:
    router, wr = _need(mlp, "router", dict, where), f"{where}.router"
    groups = _optional(router, "groups", wr)
    count = keep = 1
    if groups is not None:
        count, keep = (_positive(groups, key, f"{wr}.groups") for key in ("count", "keep"))
    shared = _optional(mlp, "shared", where)
    out = NemasunExperts(
        ff=_positive(_need(mlp, "expert", dict, where), "ff", f"{where}.expert"),
        experts=_positive(router, "experts", wr), top=_positive(router, "top", wr),
        identity=_count(router, "identity", wr), group_count=count, group_keep=keep,
        shared_ff=0 if shared is None else _positive(shared, "ff", f"{where}.shared"))
    outputs = out.experts + out.identity
    if outputs % count or keep > count or keep * (outputs // count) < out.top:
        raise errors.ConfigJson(f"{wr}: {outputs} experts in {count} groups, {keep} kept, "
                                f"{out.top} chosen")
    return out


def _parse_layer(entry, where: str) -> NemasunLayer:
    if not isinstance(entry, dict):
        raise errors.ConfigJson(f"{where} is not an object")
    kind = _need(entry, "type", str, where)
    if kind not in MIXER_TYPES:
        raise errors.UnsupportedOption(f"{where}: mixer type {kind!r}; known: {MIXER_TYPES}")
    attention = _parse_attention(_need(entry, "mixer", dict, where), f"{where}.mixer")
    mlp, wm = _optional(entry, "mlp", where), f"{where}.mlp"
    if mlp is None:
        return NemasunLayer(kind, attention)
    mlp_kind = _need(mlp, "kind", str, wm)
    if mlp_kind not in MLP_KINDS:
        raise errors.UnsupportedOption(f"{wm}.kind {mlp_kind!r}; known: {MLP_KINDS}")
    if mlp_kind == "moe":
        return NemasunLayer(kind, attention, experts=_parse_experts(mlp, wm))
    limit = _need(mlp, "limit", float, wm)
    if limit <= 0.0:
        raise errors.ConfigJson(f"{wm}: limit = {limit} must be positive")
    return NemasunLayer(kind, attention, dense=NemasunDense(_positive(mlp, "ff", wm), limit))
