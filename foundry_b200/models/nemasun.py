"""The Nemasun decoder as data: config.json -> `ModelSpec`.

The table lookup times a constant as embedding; several copies of the stream, which every
layer's two parts read as a weighted sum and write back while they are mixed
(`stream_mix_residual`); RMS norms in front of the parts; as mixer grouped attention whose
values are the keys before their norm (`shared_row_attention`: a bias by distance, a window
that keeps the first tokens, an output gate); as feed-forward a dense one with clamped halves
and biases (`clamped_glu`) or routed experts with softmax scores, a correction of the choice,
groups, identity experts and a shared expert; a final norm of the streams' sum and a separate
output head. Tensor names: `embed`, `head`, `final.norm`, `l<i>.{norm1,norm2}`, `l<i>.mix.*`,
`l<i>.mlp.*`, `l<i>.{hc1,hc2}.{in,out,mix}`.
"""
from __future__ import annotations

from ..config.nemasun import (ARCHITECTURE, MAX_POSITIONS, NemasunConfig, NemasunLayer,
                              complete_from_files)
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, default_schedule

NAMES = {"mixer": "mix", "feed_forward": "mlp", "mixer_norm": "norm1",
         "feed_forward_norm": "norm2"}
MIXER_STREAMS, FEED_FORWARD_STREAMS = "hc1", "hc2"  # where a layer's mixing weights lie
GATE_SLOPE = 1.702   # of the dense feed-forward's gate: g * sigmoid(slope g)
UP_SHIFT = 1.0       # what joins its other half
WEIGHT_SUM_FLOOR = 1e-20  # joins the sum of the chosen experts' scores under the division
DEFAULT_BIAS_ROWS = 32  # of a distance table that neither a file nor the document sizes


def _mixer(config: NemasunConfig, layer: NemasunLayer) -> PartSpec:
    a = layer.attention
    return PartSpec("shared_row_attention", {
        "width": config.width, "heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim,
        "scale": a.scale, "eps": config.norm_eps, "bias_max": a.bias_max,
        "bias_rows": a.bias_rows or min(DEFAULT_BIAS_ROWS, 2 * a.bias_max - 1),
        "window": a.window, "keep_first": a.keep_first, "output_gate": True})


def _feed_forward(config: NemasunConfig, layer: NemasunLayer):
    if layer.dense is not None:
        return PartSpec("clamped_glu", {
            "hidden_size": config.width, "intermediate_size": layer.dense.ff,
            "limit": layer.dense.limit, "alpha": GATE_SLOPE, "shift": UP_SHIFT, "bias": True})
    e = layer.experts
    if e is None:
        return None
    return PartSpec("routed_experts", {
        "width": config.width, "ff": e.ff, "experts": e.experts, "identity": e.identity,
        "top": e.top, "limit": float("inf"), "alpha": 1.0, "shift": 0.0, "score": "softmax",
        "groups": e.group_count, "keep": e.group_keep, "group_best": 1, "router_bias": False,
        "choice_correction": True, "correction_name": "correction", "normalise": True,
        "sum_floor": WEIGHT_SUM_FLOOR, "shared_ff": e.shared_ff, "shared_name": "shared"})


def build_nemasun_spec(config: NemasunConfig) -> ModelSpec:
    norm = PartSpec("rms_norm", {"size": config.width, "eps": config.norm_eps,
                                 "weight_suffix": ""})
    block = PartSpec("stream_mix_residual", {
        "streams": config.streams, "mixer_name": MIXER_STREAMS,
        "feed_forward_name": FEED_FORWARD_STREAMS})
    layers, ignorable = [], []
    for i, layer in enumerate(config.layers):
        ff = _feed_forward(config, layer)
        layers.append(LayerSpec(
            prefix=f"l{i}", block=block, mixer=_mixer(config, layer), feed_forward=ff,
            mixer_norm=norm, feed_forward_norm=norm if ff is not None else None, names=NAMES))
        if ff is None:  # tensors for which such a layer has no use; a file may carry them
            ignorable += [f"l{i}.norm2", f"l{i}.{FEED_FORWARD_STREAMS}.*"]
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=config.width, vocab_size=config.vocab,
        max_positions=MAX_POSITIONS, layers=tuple(layers), schedule=default_schedule(len(layers)),
        final_norm=norm, embedding_name="embed", final_norm_prefix="final.norm",
        output_head_name="head", embedding=PartSpec("lookup", {"scale": config.embedding_scale}),
        ignorable_tensors=tuple(ignorable), streams=config.streams)
    spec.validate()
    return spec


NEMASUN = register_architecture(Architecture(
    name=ARCHITECTURE, model_type="nemasun", parse_config=NemasunConfig.parse,
    build_spec=build_nemasun_spec, complete_from_files=complete_from_files), replace=True)
