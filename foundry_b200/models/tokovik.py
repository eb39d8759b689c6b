"""The Tokovik decoder as data: config.json -> `ModelSpec`.

The table lookup times a constant as embedding; layers whose parts read the stream
itself and have a norm behind them, `x <- x + norm1(mixer(x)); x <- x + norm2(ff(x))`
(`post_norm_residual`; RMS norms whose stored weight is the distance from one); as
mixer two mixers side by side (`parallel`): an attention inside a sliding window
(`window_attention`, YaRN-scaled rotation) and gated linear attention
(`gated_linear_attention`), each result with an RMS norm of its own, half their sum; a
SiLU-gated feed-forward or none; a final norm, whose weight also carries the constant
on the logits, and a separate output head. Tensor names: `embed`, `head`, `final.norm`,
`l<i>.{norm1,norm2}`, `l<i>.mix.{left,right}.*`, `l<i>.mlp.{gate,up,down}`.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, default_schedule
from ..config.tokovik import (ARCHITECTURE, MAX_POSITIONS, TokovikConfig, TokovikLayer,
                              complete_from_files)
from ..parts.rope import banded_frequencies, yarn_frequencies

NAMES = {"mixer": "mix", "feed_forward": "mlp", "mixer_post_norm": "norm1",
         "feed_forward_post_norm": "norm2"}
PAIR_SCALE = 0.5  # on the sum of the two mixers' normalised results


def _mixer(config: TokovikConfig, layer: TokovikLayer) -> PartSpec:
    a, r = layer.left, layer.right
    factor = 1.0
    if a.rot_scaling is None:
        freq = banded_frequencies(a.rot_dims, a.rot_base)
    else:
        s = a.rot_scaling
        freq, factor = yarn_frequencies(a.rot_dims, a.rot_base, s.factor, s.original, s.fast, s.slow)
    left = PartSpec("window_attention", {
        "width": config.width, "heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim,
        "vdim": a.vdim, "scale": a.scale, "eps": config.norm_eps, "window": a.window,
        "frequencies": tuple(float(f) for f in freq), "rot_factor": factor, "bias": True})
    right = PartSpec("gated_linear_attention", {
        "width": config.width, "heads": r.heads, "dim": r.dim, "vdim": r.vdim,
        "decay_rank": r.decay_rank, "tau": r.tau, "eps": config.norm_eps, "gate": "silu"})
    return PartSpec("parallel", {"left": left, "right": right, "names": ("left", "right"),
                                 "out_norm": (config.norm_eps, PAIR_SCALE)})


def build_tokovik_spec(config: TokovikConfig) -> ModelSpec:
    stream = PartSpec("stream_input", {"size": config.width, "eps": config.norm_eps})
    norm = PartSpec("rms_norm", {"size": config.width, "eps": config.norm_eps,
                                 "weight_suffix": "", "weight_offset": 1.0})
    # the head is linear in its input, so the constant on the logits is a constant on it
    final = PartSpec("rms_norm", {**norm.params, "out_scale": config.logit_scale})
    layers = []
    for i, layer in enumerate(config.layers):
        ff = None
        if layer.ff is not None:
            ff = PartSpec("swiglu", {"hidden_size": config.width, "intermediate_size": layer.ff,
                                     "names": ("gate", "up", "down"), "suffix": "",
                                     "activation": "silu", "float_out": True})
        layers.append(LayerSpec(
            prefix=f"l{i}", block=PartSpec("post_norm_residual"), mixer=_mixer(config, layer),
            feed_forward=ff, mixer_norm=stream, names=NAMES,
            feed_forward_norm=stream if ff is not None else None, mixer_post_norm=norm,
            feed_forward_post_norm=norm if ff is not None else None))
    spec = ModelSpec(
        architecture=ARCHITECTURE, hidden_size=config.width, vocab_size=config.vocab,
        max_positions=MAX_POSITIONS, layers=tuple(layers), schedule=default_schedule(len(layers)),
        final_norm=final, embedding_name="embed", final_norm_prefix="final.norm",
        output_head_name="head", embedding=PartSpec("lookup", {"scale": config.embedding_scale}),
        # a layer without a feed-forward has no use for the norm behind one; a file that
        # carries it all the same is still this model
        ignorable_tensors=tuple(f"l{i}.norm2" for i, layer in enumerate(config.layers)
                                if layer.ff is None))
    spec.validate()
    return spec


TOKOVIK = register_architecture(Architecture(
    name=ARCHITECTURE, model_type="tokovik", parse_config=TokovikConfig.parse,
    build_spec=build_tokovik_spec, complete_from_files=complete_from_files), replace=True)
