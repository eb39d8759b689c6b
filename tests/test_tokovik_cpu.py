"""Tokovik without a GPU: configuration, the model as data, the tensor list, the
frequencies, the plan of the chunked scan, and the plain implementation against
its own token-by-token form and against cases worked by hand."""
import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tokovik as plain
import tokovik_tiny as tiny


def parsed(name):
    """The typed configuration with the sizes that only the tensors' shapes give."""
    from foundry_b200.config.tokovik import TokovikConfig, complete_from_files
    shapes = tiny.tensor_shapes(tiny.CONFIGS[name], tiny.RANKS[name])

    class Files(dict):
        def entry(self, key):
            return SimpleNamespace(shape=self[key])
    return complete_from_files(TokovikConfig.parse(tiny.CONFIGS[name]), Files(shapes))


def double(weights):
    return {k: v.double() for k, v in weights.items()}


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_config_round_trip_and_registry(name):
    from foundry_b200.config.registry import resolve_architecture
    cfg, doc = parsed(name), tiny.CONFIGS[name]
    assert type(cfg).parse(json.dumps(cfg.to_json())) == cfg
    assert resolve_architecture(doc).name == "Tokovik"
    assert (cfg.width, cfg.vocab_size, len(cfg.layers)) == (doc["width"], doc["vocab"],
                                                            len(doc["layers"]))
    assert (cfg.embedding_scale, cfg.logit_scale) == (doc["embedding"]["scale"], doc["logit_scale"])
    for layer, entry, rank in zip(cfg.layers, doc["layers"], tiny.RANKS[name]):
        assert layer.left.window == entry["mixer"]["left"]["mask"]["size"]
        assert (layer.right.tau, layer.right.decay_rank) == (entry["mixer"]["right"]["tau"], rank)
        assert (layer.left.rot_scaling is None) == ("scaling" not in entry["mixer"]["left"]["rot"])
        assert layer.ff == (entry["mlp"] or {}).get("ff")


def test_config_defaults_of_absent_keys():
    from foundry_b200.config.tokovik import TokovikConfig
    doc = json.loads(json.dumps(tiny.CONFIGS["other"]))
    left = doc["layers"][0]["mixer"]["left"]
    del left["mask"], left["rot"], doc["embedding"], doc["logit_scale"], doc["layers"][1]["mlp"]
    cfg = TokovikConfig.parse(doc)
    assert cfg.layers[0].left.window is None and cfg.layers[0].left.rot_dims == 0
    assert cfg.layers[1].ff is None and (cfg.embedding_scale, cfg.logit_scale) == (1.0, 1.0)
    assert type(cfg).parse(json.dumps(cfg.to_json())) == cfg


@pytest.mark.parametrize("path, value, error", [
    (("layers", 0, "mixer", "left", "kv_heads"), 4, "HeadRatio"),
    (("layers", 1, "type"), "serial", "UnsupportedOption"),
    (("layers", 0, "mlp", "kind"), "moe", "UnsupportedOption"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 26, "ConfigJson"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 7, "ConfigJson"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0, "ConfigJson"),
    (("layers", 0, "mixer", "left", "mask", "size"), 0, "ConfigJson"),
    (("layers", 2, "mixer", "right", "tau"), -1.0, "ConfigJson"),
    (("norm",), None, "ConfigJson"),
    (("layers",), [], "ConfigJson"),
])
def test_config_refusals(path, value, error):
    from foundry_b200.config import errors
    from foundry_b200.config.tokovik import TokovikConfig
    doc = json.loads(json.dumps(tiny.CONFIGS["mixed"]))
    at = doc
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(getattr(errors, error)):
        TokovikConfig.parse(doc)


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_tensor_list_and_the_model_as_data(name):
    from foundry_b200.cache import JointRequest
    from foundry_b200.engine.model import Model, expected_tensors
    from foundry_b200.models.tokovik import build_tokovik_spec
    doc = tiny.CONFIGS[name]
    spec = build_tokovik_spec(parsed(name))
    listed = {k: tuple(v.shape) for k, v in expected_tensors(spec).items()}
    assert listed == tiny.tensor_shapes(doc, tiny.RANKS[name])
    assert [(e.layer, e.cache) for e in spec.schedule] == [(i, i) for i in range(len(spec.layers))]
    model = Model(spec, torch.bfloat16, torch.device("meta"))
    assert model.replay_safe()
    for block, entry in zip(model.blocks, doc["layers"]):
        want = block.cache_request()
        left, right = entry["mixer"]["left"], entry["mixer"]["right"]
        assert isinstance(want, JointRequest)
        assert (want.kv.kv_heads, want.kv.head_dim, want.kv.v_head_dim, want.kv.window) == \
            (left["kv_heads"], left["dim"], left["vdim"], None)
        assert want.state.shape == (right["heads"] * right["dim"] * right["vdim"],)
        assert want.state.dtype == torch.float32


def test_a_norm_behind_nothing_may_lie_in_the_file():
    """A layer without feed-forward has no `norm2`; a file that has one is still read."""
    import fnmatch
    from foundry_b200.models.tokovik import build_tokovik_spec
    spec = build_tokovik_spec(parsed("mixed"))
    assert any(fnmatch.fnmatch("l1.norm2", p) for p in spec.ignorable_tensors)
    assert not any(fnmatch.fnmatch("l0.norm2", p) for p in spec.ignorable_tensors)


@pytest.mark.parametrize("rot", [
    {"dims": 12, "base": 500.0, "scaling": {"factor": 3.0, "original": 64, "fast": 6.0, "slow": 0.5}},
    {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}},
    # every element in front of the ramp; every one behind it; first and last of the ramp the same
    {"dims": 16, "base": 10000.0, "scaling": {"factor": 2.0, "original": 10 ** 9, "fast": 4.0, "slow": 2.0}},
    {"dims": 16, "base": 10000.0, "scaling": {"factor": 2.0, "original": 2, "fast": 4.0, "slow": 2.0}},
    {"dims": 8, "base": 7.0, "scaling": {"factor": 1.0, "original": 100, "fast": 3.0, "slow": 3.0}},
])
def test_yarn_frequencies(rot):
    from foundry_b200.parts.rope import yarn_frequencies
    s = rot["scaling"]
    f, factor = yarn_frequencies(rot["dims"], rot["base"], s["factor"], s["original"], s["fast"],
                                 s["slow"])
    want, want_factor = plain.yarn(rot)
    assert f.dtype == np.float64 and np.abs(f - want.numpy()).max() < 1e-14
    assert abs(factor - want_factor) < 1e-15


def test_yarn_by_hand():
    """dims 8, base 10^4, original 2 pi 10^3: an element of t turns is number
    8 ln(1000 / t) / (2 ln 10^4); fast = 100 gives 1, slow = 1 gives 3."""
    rot = {"dims": 8, "base": 1e4, "scaling": {"factor": 4.0, "original": 2000.0 * math.pi,
                                               "fast": 100.0 * (1 - 1e-12), "slow": 1.0}}
    f, factor = plain.yarn(rot)
    plain_f = [1.0, 0.1, 0.01, 0.001]
    want = [plain_f[0], plain_f[1], plain_f[2] * (0.5 + 0.5 / 4.0), plain_f[3] / 4.0]
    assert max(abs(float(a) - b) for a, b in zip(f, want)) < 1e-9
    assert abs(factor - (0.1 * math.log(4.0) + 1.0)) < 1e-15


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_plain_linear_attention_equals_its_stepwise_form(name):
    cfg, w = tiny.CONFIGS[name], double(tiny.random_weights(name))
    torch.manual_seed(3)
    h = torch.randn(13, cfg["width"], dtype=torch.float64)
    for i, layer in enumerate(cfg["layers"]):
        args = (layer["mixer"]["right"], w, f"l{i}.mix.right", h, cfg["norm"]["eps"])
        a, b = plain.gated_linear(*args), plain.gated_linear_stepwise(*args)
        assert float((a - b).abs().max()) < 1e-10 * max(1.0, float(a.abs().max()))


def test_plain_linear_attention_by_hand():
    """One head of two key channels and one value, three tokens: decays 1/2 and 1/4 a token
    (sigmoid of the bias, root 1), the newest token undecayed."""
    F = plain.F
    m = {"heads": 1, "dim": 2, "vdim": 1, "tau": 1.0}
    w = {"a.q": torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F),
         "a.k": torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F), "a.v": torch.tensor([[1.0, 1.0]], dtype=F),
         "a.g": torch.tensor([[5.0, 5.0]], dtype=F), "a.a1": torch.zeros(1, 2, dtype=F),
         "a.a2": torch.zeros(2, 1, dtype=F),
         "a.a2.b": torch.tensor([0.0, -math.log(3.0)], dtype=F),  # sigmoid: 1/2, 1/4
         "a.norm": torch.ones(1, dtype=F), "a.o": torch.ones(1, 1, dtype=F)}
    h = torch.tensor([[1.0, 2.0], [0.0, 0.0], [1.0, 1.0]], dtype=F)
    q, k, v, log_a = plain._linear_inputs(m, w, "a", h)
    assert torch.allclose(torch.exp(log_a[:, 0]), torch.tensor([[0.5, 0.25]] * 3, dtype=F))
    # S after token 0: (1, 2) * 3; behind two more decays (1/4, 1/16); token 2 adds (1, 1) * 2
    S = torch.tensor([3.0 / 4 + 2.0, 6.0 / 16 + 2.0], dtype=F)
    want = float(S.sum()) / math.sqrt(2.0)  # q = (1, 1) / sqrt(2)
    big = 1e6  # eps so large that the norm is a constant factor: o / 1000
    got = float(plain.gated_linear(m, w, "a", h, big)[2, 0]) / float(plain.silu(torch.tensor(10.0, dtype=F)))
    assert abs(got * math.sqrt(want ** 2 + big) - want) < 1e-9


def test_plain_window_attention_by_hand():
    """One head, a window of two: biases join before the heads' norms, the query's own
    key and the one in front of it are seen, the key before that is not."""
    F = plain.F
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.5, "mask": {"size": 2}}
    eye = torch.eye(2, dtype=F)
    w = {"a.q": eye, "a.k": eye, "a.v": eye, "a.o": eye, "a.q.b": torch.tensor([0.0, 1.0], dtype=F),
         "a.k.b": torch.zeros(2, dtype=F), "a.v.b": torch.tensor([10.0, 0.0], dtype=F),
         "a.q.norm": torch.tensor([2.0, 1.0], dtype=F), "a.k.norm": torch.ones(2, dtype=F)}
    h = torch.tensor([[5.0, 0.0], [0.0, 3.0], [4.0, 0.0]], dtype=F)
    out = plain.window_attention(m, w, "a", h, 1e-12)
    # token 2: query (4, 1) normed and weighted; keys of tokens 1 and 2 are sqrt(2) (0, 1), sqrt(2) (1, 0)
    rms = math.sqrt(17.0 / 2.0)
    s1, s2 = 0.5 * math.sqrt(2.0) * 1.0 / rms, 0.5 * math.sqrt(2.0) * 8.0 / rms
    p2 = 1.0 / (1.0 + math.exp(s1 - s2))
    assert abs(float(out[2, 0]) - (10.0 + 4.0 * p2)) < 1e-9
    assert abs(float(out[2, 1]) - 3.0 * (1.0 - p2)) < 1e-9
    assert plain.window_visible(5, 4, 2) and not plain.window_visible(5, 3, 2)
    assert not plain.window_visible(4, 5, 2) and plain.window_visible(700, 0, None)
    assert plain.window_visible(3, 3, 1) and not plain.window_visible(3, 2, 1)


def test_plain_rotation_pairs_halves_and_scales_the_rotated_elements_only():
    x = torch.tensor([[[1.0, 2.0, 0.0, 0.0, 7.0, 9.0]]], dtype=plain.F).repeat(3, 1, 1)
    y = plain.rotate_half(x, [0, 1, 5], torch.tensor([1.0, 0.1], dtype=plain.F), 1.5)
    assert torch.equal(y[:, :, 4:], x[:, :, 4:]) and torch.equal(y[0, :, :4], 1.5 * x[0, :, :4])
    assert abs(float(y[2, 0, 0]) - 1.5 * math.cos(5.0)) < 1e-12
    assert abs(float(y[2, 0, 2]) - 1.5 * math.sin(5.0)) < 1e-12
    assert abs(float(y[1, 0, 3]) - 3.0 * math.sin(0.1)) < 1e-12


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_plain_model_is_causal(name):
    cfg, w = tiny.CONFIGS[name], double(tiny.random_weights(name))
    tokens = torch.randint(0, cfg["vocab"], (27,), generator=torch.Generator().manual_seed(4)).tolist()
    streams = []
    full = plain.forward(cfg, w, tokens, streams)
    assert len(streams) == len(cfg["layers"]) and full.shape == (27, cfg["vocab"])
    assert float((full[:12] - plain.forward(cfg, w, tokens[:12])).abs().max()) < 1e-9


def test_plan_of_the_chunked_scan():
    """Chunks cover the longest sequence, no chunk starts behind its end, single tokens, the
    delta rule and full devices are scanned in order."""
    from foundry_b200.kernels import ops
    for longest in (1, 63, 255, 256, 257, 1000, 2048, 5000, 100000):
        for seqs, heads, dim, vdim in ((1, 4, 32, 32), (1, 16, 128, 128), (3, 2, 12, 20), (64, 32, 128, 64)):
            ctx = SimpleNamespace(max_q_len=longest, n_seqs=seqs, is_decode=False)
            count, chunk = ops.scan_chunks(ctx, ops.SCAN_LINEAR, heads, dim, vdim)
            if count > 1:
                assert (count - 1) * chunk < longest <= count * chunk and chunk >= ops.SCAN_CHUNK_TOKENS
            if longest < 4 * ops.SCAN_CHUNK_TOKENS or seqs == 64:
                assert count == 1
    ctx = SimpleNamespace(max_q_len=4096, n_seqs=1, is_decode=False)
    assert ops.scan_chunks(ctx, ops.SCAN_DELTA, 4, 32, 32)[0] == 1
    ctx.is_decode = True
    assert ops.scan_chunks(ctx, ops.SCAN_LINEAR, 4, 32, 32)[0] == 1
