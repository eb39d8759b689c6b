"""Nemasun without a GPU: configuration, the model as data, the tensor list, the distance
buckets, the cache's rows with numbers beside them, and the plain implementation against cases
worked by hand."""
import fnmatch
import json
import math
from types import SimpleNamespace

import pytest
import torch

import nemasun_tiny as tiny
import plain_nemasun as plain

F = plain.F


class Files(dict):
    def entry(self, key):
        return SimpleNamespace(shape=self[key])


def parsed(name):
    """The typed configuration with the sizes that only the tensors' shapes give."""
    from foundry_b200.config.nemasun import NemasunConfig, complete_from_files
    shapes = tiny.tensor_shapes(tiny.CONFIGS[name], tiny.BIAS_ROWS[name])
    return complete_from_files(NemasunConfig.parse(tiny.CONFIGS[name]), Files(shapes))


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_config_round_trip_and_registry(name):
    from foundry_b200.config.registry import resolve_architecture
    cfg, doc = parsed(name), tiny.CONFIGS[name]
    assert type(cfg).parse(json.dumps(cfg.to_json())) == cfg
    assert resolve_architecture(doc).name == "Nemasun"
    assert (cfg.width, cfg.vocab_size, cfg.streams, len(cfg.layers)) == (
        doc["width"], doc["vocab"], doc["streams"], len(doc["layers"]))
    assert cfg.embedding_scale == doc["embedding"]["scale"]
    for layer, entry, rows in zip(cfg.layers, doc["layers"], tiny.BIAS_ROWS[name]):
        m, mlp = entry["mixer"], entry["mlp"] or {}
        mask = m.get("mask") or {}
        assert layer.attention.bias_rows == rows and layer.attention.bias_max == m["bias_max"]
        assert layer.attention.window == mask.get("size")
        assert layer.attention.keep_first == mask.get("keep_first", 0)
        assert (layer.dense is None) == (mlp.get("kind") != "dense")
        assert (layer.experts is None) == (mlp.get("kind") != "moe")
        if layer.experts is not None:
            router = mlp["router"]
            assert layer.experts.identity == router.get("identity", 0)
            assert layer.experts.shared_ff == (mlp.get("shared") or {}).get("ff", 0)
            assert layer.experts.group_count == router.get("groups", {}).get("count", 1)


@pytest.mark.parametrize("path, value, error", [
    (("layers", 0, "mixer", "kv_heads"), 4, "HeadRatio"),
    (("layers", 0, "mixer", "vdim"), 16, "UnsupportedOption"),
    (("layers", 1, "type"), "recurrent", "UnsupportedOption"),
    (("layers", 0, "mlp", "kind"), "wide", "UnsupportedOption"),
    (("layers", 0, "mlp", "limit"), 0.0, "ConfigJson"),
    (("layers", 0, "mixer", "mask", "size"), 0, "ConfigJson"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "ConfigJson"),
    (("layers", 1, "mlp", "router", "top"), 5, "ConfigJson"),
    (("layers", 1, "mlp", "router", "groups", "count"), 3, "ConfigJson"),
    (("layers", 1, "mlp", "router", "identity"), 1, "ConfigJson"),
    (("streams",), 17, "UnsupportedOption"),
    (("streams",), None, "ConfigJson"),
    (("norm",), None, "ConfigJson"),
    (("layers",), [], "ConfigJson"),
])
def test_config_refusals(path, value, error):
    from foundry_b200.config import errors
    from foundry_b200.config.nemasun import NemasunConfig
    doc = json.loads(json.dumps(tiny.CONFIGS["mixed"]))
    at = doc
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(getattr(errors, error)):
        NemasunConfig.parse(doc)


def test_a_table_too_long_for_its_last_distance_is_refused():
    from foundry_b200.config import errors
    from foundry_b200.config.nemasun import NemasunConfig, complete_from_files
    cfg = NemasunConfig.parse(tiny.CONFIGS["mixed"])
    with pytest.raises(errors.ConfigJson):
        complete_from_files(cfg, Files({"l1.mix.rel": (18, 4)}))  # last distance 9


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_tensor_list_and_the_model_as_data(name):
    from foundry_b200.cache import KVRequest
    from foundry_b200.engine.model import Model, expected_tensors
    from foundry_b200.models.nemasun import build_nemasun_spec
    doc = tiny.CONFIGS[name]
    spec = build_nemasun_spec(parsed(name))
    listed = {k: tuple(v.shape) for k, v in expected_tensors(spec).items()}
    assert listed == tiny.tensor_shapes(doc, tiny.BIAS_ROWS[name])
    assert spec.streams == doc["streams"]
    model = Model(spec, torch.bfloat16, torch.device("meta"))
    assert model.replay_safe()
    for block, entry in zip(model.blocks, doc["layers"]):
        m = entry["mixer"]
        assert block.cache_request() == KVRequest(m["kv_heads"], m["dim"], None, 0, row_scales=True)


def test_weights_of_a_part_that_is_not_there_may_lie_in_the_file():
    from foundry_b200.models.nemasun import build_nemasun_spec
    patterns = build_nemasun_spec(parsed("mixed")).ignorable_tensors
    hit = lambda n: any(fnmatch.fnmatch(n, p) for p in patterns)
    assert hit("l2.norm2") and hit("l2.hc2.mix")
    assert not hit("l0.norm2") and not hit("l2.hc1.mix") and not hit("l2.norm1")


@pytest.mark.parametrize("rows, last", [(16, 40), (8, 9), (30, 128), (32, 130), (20, 11), (6, 300),
                                        (2, 5), (64, 4096), (24, 70)])
def test_distance_buckets(rows, last):
    from foundry_b200.parts.shared_row_attention import distance_buckets
    got = distance_buckets(rows, last)
    assert got == [plain.distance_bucket(n, rows, last) for n in range(last + 1)]
    assert all(0 <= b - a for a, b in zip(got, got[1:])) and got[-1] == rows - 1
    assert plain.distance_bucket(10 * last, rows, last) == rows - 1


def test_distance_buckets_at_whole_powers():
    """Where the logarithms' quotient is a whole number the floor is that number: 10 single
    distances, then steps at 10 * 32^(k / 10), whole at k = 2, 4, 6 and 8."""
    from foundry_b200.parts.shared_row_attention import distance_buckets
    got = distance_buckets(20, 320)
    for k in (2, 4, 6, 8):
        n = 10 * 2 ** (k // 2)
        assert (got[n - 1], got[n]) == (10 + k - 1, 10 + k)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_rows_with_numbers_beside_them(dtype):
    """Rows and numbers of a page share a block and do not overlap."""
    from foundry_b200.cache import KVRequest, SequenceCache
    from foundry_b200.cache.pages import PAGE
    want = KVRequest(3, 10, None, 0, row_scales=True)
    cache = SequenceCache({0: want, 1: want}, 4 * PAGE, 2, dtype, torch.device("cpu"))
    a, b = cache.view(0, True), cache.view(1, True)
    assert a.k.shape == (4, 3, PAGE, 10) and a.v.data_ptr() == a.k.data_ptr()
    assert a.row_scales.shape == (4, 3, PAGE) and a.row_scales.dtype == torch.float32
    assert a.k.stride()[2:] == (10, 1) and a.row_scales.stride(2) == 1
    a.k.fill_(2.0)
    a.row_scales.copy_(torch.arange(4 * 3 * PAGE, dtype=torch.float32).view(4, 3, PAGE))
    assert bool((a.k == 2.0).all()) and not b.k.any() and not b.row_scales.any()
    assert torch.equal(a.row_scales.reshape(-1), torch.arange(4 * 3 * PAGE, dtype=torch.float32))
    size = torch.empty((), dtype=dtype).element_size()
    assert cache.bytes_per_token() == 2 * 3 * (10 * size + 4)


def test_row_scales_need_rows_that_are_keys_and_values():
    from foundry_b200.cache import KVRequest, SequenceCache
    with pytest.raises(ValueError):
        SequenceCache({0: KVRequest(1, 8, None, 8, row_scales=True)}, 64, 1, torch.float32,
                      torch.device("cpu"))


# ------------------------------------------------------ the plain implementation by hand
def test_plain_mask():
    mask = {"size": 3, "keep_first": 2}
    assert [j for j in range(9) if plain.visible(7, j, mask)] == [0, 1, 5, 6, 7]
    assert [j for j in range(9) if plain.visible(2, j, mask)] == [0, 1, 2]
    assert [j for j in range(9) if plain.visible(4, j, None)] == [0, 1, 2, 3, 4]


def test_plain_attention_by_hand():
    """One head of two elements, no window: the values are the keys before their norm, the
    bias goes by the distance and is not scaled, the gate multiplies the output."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.5, "bias_max": 3}
    eye = torch.eye(2, dtype=F)
    w = {"a.q": eye, "a.k": eye, "a.g": torch.zeros(2, 2, dtype=F), "a.o": eye,
         "a.q.norm": torch.tensor([2.0, 1.0], dtype=F), "a.k.norm": torch.tensor([1.0, 3.0], dtype=F),
         "a.rel": torch.tensor([[0.7], [-0.2], [0.1], [9.0]], dtype=F)}
    h = torch.tensor([[0.0, 6.0], [4.0, 0.0]], dtype=F)
    out = plain.attention(m, w, "a", h, 1e-13)
    # token 1: query sqrt(2) (2, 0); keys sqrt(2) (0, 3) and sqrt(2) (1, 0)
    s0, s1 = 0.0 - 0.2, 0.5 * 2.0 * 2.0 + 0.7
    p0 = 1.0 / (1.0 + math.exp(s1 - s0))
    assert abs(float(out[1, 0]) - 0.5 * 4.0 * (1.0 - p0)) < 1e-9
    assert abs(float(out[1, 1]) - 0.5 * 6.0 * p0) < 1e-9


def test_plain_dense_by_hand():
    w = {"a.gate": torch.tensor([[1.0], [1.0]], dtype=F), "a.up": torch.tensor([[1.0], [-1.0]], dtype=F),
         "a.gate.b": torch.tensor([0.0, -8.0], dtype=F), "a.up.b": torch.tensor([0.5, 0.0], dtype=F),
         "a.down": torch.tensor([[1.0, 0.0]], dtype=F), "a.down.b": torch.tensor([0.25], dtype=F)}
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))
    y = plain.dense({"limit": 2.0}, w, "a", torch.tensor([[5.0]], dtype=F))
    assert abs(float(y) - (2.0 * sig(3.404) * (2.0 + 1.0) + 0.25)) < 1e-12  # both halves clamped
    w["a.down"] = torch.tensor([[0.0, 1.0]], dtype=F)
    y = plain.dense({"limit": 2.0}, w, "a", torch.tensor([[5.0]], dtype=F))
    # gate -3 has no lower limit; up -5 is clamped to -2
    assert abs(float(y) - (-3.0 * sig(-3.0 * 1.702) * (-2.0 + 1.0) + 0.25)) < 1e-12


def test_plain_choice_by_hand():
    """A group counts by its best choice score; scores below zero in a kept group go in front
    of scores of a group that is closed; the weights are shares of the scores alone."""
    z = torch.log(torch.tensor([0.3, 0.1, 0.2, 0.15, 0.05, 0.2], dtype=F))
    correction = torch.tensor([-1.0, -2.0, -0.5, -0.6, -0.1, -3.0], dtype=F)
    router = {"top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, weights = plain.choose(z, correction, router)  # the groups' scores: -0.7, -0.3, -0.05
    assert chosen == [4, 5]
    assert [round(x, 12) for x in weights] == [0.2, 0.8]
    chosen, weights = plain.choose(z, correction, {"top": 2})
    assert chosen == [4, 2] and abs(weights[1] - 0.8) < 1e-12


def test_plain_streams_by_hand():
    """Two streams: what is read, and all new streams from the old ones."""
    w = {"a.in": torch.tensor([1.0, 2.0], dtype=F), "a.out": torch.tensor([10.0, 100.0], dtype=F),
         "a.mix": torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F)}
    xs = torch.tensor([[[1.0]], [[5.0]]], dtype=F)
    seen = []
    new = plain.connect(w, "a", xs, lambda u: seen.append(float(u)) or u * 0 + 0.5)
    assert seen == [11.0]
    # from 1 to 1 and from 2 to 1; from 1 to 2 and from 2 to 2
    assert new[:, 0, 0].tolist() == [1.0 + 15.0 + 5.0, 2.0 + 20.0 + 50.0]


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_plain_model_is_causal(name):
    cfg, w = tiny.CONFIGS[name], tiny.named_weights(name)
    tokens = torch.randint(0, cfg["vocab"], (27,), generator=torch.Generator().manual_seed(4)).tolist()
    streams = []
    full = plain.forward(cfg, w, tokens, streams)
    assert len(streams) == len(cfg["layers"]) and full.shape == (27, cfg["vocab"])
    assert float((full[:12] - plain.forward(cfg, w, tokens[:12])).abs().max()) < 1e-9
