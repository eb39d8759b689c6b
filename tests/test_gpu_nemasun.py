"""Nemasun on the GPU against the plain implementation (tests/plain_nemasun.py): every
mechanism alone, then whole models in every cutting of the same tokens (whole prompts, token
by token, portions down to two tokens, mixed batches), slots and pages that are used again,
keys far back, at the borders of cache pages, on both sides of every window's edge and of the
kept first tokens, long decoding, and greedy generation through the engine's own loop and the
command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nemasun_tiny as tiny
import plain_nemasun as plain

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
ROOT = os.path.normpath(os.path.join(os.path.dirname(os.path.abspath(__file__)), ".."))
DTYPES = [torch.float32, torch.bfloat16]


def rel_error(got, want):
    """Largest row error: rms of the difference over rms of the wanted values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    scale = max(np.sqrt((want ** 2).mean()), 1e-12)
    return float(np.sqrt(((got - want) ** 2).mean(-1)).max() / scale)


def bound(dtype, loose=1.0):
    return (3e-5 if dtype in (torch.float32, "float32") else 4e-2) * loose


def double(weights):
    return {k: v.double() for k, v in weights.items()}


def loader(weights, dtype):
    return lambda n: weights[n].to(DEV).to(dtype if weights[n].dim() > 1 else torch.float32)


def spec_of(mixer, mlp, W, eps, rows, streams=2):
    """The description of a model of one such layer, as the architecture makes it."""
    from foundry_b200.config.registry import resolve_architecture
    doc = {"architecture": "Nemasun", "vocab": 8, "width": W, "streams": streams,
           "norm": {"eps": eps},
           "layers": [{"type": "attention", "mixer": dict(mixer, bias_rows=rows), "mlp": mlp}]}
    arch = resolve_architecture(doc)
    return arch.build_spec(arch.parse_config(doc)).layers[0]


def mixer_part(m, W, eps, rows, weights, dtype, prefix="a"):
    from foundry_b200.parts import MIXERS
    part = MIXERS.build(spec_of(m, None, W, eps, rows).mixer, dtype=dtype, device=DEV)
    assert set(part.expected_tensors(prefix)) == set(weights)
    part.load(prefix, loader(weights, dtype))
    return part


def mlp_part(mlp, W, weights, dtype, prefix="a"):
    from foundry_b200.parts import FEED_FORWARDS
    m = {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 1.0, "bias_max": 9}
    part = FEED_FORWARDS.build(spec_of(m, mlp, W, 1e-5, 8).feed_forward, dtype=dtype, device=DEV)
    assert set(part.expected_tensors(prefix)) == set(weights)
    part.load(prefix, loader(weights, dtype))
    return part


def rows_of(y):
    from foundry_b200.kernels import ops
    return y.sum(torch.float32) if isinstance(y, ops.Planes) else y


def make_ctx(cache, slots, counts, vocab=1000):
    from foundry_b200.engine import SequenceStep, build_context
    return build_context(cache, [SequenceStep(s, [0] * n, []) for s, n in zip(slots, counts)],
                         vocab, DEV)


def new_cache(part, tokens, slots, dtype):
    from foundry_b200.cache import SequenceCache
    return SequenceCache({0: part.cache_request()}, tokens, slots, dtype, DEV)


def run_mixer(part, cache, xs, cuts, dtype):
    """Feed the sequences `xs` through the mixer in rounds (`cuts[k]`: the rows sequence k
    brings round by round); every sequence's outputs in order."""
    slots = [cache.open_sequence() for _ in xs]
    pieces, done = [[] for _ in xs], [0] * len(xs)
    for step in range(max(len(c) for c in cuts)):
        live = [k for k in range(len(xs)) if step < len(cuts[k])]
        counts = [cuts[k][step] for k in live]
        x = torch.cat([xs[k][done[k]:done[k] + c] for k, c in zip(live, counts)]).to(DEV).to(dtype)
        out = rows_of(part.forward(make_ctx(cache, [slots[k] for k in live], counts), x,
                                   cache.view(0, True)))
        for k, rows in zip(live, torch.split(out, counts)):
            pieces[k].append(rows.float().cpu())
            done[k] += rows.shape[0]
    for s in slots:
        cache.close_sequence(s)
    return [torch.cat(p) for p in pieces]


def counted(fn):
    """(fn's result, launches of this library's kernels by name while it ran)."""
    from foundry_b200.kernels import ops
    ops.PROFILER.start("steps")
    try:
        out = fn()
        taken = ops.PROFILER.take()["kernels"]
    finally:
        ops.PROFILER.start(None)
    counts = {}
    for key, entry in taken.items():
        kind = key.split(" ")[0]
        counts[kind] = counts.get(kind, 0) + entry["dispatch_count"]
    return out, counts


# ------------------------------------------------------------------- attention alone
OTHER_SIZES = [
    # (heads, key heads, size, window, kept, table rows, last distance)
    (4, 1, 64, 64, 1, 32, 128),
    (2, 2, 128, 128, 0, 20, 11),
    (8, 2, 32, 77, 65, 16, 40),
    (3, 1, 72, None, 0, 30, 1000),
    (16, 1, 128, 200, 64, 26, 110),
    (20, 1, 16, 1, 3, 8, 9),
    (2, 1, 264, 90, 5, 12, 50),
    (5, 5, 13, 65, 128, 24, 70),
    (32, 4, 64, 1000, 4, 64, 4096),
    (6, 3, 104, 80, 7, 28, 90),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", OTHER_SIZES, ids=lambda s: "-".join(map(str, s)))
def test_attention_in_two_cuttings(sizes, dtype):
    """Unequal sequences in one step, then on the slots and pages that were just given back
    the same rows as prompt parts, portions of two tokens and single tokens."""
    H, G, d, window, kept, rows, last = sizes
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 1.5 / d ** 0.5, "bias_max": last}
    if window:
        m["mask"] = {"size": window, "keep_first": kept}
    W, eps = 64, 1e-5
    weights = tiny.random_weights(tiny.mixer_shapes("a", m, W, rows), seed=d + H)
    part = mixer_part(m, W, eps, rows, weights, dtype)
    cache = new_cache(part, 1536, 4, dtype)
    torch.manual_seed(d)
    xs = [torch.randn(n, W).to(dtype).float() for n in (333, 6, 129)]
    want = [plain.attention(m, double(weights), "a", x.double(), eps) for x in xs]
    for cuts in ([[333], [6], [129]], [[70, 2, 1, 1, 200, 58, 1], [3, 2, 1], [64, 65]],
                 [[300] + [1] * 33, [1] * 6, [100] + [1] * 29]):
        got = run_mixer(part, cache, xs, cuts, dtype)
        for g, w in zip(got, want):
            assert rel_error(g, w) < bound(dtype), (sizes, cuts)


@pytest.mark.parametrize("last", [33, 110, 2000, 9000])
@pytest.mark.parametrize("mask", [(37, 0), (64, 64), (150, 5), (300, 130), (1000, 1), (None, 0)])
@pytest.mark.parametrize("sizes", [(64, 4, 2), (128, 2, 1), (88, 3, 1), (40, 2, 2)])
def test_prompts_and_single_tokens_on_the_tensor_cores(sizes, mask, last):
    """bfloat16 steps on the tensor cores against the CUDA-core kernel on the same rows:
    windows that end inside a block of queries and inside a page, kept tokens of less and more
    than a page, distance tables that fit shared memory and one that does not, portions that
    begin in the middle of a page; and the kernels counted, so that nothing stands in."""
    from foundry_b200.kernels import ops
    d, heads, kv_heads = sizes
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": d, "scale": d ** -0.5,
         "bias_max": last}
    if mask[0]:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    W, eps = 64, 1e-5
    weights = tiny.random_weights(tiny.mixer_shapes("a", m, W, 32), seed=d)
    part = mixer_part(m, W, eps, 32, weights, torch.bfloat16)
    cache = new_cache(part, 2048, 3, torch.bfloat16)
    torch.manual_seed(d)
    xs = [torch.randn(n, W).to(torch.bfloat16).float() for n in (533, 70, 129)]
    results = {}
    for tc in (True, False):
        ops.SHARED_ROWS_TC = tc
        try:
            for cuts in ([[533], [70], [129]], [[100, 133, 2, 297, 1], [5, 63, 1, 1], [64, 65]],
                         [[520] + [1] * 13, [60] + [1] * 10, [116] + [1] * 13]):
                got, counts = counted(lambda: run_mixer(part, cache, xs, cuts, torch.bfloat16))
                assert (counts.get("attention_prefill_shared", 0) > 0) == tc, counts
                assert (counts.get("attention_decode_shared", 0) > 0) == (
                    tc and d in ops.FAST_HEAD_DIMS and len(cuts[0]) > 1), counts
                results[tc, len(cuts[0])] = got
        finally:
            ops.SHARED_ROWS_TC = True
    for cut in (1, 5, 14):
        for g, w in zip(results[True, cut], results[False, cut]):
            assert rel_error(g, w) < 0.75 * bound(torch.bfloat16), cut


def crafted_attention(W, d, window, kept, heads, kv_heads):
    """An attention made so that a query that carries input 1 matches only a key that carries
    input 2: that score is about 20, every other key's about +-1. Keys are values, so what
    marks a key also tells it from the others in the output. The distance table is flat but
    for its first and last rows."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": d, "scale": 20.0 / d,
         "bias_max": 30, "mask": {"size": window, "keep_first": kept} if window else None}
    q, k = torch.zeros(heads * d, W), torch.zeros(kv_heads * d, W)
    for h in range(heads):
        q[h * d, 1] = 1.0
    for g in range(kv_heads):
        k[g * d, 2] = 1.0       # a marker's key points along element 0
        k[g * d + 1, 0] = 1.0   # an ordinary one along element 1
    out = torch.zeros(W, heads * d)  # the mean over the heads
    n = min(W, d)
    for h in range(heads):
        out[:n, h * d:h * d + n] += torch.eye(n) / heads
    rel = torch.zeros(8, heads)
    rel[0], rel[7] = 0.5, -1.0
    return m, {"a.q": q, "a.k": k, "a.g": torch.zeros(heads * d, W), "a.rel": rel,
               "a.o": out.to(torch.bfloat16).float(), "a.q.norm": torch.ones(d),
               "a.k.norm": torch.ones(d)}


def marked_inputs(query_at, marker_at, width, behind=0):
    """Rows in which only the query of `query_at` (input 1) and the key of `marker_at`
    (input 2) match; ordinary rows carry input 0."""
    gen = torch.Generator().manual_seed(query_at * 1000 + marker_at)
    x = torch.zeros(query_at + 1 + behind, width)
    x[:, 0] = 1.0
    x += 0.05 * torch.randn(x.shape, generator=gen)
    x[query_at] = 0.05 * torch.randn(width, generator=gen)
    x[query_at, 0] += 1.0
    x[query_at, 1] = 1.0
    if marker_at != query_at:
        x[marker_at] = 0.05 * torch.randn(width, generator=gen)
    x[marker_at, 2] = 3.0
    return x.to(torch.bfloat16).float()


def places(window, kept):
    """(query, marker, visible): the window's first key and the key in front of it, the last
    kept token and the one behind it, the first token, the query itself and its neighbour."""
    out = []
    for q in (2, 63, 64, 130, 300):
        lo = max(0, q - window + 1) if window else 0
        seen = {lo, q, max(lo, q - 1)} | ({0, min(kept, q + 1) - 1} if kept else set())
        hidden = {lo - 1, kept, max(kept, lo - 64)} if kept < lo else set()
        out += [(q, j, True) for j in sorted(seen)]
        out += [(q, j, False) for j in sorted(hidden) if kept <= j < lo]
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mask", [(1, 0), (64, 1), (65, 70), (200, 3), (None, 0)])
@pytest.mark.parametrize("sizes", [(8, 1, 1), (64, 2, 1), (128, 4, 1), (40, 20, 1), (16, 2, 2)])
def test_one_key_that_stands_out_on_both_sides_of_every_edge(sizes, mask, dtype):
    """The key that dominates a query lies just inside or just outside the query's window or
    the kept first tokens, at the sequence's first token, hundreds of tokens back, or is the
    query's own; the query is the last token of a prompt, stands in front of others in its
    portion, or is decoded alone."""
    d, heads, kv_heads = sizes
    W = 16
    m, weights = crafted_attention(W, d, *mask, heads, kv_heads)
    part = mixer_part(m, W, 1e-6, 8, weights, dtype)
    cache = new_cache(part, 1024, 2, dtype)
    wd = double(weights)
    for query_at, marker_at, visible in places(*mask):
        x = marked_inputs(query_at, marker_at, W, behind=3)
        want = plain.attention(m, wd, "a", x[:query_at + 1].double(), 1e-6)[-1]
        # the plain implementation itself sees the marker where it should and only there
        assert (float(want[0]) > 0.75) == visible, (query_at, marker_at, float(want[0]))
        for cut in ([query_at + 1, 3], [query_at, 1, 3], [query_at - 1, 5]):
            got = run_mixer(part, cache, [x], [cut], dtype)[0][query_at].double()
            err = float((got - want).norm()) / max(float(want.norm()), 1.0)
            assert err < bound(dtype, 3.0), (query_at, marker_at, visible, cut, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [16, 64, 128])
def test_every_distance_takes_its_own_row(d, dtype):
    """Queries and keys that match equally everywhere, so that the weights are the table's
    alone; every row of the table is unlike its neighbours, and the last distance lies within
    the sequence."""
    m = {"heads": 2, "kv_heads": 1, "dim": d, "vdim": d, "scale": 0.01, "bias_max": 90}
    W, rows = 32, 16
    weights = tiny.random_weights(tiny.mixer_shapes("a", m, W, rows), seed=d)
    weights["a.rel"] = (3.0 * torch.randn(rows, 2, generator=torch.Generator().manual_seed(1))
                        ).to(torch.bfloat16).float()
    part = mixer_part(m, W, 1e-5, rows, weights, dtype)
    cache = new_cache(part, 1024, 2, dtype)
    torch.manual_seed(2)
    xs = [torch.randn(n, W).to(dtype).float() for n in (200, 95)]
    want = [plain.attention(m, double(weights), "a", x.double(), 1e-5) for x in xs]
    for cuts in ([[200], [95]], [[150] + [1] * 50, [2, 93]]):
        for g, w in zip(run_mixer(part, cache, xs, cuts, dtype), want):
            assert rel_error(g, w) < bound(dtype), cuts


# ----------------------------------------------------------------- feed-forwards alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(64, 40, 0.5), (80, 104, 1.0), (256, 512, 7.0), (36, 20, 0.1),
                                   (52, 18, 2.0), (512, 640, 0.9)])
def test_clamped_feed_forward(sizes, dtype):
    """From one token to prompts, with inputs large enough that both clamps are met on both
    sides; the bias behind it added here and handed out."""
    W, ff, limit = sizes
    mlp = {"kind": "dense", "ff": ff, "limit": limit}
    weights = tiny.random_weights(tiny.mlp_shapes("a", mlp, W), seed=ff)
    part = mlp_part(mlp, W, weights, dtype)
    torch.manual_seed(ff)
    for T in (1, 7, 16, 40, 130, 300):
        x = (2.0 * torch.randn(T, W)).to(dtype).float()
        want = plain.dense(mlp, double(weights), "a", x.double())
        got = rows_of(part.forward(None, x.to(DEV).to(dtype)))
        assert rel_error(got.float().cpu(), want) < bound(dtype), T
        y, bias = part.forward(None, x.to(DEV).to(dtype), defer_bias=True)
        assert rel_error((rows_of(y).float() + bias).cpu(), want) < bound(dtype), T


MOE = [(64, 32, 9, 3, 4, (2, 1), 120), (80, 56, 6, 2, 3, (4, 2), 40), (36, 12, 4, 4, 4, None, None),
       (128, 64, 12, 0, 5, (3, 2), 64), (256, 96, 100, 28, 8, (16, 4), 96), (64, 64, 1, 1, 1, None, None),
       (64, 30, 5, 1, 2, (6, 5), None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", MOE, ids=lambda s: "-".join(map(str, s)))
def test_routed_experts(sizes, dtype):
    """Against the plain choice, token by token, from one token to prompts. Tokens whose
    choice hangs on less than a rounding are left out (they are few)."""
    W, ff, experts, identity, top, groups, shared = sizes
    mlp = tiny._moe(ff, experts, top, identity, groups, shared)
    weights = tiny.random_weights(tiny.mlp_shapes("a", mlp, W), seed=experts + top)
    part = mlp_part(mlp, W, weights, dtype)
    wd = double(weights)
    torch.manual_seed(experts)
    for T in (1, 5, 40, 200):
        x = torch.randn(T, W).to(torch.bfloat16).float()
        want = plain.routed(mlp, wd, "a", x.double())
        got = rows_of(part.forward(None, x.to(DEV).to(dtype))).float().cpu()
        nudged = [plain.choose(z, wd["a.correction"] + s * 1e-5 * torch.randn(
            experts + identity, dtype=plain.F), mlp["router"])[0]
            for z in x.double() @ wd["a.router"].T for s in (0.0, 1.0, 1.0)]
        sure = [t for t in range(T) if len({tuple(sorted(c)) for c in nudged[3 * t:3 * t + 3]}) == 1]
        assert len(sure) >= 0.95 * T
        assert rel_error(got[sure], want[sure]) < bound(dtype), T


@pytest.mark.parametrize("correction", [[0.0] * 6, [-3.0, -3.0, -3.0, -1.0, -1.0, -1.0],
                                        [-1.0, -9.0, -9.0, -0.5, -9.0, -9.0]])
@pytest.mark.parametrize("T", [3, 100])
def test_choice_of_experts_one_by_one(correction, T):
    """The chosen experts and their weights themselves: groups by their best choice score (also
    where all are below zero), weights without the correction, identity experts chosen."""
    from foundry_b200.kernels import ops
    torch.manual_seed(T)
    z = (2.0 * torch.randn(T, 6)).to(DEV)
    c = torch.tensor(correction)
    for router in ({"top": 2, "groups": {"count": 2, "keep": 1}}, {"top": 3}, {"top": 2, "groups": {"count": 3, "keep": 2}}):
        chosen = torch.empty((T, router["top"]), dtype=torch.int32, device=DEV)
        weights = torch.empty((T, router["top"]), dtype=torch.float32, device=DEV)
        g = router.get("groups", {"count": 1, "keep": 1})
        order = ops.moe_route_sorted(z, None, router["top"], chosen, weights, score="softmax",
                                     groups=g["count"], keep=g["keep"], correction=c.to(DEV),
                                     normalise=True, sum_floor=1e-20, group_best=1, experts=4)
        kept = 0
        for t in range(T):
            want, shares = plain.choose(z[t].double().cpu(), c.double(), router)
            assert chosen[t].tolist() == want
            assert np.allclose(weights[t].tolist(), shares, rtol=1e-5)
            assert [p >= 0 for p in order.place[t].tolist()] == [e < 4 for e in want]
            kept += sum(e < 4 for e in want)
        assert int(order.starts[-1]) == kept and order.starts.numel() == 5


# ----------------------------------------------------------------------- the streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W, S", [(64, 1), (256, 2), (80, 3), (2048, 4), (37, 5), (3072, 2), (100, 16),
                                  (8192, 3), (9000, 2)])
def test_streams_mixed_in_the_norms_pass(W, S, dtype):
    """Two results after one another, from one row that all streams are equal to up to the
    sum at the end: rows in both types, split-K planes, with and without a bias."""
    from foundry_b200.kernels import ops
    from foundry_b200.parts import NORMS
    from foundry_b200.config.spec import PartSpec
    g = torch.Generator().manual_seed(W + S)
    r = lambda *s: torch.randn(*s, generator=g)
    T, eps = 5, 1e-5
    norm = NORMS.build(PartSpec("rms_norm", {"size": W, "eps": eps, "weight_suffix": ""}), dtype=dtype,
                       device=DEV)
    w = 1.0 + 0.2 * r(W)
    norm.load("n", lambda n: w.to(DEV))
    x0, ins, mix, share, bias = r(T, W), r(3, S), r(2, S, S), r(2, S), r(W)
    planes = r(3, T, W)
    rows = r(T, W).to(dtype).float()
    to = lambda t: t.to(DEV).contiguous()
    streams = ops.Streams(S, first=to(x0))
    out = [norm.add_norm(streams.read(to(ins[0])), None)]
    out.append(norm.add_norm(streams.read(to(ins[1])),
                             ops.StreamDelta(ops.Planes(to(planes)), to(mix[0]), to(share[0]), to(bias))))
    last = ops.StreamDelta(rows.to(DEV).to(dtype), to(mix[1]), to(share[1]))
    some = torch.tensor([4, 1], dtype=torch.int32, device=DEV)
    end = norm.add_norm(streams.take(some, 2).read(None), last.take(some, 2))
    out.append(norm.add_norm(streams.read(to(ins[2])), last))
    xs = torch.stack([x0.double()] * S)
    weights = {"a.mix": mix[0].double(), "a.out": share[0].double(), "a.in": ins[1].double(),
               "b.mix": mix[1].double(), "b.out": share[1].double(), "b.in": ins[2].double()}
    read = lambda i: plain.rms_norm(torch.einsum("s,stw->tw", ins[i].double(), xs), w.double(), eps)
    want = [read(0)]
    xs = plain.connect(weights, "a", xs, lambda u: planes.double().sum(0) + bias.double())
    want.append(read(1))
    xs = plain.connect(weights, "b", xs, lambda u: rows.double())
    want.append(read(2))
    for got, ref in zip(out, want):
        assert rel_error(got.float().cpu(), ref) < bound(dtype, 0.3)
    assert rel_error(streams.values.permute(1, 0, 2).cpu(), xs) < 1e-5
    ref = plain.rms_norm(xs.sum(0), w.double(), eps)[[4, 1]]
    assert rel_error(end.float().cpu(), ref) < bound(dtype, 0.3)


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("nemasun")
    return {name: tiny.write_folder(str(root / name), name) for name in tiny.CONFIGS}


def plain_logits(name, weights, tokens):
    return plain.forward(tiny.CONFIGS[name], double(weights), tokens).numpy()


def run_cutting(engine, prompts, cuts):
    """Feed `prompts` through `engine.step` in rounds; `cuts[k]` are the token
    counts sequence k brings round by round. Logits of every position."""
    from foundry_b200.engine import SequenceStep
    slots = [engine.open_sequence() for _ in prompts]
    done = [0] * len(prompts)
    rows = [[] for _ in prompts]
    for r in range(max(len(c) for c in cuts)):
        live = [k for k in range(len(prompts)) if r < len(cuts[k])]
        steps = [SequenceStep(slots[k], prompts[k][done[k]:done[k] + cuts[k][r]],
                              list(range(cuts[k][r]))) for k in live]
        logits = engine.step(steps).cpu().numpy()
        at = 0
        for k in live:
            n = cuts[k][r]
            rows[k].append(logits[at:at + n])
            at += n
            done[k] += n
            if done[k] == len(prompts[k]):
                engine.close_sequence(slots[k])
    assert done == [len(p) for p in prompts]
    return [np.concatenate(r) for r in rows]


def close_calls(doc, weights, tokens, gap):
    """Positions at which some layer's choice of experts hangs on less than `gap`: rounding may
    turn it, and every later position that attends to them may differ a little."""
    w = {k: v.double() for k, v in weights.items()}
    out = set()
    original = plain.choose

    def spy(z, correction, router):
        chosen, shares = original(z, correction, router)
        spy.at += 1
        torch.manual_seed(spy.at)
        for _ in range(3):
            again = original(z, correction + gap * torch.randn(z.shape, dtype=plain.F), router)[0]
            if sorted(again) != sorted(chosen):
                out.add((spy.at - 1) % len(tokens))
        return chosen, shares
    spy.at = 0
    plain.choose = spy
    try:
        logits = plain.forward(doc, w, tokens)
    finally:
        plain.choose = original
    return logits.numpy(), sorted(out)


def most_rows(got, want, unsure, dtype, loose):
    """Rows whose choices are sure must be right; in bfloat16 a turned choice also moves what
    later tokens read a little, so nearly all of them."""
    sure = [t for t in range(len(want)) if t not in unsure]
    scale = np.sqrt((np.asarray(want) ** 2).mean())
    assert np.isfinite(got).all()
    err = np.sqrt(((np.asarray(got) - want) ** 2).mean(-1)) / scale
    if dtype == "float32":
        return float(err[sure].max()) < bound(dtype, loose) if sure else True
    return float((err[sure] > bound(dtype, loose)).mean()) < 0.04 if sure else True


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_model_in_every_cutting(name, dtype, folders):
    """Whole prompts alone; token by token from the first token on; portions of several sizes
    down to two tokens; a batch of unequal requests decoded together while the shorter ones
    end; all on slots and pages that the earlier cuttings used and gave back."""
    import foundry_b200 as fb
    folder, weights = folders[name]
    doc = tiny.CONFIGS[name]
    rng = np.random.default_rng(11)
    prompts = [[int(t) for t in rng.integers(0, doc["vocab"], n)] for n in (310, 1, 3, 81)]
    gap = 1e-6 if dtype == "float32" else 4e-3
    want = [close_calls(doc, weights, p, gap) for p in prompts]
    engine = fb.Engine.from_folder(folder, dtype=dtype, max_tokens=1024, max_slots=6)
    results = {}
    results["whole, alone"] = [run_cutting(engine, [p], [[len(p)]])[0] for p in prompts]
    results["token by token"] = [run_cutting(engine, [prompts[k]], [[1] * len(prompts[k])])[0]
                                 for k in (2, 3)]
    results["portions"] = run_cutting(engine, [prompts[0], prompts[3]],
                                      [[2, 62, 1, 64, 2, 177, 2], [77, 2, 2]])
    results["batch, then decoded together"] = run_cutting(
        engine, prompts, [[280] + [1] * 30, [1], [2, 1], [70] + [1] * 11])
    wanted = {"whole, alone": want, "token by token": [want[2], want[3]],
              "portions": [want[0], want[3]], "batch, then decoded together": want}
    for cutting, got in results.items():
        for g, (w, unsure) in zip(got, wanted[cutting]):
            assert most_rows(g, w, unsure, dtype, 3.0), (name, dtype, cutting, len(w))
    engine.cache.table.check()
    assert engine.free_slots() == 6


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_long_decoding_and_reused_slots(name, folders):
    """260 tokens decoded one by one behind a short prompt (across cache pages and far beyond
    every window), twice on the same slot with another sequence between."""
    import foundry_b200 as fb
    folder, weights = folders[name]
    doc = tiny.CONFIGS[name]
    rng = np.random.default_rng(12)
    tokens = [int(t) for t in rng.integers(0, doc["vocab"], 265)]
    other = [int(t) for t in rng.integers(0, doc["vocab"], 40)]
    want, unsure = close_calls(doc, weights, tokens, 1e-6)
    engine = fb.Engine.from_folder(folder, dtype="float32", max_tokens=512, max_slots=2)
    first = run_cutting(engine, [tokens], [[5] + [1] * 260])[0]
    run_cutting(engine, [other], [[40]])
    again = run_cutting(engine, [tokens], [[5] + [1] * 260])[0]
    assert most_rows(first, want, unsure, "float32", 2.0)
    assert np.array_equal(first, again)


def test_sizes_that_fit_no_tensor_core_product(tmp_path):
    """Width 50 and inner sizes that are no multiples of 8 (in bfloat16 every product takes the
    CUDA-core kernel); the layer without a feed-forward last, so that a mixer's result meets
    the final norm; every layer with sizes, window and table of its own."""
    import foundry_b200 as fb
    base = {"heads": 3, "kv_heads": 3, "dim": 11, "vdim": 11, "scale": 0.3, "bias_max": 33,
            "mask": {"size": 33, "keep_first": 2}}
    doc = {"architecture": "Nemasun", "vocab": 77, "width": 50, "streams": 5, "norm": {"eps": 1e-5},
           "embedding": {"scale": 7.0},
           "layers": [
               tiny._layer(dict(base, heads=2, kv_heads=1, mask={"size": 2}), tiny._moe(18, 3, 1, 1, (2, 1), 30)),
               tiny._layer(base, {"kind": "dense", "ff": 27, "limit": 0.6}), tiny._layer(base, None)]}
    weights = tiny.random_weights(tiny.tensor_shapes(doc, [4, 22, 10]), seed=31)
    folder, _ = tiny.write_model(str(tmp_path / "odd"), doc, weights)
    rng = np.random.default_rng(3)
    prompts = [[int(t) for t in rng.integers(0, 77, n)] for n in (70, 9)]
    for dtype, gap in (("float32", 1e-6), ("bfloat16", 4e-3)):
        want = [close_calls(doc, weights, p, gap) for p in prompts]
        engine = fb.Engine.from_folder(folder, dtype=dtype, max_tokens=512, max_slots=3)
        got = run_cutting(engine, prompts, [[66, 2, 1, 1], [5, 1, 2, 1]])
        for g, (w, unsure) in zip(got, want):
            assert most_rows(g, w, unsure, dtype, 3.0), dtype


WIDE = {"architecture": "Nemasun", "vocab": 320, "width": 512, "streams": 2, "norm": {"eps": 1e-5},
        "embedding": {"scale": 2.0},
        "layers": [
            tiny._layer({"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.125,
                         "bias_max": 200, "mask": {"size": 130, "keep_first": 5}},
                        {"kind": "dense", "ff": 768, "limit": 1.2}),
            tiny._layer({"heads": 4, "kv_heads": 1, "dim": 128, "vdim": 128, "scale": 0.09,
                         "bias_max": 400, "mask": {"size": 300, "keep_first": 70}},
                        {"kind": "dense", "ff": 1024, "limit": 5.0})]}


def test_wider_heads_through_the_serving_kernels(tmp_path):
    """Sizes whose bfloat16 steps take the tensor-core products and attentions in prompts, in
    replayed short prompts and in single tokens (graphs), with windows that pass over decoded
    tokens."""
    import foundry_b200 as fb
    weights = tiny.random_weights(tiny.tensor_shapes(WIDE, [32, 16]), seed=41)
    folder, _ = tiny.write_model(str(tmp_path / "wide"), WIDE, weights)
    rng = np.random.default_rng(5)
    prompts = [[int(t) for t in rng.integers(0, 320, n)] for n in (700, 150, 40)]
    want = [plain.forward(WIDE, double(weights), p).numpy() for p in prompts]
    engine = fb.Engine.from_folder(folder, dtype="bfloat16", max_tokens=2048, max_slots=4)
    for cuts in ([[700], [150], [40]], [[600, 60] + [1] * 40, [100, 2, 8] + [1] * 40, [1, 2, 3] + [1] * 34]):
        for g, w in zip(run_cutting(engine, prompts, cuts), want):
            assert rel_error(g, w) < bound("bfloat16", 1.5), (cuts[0][:3], len(w))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(dtype, folders):
    """`Engine.generate` (the scheduler's batches, graphs, slot reuse) against the plain
    model's greedy tokens; five prompts through batches of two."""
    import foundry_b200 as fb
    folder, weights = folders["mixed"]
    cfg = tiny.CONFIGS["mixed"]
    rng = np.random.default_rng(13)
    prompts = [[int(t) for t in rng.integers(0, cfg["vocab"], n)] for n in (9, 1, 30, 4, 17)]
    engine = fb.Engine.from_folder(folder, dtype=dtype, max_tokens=512, max_slots=4)
    got = engine.generate(prompts, 8, eos_token_id=[], max_batch=2).token_ids
    wd = double(weights)
    for g, p in zip(got, prompts):
        w = plain.greedy_generate(cfg, wd, p, 8)
        if g == w:
            continue
        k = next(i for i, (a, b) in enumerate(zip(g, w)) if a != b)
        logits = plain.forward(cfg, wd, list(p) + w[:k])[-1]
        gap = float(logits[w[k]] - logits[g[k]])
        assert dtype == "bfloat16" and gap < 0.1 * float(logits.abs().max()), (g, w, gap)


def test_trace_replay_and_command_line(folders, tmp_path):
    """`bin/trace_run` on a Nemasun folder: a prompt step of two requests, then single tokens,
    one request ending early; `foundry run` generating; `foundry bench` reporting."""
    folder, weights = folders["other"]
    cfg = tiny.CONFIGS["other"]
    rng = np.random.default_rng(14)
    a = [int(t) for t in rng.integers(0, cfg["vocab"], 12)]
    b = [int(t) for t in rng.integers(0, cfg["vocab"], 5)]
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": [0, 9]},
                                     {"id": "b", "tokens": b[:4], "want": [3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[10:11], "want": []},
                                     {"id": "b", "tokens": b[4:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[11:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder,
                           "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                          input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True,
                          text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = plain_logits("other", weights, a), plain_logits("other", weights, b)
    V = cfg["vocab"]
    read = lambda n: np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, V)
    assert rel_error(read(0), np.stack([wa[0], wa[9], wb[3]])) < bound("float32", 2.0)
    assert rel_error(read(1), wb[4:5]) < bound("float32", 2.0)
    assert rel_error(read(2), wa[11:12]) < bound("float32", 2.0)
    foundry = [sys.executable, os.path.join(ROOT, "bin", "foundry")]
    run = subprocess.run(foundry + ["run", "--model", folder, "--dtype", "float32", "--prompt-ids",
                                    ",".join(map(str, a)), "--max-new-tokens", "4", "--ignore-eos"],
                         capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert json.loads(run.stdout.strip().split("\n")[-1]) == plain.greedy_generate(
        cfg, double(weights), a, 4)
    run = subprocess.run(foundry + ["bench", "--model", folder, "--prompt-tokens", "20", "--new-tokens",
                                    "5", "--runs", "2", "--batch-size", "3", "--out", str(tmp_path)],
                         capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    report = json.loads((tmp_path / "report.json").read_text())
    assert len(report["runs"]) == 2 and all(len(r) == 5 for r in report["runs"][0]["token_ids"])
    assert report["runs"][0]["token_ids"] == report["runs"][1]["token_ids"]
