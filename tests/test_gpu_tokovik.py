"""Tokovik on the GPU against the plain implementation (tests/plain_tokovik.py):
every mechanism alone, then whole models in every cutting of the same tokens
(whole prompts, token by token, portions down to two tokens, mixed batches),
slots and pages that are used again, keys far back, at the borders of cache
pages and on both sides of every window's edge, states whose first token still
weighs on the last, chunked scans, long decoding, and greedy generation through
the engine's own loop and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tokovik as plain
import tokovik_tiny as tiny

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


def make_ctx(cache, slots, counts, vocab=1000):
    from foundry_b200.engine import SequenceStep, build_context
    return build_context(cache, [SequenceStep(s, [0] * n, []) for s, n in zip(slots, counts)],
                         vocab, DEV)


def spec_of(doc, ranks):
    from foundry_b200.config.registry import resolve_architecture
    doc = json.loads(json.dumps(doc))
    for layer, rank in zip(doc["layers"], ranks):
        layer["mixer"]["right"]["decay_rank"] = rank
    arch = resolve_architecture(doc)
    return arch.build_spec(arch.parse_config(doc))


def loader(weights, dtype):
    return lambda n: weights[n].to(DEV).to(dtype if weights[n].dim() > 1 else torch.float32)


def one_layer(m, W, eps, mlp=None):
    return {"architecture": "Tokovik", "vocab": 8, "width": W, "norm": {"eps": eps},
            "layers": [{"type": "parallel", "mixer": m, "mlp": mlp}]}


def mixer_part(m, W, eps, weights, dtype, rank, prefix="a", side=None):
    """The parallel mixer of the library, built the way the architecture builds it; or
    one of its sides alone (`side`: "left" or "right"; tensors under `prefix.side`)."""
    from foundry_b200.parts import MIXERS
    spec = spec_of(one_layer(m, W, eps), [rank]).layers[0].mixer
    if side is not None:
        spec, prefix = spec.params[side], f"{prefix}.{side}"
    part = MIXERS.build(spec, dtype=dtype, device=DEV)
    mine = {k for k in weights if k.startswith(prefix + ".") and (side is None or not k.endswith(".out"))}
    assert set(part.expected_tensors(prefix)) == mine
    part.load(prefix, loader(weights, dtype))
    return part


def joined(y):
    """A mixer's output as float32 rows; a pair is joined as its definition says."""
    from foundry_b200.kernels import ops
    if isinstance(y, ops.NormedPair):
        a, b = (joined(t).double() for t in (y.a, y.b))
        unit = lambda t: t / torch.sqrt((t * t).mean(-1, keepdim=True) + y.eps)
        return (y.scale * (unit(a) * y.weight_a.double() + unit(b) * y.weight_b.double())).float()
    return y.sum(torch.float32) if isinstance(y, ops.Planes) else y


def run_mixer(part, cache, xs, cuts, dtype):
    """Feed the sequences `xs` through the mixer in rounds (`cuts[k]`: the rows sequence k
    brings round by round); every sequence's outputs in order."""
    slots = [cache.open_sequence() for _ in xs]
    pieces, done = [[] for _ in xs], [0] * len(xs)
    for step in range(max(len(c) for c in cuts)):
        live = [k for k in range(len(xs)) if step < len(cuts[k])]
        counts = [cuts[k][step] for k in live]
        x = torch.cat([xs[k][done[k]:done[k] + c] for k, c in zip(live, counts)]).to(DEV).to(dtype)
        out = joined(part.forward(make_ctx(cache, [slots[k] for k in live], counts), x,
                                  cache.view(0, True)))
        for k, rows in zip(live, torch.split(out, counts)):
            pieces[k].append(rows.float().cpu())
            done[k] += rows.shape[0]
    for s in slots:
        cache.close_sequence(s)
    return [torch.cat(p) for p in pieces]


def new_cache(part, tokens, slots, dtype):
    from foundry_b200.cache import SequenceCache
    return SequenceCache({0: part.cache_request()}, tokens, slots, dtype, DEV)


PLAIN_SIDE = {"left": plain.window_attention, "right": plain.gated_linear}


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


# ------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_each_side_and_the_pair_in_two_cuttings(name, dtype):
    """Every layer's attention alone, its linear attention alone, and the pair, each with a
    cache of its own: two sequences of unequal lengths in one step, then on the slots and
    pages that were just given back the same rows as a prompt part, portions of two tokens
    and single tokens."""
    cfg, weights = tiny.CONFIGS[name], tiny.random_weights(name)
    eps, W = cfg["norm"]["eps"], cfg["width"]
    torch.manual_seed(5)
    lens = [139, 6]
    xs = [torch.randn(n, W).to(dtype).float() for n in lens]
    for i, layer in enumerate(cfg["layers"]):
        prefix, m = f"l{i}.mix", layer["mixer"]
        mine = {k: v for k, v in weights.items() if k.startswith(prefix + ".")}
        for side in ("left", "right", None):
            part = mixer_part(m, W, eps, mine, dtype, tiny.RANKS[name][i], prefix, side)
            cache = new_cache(part, 1024, 4, dtype)
            if side is None:
                want = [plain.parallel_mixer(m, double(mine), prefix, x.double(), eps) for x in xs]
            else:
                want = [PLAIN_SIDE[side](m[side], double(mine), f"{prefix}.{side}", x.double(), eps)
                        for x in xs]
            for cuts in ([[139], [6]], [[70, 2, 1, 1, 63, 2], [3, 2, 1]]):
                got = run_mixer(part, cache, xs, cuts, dtype)
                for g, w in zip(got, want):
                    assert rel_error(g, w) < bound(dtype), (name, i, side, cuts)


OTHER_SIZES = [
    # keys and values of the tensor-core kernels' sizes; windows of one page, of two, of a
    # size no page divides; one key head for all; every element rotated, none rotated
    ({"left": {"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 64, "scale": 0.125, "mask": {"size": 64},
               "rot": {"dims": 64, "base": 10000.0}},
      "right": {"heads": 1, "dim": 16, "vdim": 64, "tau": 4.0}}, 6),
    ({"left": {"heads": 2, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 0.09, "mask": {"size": 128}},
      "right": {"heads": 8, "dim": 128, "vdim": 8, "tau": 16.0}}, 16),
    ({"left": {"heads": 3, "kv_heads": 3, "dim": 32, "vdim": 64, "scale": 0.2, "mask": {"size": 77},
               "rot": {"dims": 16, "base": 77.0,
                       "scaling": {"factor": 2.0, "original": 32, "fast": 2.0, "slow": 0.3}}},
      "right": {"heads": 3, "dim": 20, "vdim": 36, "tau": 2.5}}, 7),
    # no window at all (every earlier key visible), odd sizes everywhere
    ({"left": {"heads": 5, "kv_heads": 5, "dim": 12, "vdim": 20, "scale": 0.4,
               "rot": {"dims": 2, "base": 3.0}},
      "right": {"heads": 6, "dim": 6, "vdim": 10, "tau": 1.0}}, 1),
    # a window of one position: a token sees itself only; a state wider than 256 key rows
    ({"left": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.3, "mask": {"size": 1},
               "rot": {"dims": 8, "base": 100.0}},
      "right": {"heads": 1, "dim": 300, "vdim": 33, "tau": 8.0}}, 40),
    # a window longer than every sequence of the test; keys and values of unequal sizes
    ({"left": {"heads": 8, "kv_heads": 4, "dim": 64, "vdim": 128, "scale": 0.1, "mask": {"size": 4096},
               "rot": {"dims": 16, "base": 5000.0}},
      "right": {"heads": 4, "dim": 64, "vdim": 64, "tau": 20.0}}, 32),
    # tensor-core tiles that are only partly filled, twenty query heads on one key head
    ({"left": {"heads": 20, "kv_heads": 1, "dim": 48, "vdim": 88, "scale": 0.14, "mask": {"size": 90},
               "rot": {"dims": 24, "base": 1000.0}},
      "right": {"heads": 2, "dim": 96, "vdim": 128, "tau": 10.0}}, 64),
    ({"left": {"heads": 4, "kv_heads": 2, "dim": 104, "vdim": 72, "scale": 0.1, "mask": {"size": 65}},
      "right": {"heads": 2, "dim": 256, "vdim": 40, "tau": 16.0}}, 100),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(OTHER_SIZES)))
def test_mixers_at_other_sizes(case, dtype):
    m, rank = OTHER_SIZES[case]
    W, eps = 96, 1e-5
    weights = tiny.random_tensors(tiny.mixer_shapes("a", m, W, rank), seed=case)
    torch.manual_seed(8 + case)
    xs = [torch.randn(n, W).to(dtype).float() for n in (300, 90)]
    for side in ("left", "right", None):
        part = mixer_part(m, W, eps, weights, dtype, rank, side=side)
        cache = new_cache(part, 1024, 3, dtype)
        plain_of = plain.parallel_mixer if side is None else PLAIN_SIDE[side]
        want = [plain_of(m if side is None else m[side], double(weights),
                         "a" if side is None else f"a.{side}", x.double(), eps) for x in xs]
        for cuts in ([[300], [90]], [[130, 2, 100, 1, 1, 66], [66, 2, 20, 1, 1]]):
            got = run_mixer(part, cache, xs, cuts, dtype)
            for g, w in zip(got, want):
                assert rel_error(g, w) < bound(dtype), (m, side, cuts)


@pytest.mark.parametrize("width", [64, 100, 51, 2048, 5000])
@pytest.mark.parametrize("planes", [1, 3])
def test_norms_behind_parts(width, planes):
    """One result and two side by side, as rows and as split-K planes, in front of the
    plain stream, of a norm, and with only the sum made; float32 and bfloat16 out."""
    from foundry_b200.kernels import ops
    gen = torch.Generator().manual_seed(width + planes)
    draw = lambda *s: torch.randn(s, generator=gen)
    T, eps = 5, 1e-3
    resid, a, b = draw(T, width), draw(planes, T, width), 3.0 * draw(planes, T, width)
    wa, wb, w1, w2 = (draw(width) for _ in range(4))
    unit = lambda x: plain.rms_unit(x, eps)
    dev = lambda t: t.to(DEV).contiguous()
    as_values = lambda t: ops.Planes(dev(t)) if planes > 1 else dev(t[0])
    sa, sb = a.double().sum(0), b.double().sum(0)
    cases = [(None, None),
             (as_values(a), sa),
             (ops.NormedPair(as_values(a), dev(wa), as_values(b), dev(wb), eps, 0.3),
              0.3 * (unit(sa) * wa.double() + unit(sb) * wb.double()))]
    for values, y in cases:
        want = resid.double() if y is None else resid.double() + unit(y) * w1.double()
        pending = None if values is None else ops.PostNormed(values, dev(w1), eps)
        for weight, expected in ((None, want), (w2, unit(want) * w2.double())):
            for dtype in DTYPES:
                stream = dev(resid)
                out = torch.empty((T, width), dtype=dtype, device=DEV)
                ops.post_norm_add(stream, pending, None if weight is None else dev(weight), eps, out)
                assert rel_error(stream.cpu(), want) < 2e-6
                assert rel_error(out.float().cpu(), expected) < (2e-6 if dtype == torch.float32 else 6e-3)
        if pending is not None:
            stream = dev(resid)
            pending.settle(stream)
            assert rel_error(stream.cpu(), want) < 2e-6
            rows = torch.tensor([3, 0], dtype=torch.int32, device=DEV)
            picked = dev(resid[[3, 0]])
            pending.take(rows, 2).settle(picked)
            assert rel_error(picked.cpu(), want[[3, 0]]) < 2e-6


@pytest.mark.parametrize("sizes", [(64, 256, 128, 128), (2048, 512, 512, 1024), (96, 40, 328, 24), (520, 100, 64, 7)])
def test_two_products_of_a_handful_of_tokens_in_one_launch(sizes):
    from foundry_b200.parts.products import product_pair
    k1, n1, k2, n2 = sizes
    gen = torch.Generator().manual_seed(k1)
    draw = lambda *s: torch.randn(s, generator=gen).to(torch.bfloat16)
    for T in (1, 3, 8, 11, 16, 40):
        x1, w1, x2, w2 = draw(T, k1), draw(n1, k1), draw(T, k2), draw(n2, k2)
        got, counts = counted(lambda: product_pair(*(t.to(DEV) for t in (x1, w1, x2, w2))))
        assert counts.get("gemm_skinny_pair", 0) == (1 if T <= 16 else 0)
        for g, x, w in zip(got, (x1, x2), (w1, w2)):
            assert rel_error(joined(g).cpu(), x.double() @ w.double().T) < 1e-5


@pytest.mark.parametrize("rank, channels, tau", [(1, 5, 1.0), (16, 200, 16.0), (40, 300, 3.0), (27, 64, 0.5)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_from_a_low_rank_projection(rank, channels, tau, dtype):
    """Also where the sigmoid is so close to 0 or to 1 that only its logarithm keeps it."""
    from foundry_b200.kernels import ops
    gen = torch.Generator().manual_seed(rank)
    for T in (1, 3, 37, 150):
        p = torch.randn(T, rank + 9, generator=gen).to(DEV)
        w = torch.randn(channels, rank, generator=gen).to(dtype).to(DEV)
        bias = (torch.randn(channels, generator=gen) * 20.0).to(DEV)
        out = torch.empty((T, channels), dtype=torch.float32, device=DEV)
        ops.low_rank_decay(p[:, 4:4 + rank], w, bias, tau, out)
        z = p[:, 4:4 + rank].cpu().double() @ w.cpu().double().T + bias.cpu().double()
        want = torch.exp(plain.log_sigmoid(z) / tau)
        err = (out.cpu().double() - want).abs() / want.clamp(min=1e-30)
        assert float(err[want > 1e-30].max()) < 1e-4 and bool((out >= 0).all())


@pytest.mark.parametrize("chunk_tokens", [16, 64])
@pytest.mark.parametrize("dims", [(4, 16, 24), (2, 64, 64), (3, 128, 40), (2, 128, 128), (1, 300, 33)])
def test_chunks_side_by_side_equal_the_scan_in_order(dims, chunk_tokens, monkeypatch):
    """The linear recurrences over sequences of unequal lengths, some shorter than one chunk,
    from states that earlier tokens left: outputs and final states of the chunked form
    against the scan in token order, for a decay a channel, for one decay a head with step
    size and skip, and for the time mixing with a bonus."""
    from foundry_b200.cache import SequenceCache, StateRequest
    from foundry_b200.kernels import ops
    H, d, e = dims
    gen = torch.Generator().manual_seed(d)
    lens = [1000, 3, 413, chunk_tokens, 1]
    T = sum(lens)
    cache = SequenceCache({0: StateRequest((H * d * e,))}, 4096, 8, torch.float32, DEV)
    slots = [cache.open_sequence() for _ in lens]
    ctx = make_ctx(cache, slots, lens)
    start = torch.randn(cache.view(0, True).rows.shape, generator=gen)
    q, k = (torch.randn(T, H * d, generator=gen).to(DEV) for _ in range(2))
    v = torch.randn(T, H * e, generator=gen).to(DEV)
    channel = (1.0 - 0.2 * torch.rand(T, H * d, generator=gen) ** 3).to(DEV)
    head = (1.0 - 0.2 * torch.rand(T, H, generator=gen)).to(DEV)
    step, skip = torch.rand(T, H, generator=gen).to(DEV), torch.randn(H, generator=gen).to(DEV)
    bonus = torch.randn(H, d, generator=gen).to(DEV)
    forms = [dict(mode=ops.SCAN_LINEAR, g=channel, out_scale=0.3),
             dict(mode=ops.SCAN_LINEAR, g=head, beta=step, bonus=skip, decay_per_head=True)]
    if d == e:
        forms.append(dict(mode=ops.SCAN_WKV, g=channel, bonus=bonus))
    for form in forms:
        form = dict(form)
        mode, g = form.pop("mode"), form.pop("g")
        results = []
        for tokens in (0, chunk_tokens):
            monkeypatch.setattr(ops, "SCAN_CHUNK_TOKENS", tokens)
            assert (ops.scan_chunks(ctx, mode, H, d, e)[0] > 1) == (tokens > 0)
            cache.view(0, True).rows.copy_(start.to(DEV))
            out = torch.empty((T, H * e), dtype=torch.float32, device=DEV)
            ops.state_scan(ctx, mode, q, k, v, g, ops.StateRows(cache.view(0, True).rows, [("S", H * d * e)]),
                           "S", out, H, 1, d, e, **form)
            results.append((out.cpu(), cache.view(0, True).rows.cpu()))
        assert rel_error(results[1][0], results[0][0]) < 1e-5
        held = [s for s in slots]
        assert rel_error(results[1][1][held], results[0][1][held]) < 1e-5
        others = [s for s in range(results[0][1].shape[0]) if s not in held]
        assert torch.equal(results[1][1][others], start[others])  # nobody else's state is touched


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 16, 24, 5), (2, 64, 64, 16), (3, 128, 128, 33), (1, 256, 256, 64),
                                   (2, 40, 20, 1), (5, 100, 80, 9)])
def test_single_tokens_in_one_kernel_equal_the_three(sizes, dtype, monkeypatch):
    """The fused single-token kernel against decays, scan and gated norm one by one, on the
    same states (each slot's moved on by the same tokens), and counted."""
    from foundry_b200.kernels import ops
    H, d, e, rank = sizes
    m = {"left": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.3},
         "right": {"heads": H, "dim": d, "vdim": e, "tau": 3.0}}
    weights = tiny.random_tensors(tiny.mixer_shapes("a", m, 64, rank), seed=rank)
    part = mixer_part(m, 64, 1e-5, weights, dtype, rank, side="right")
    torch.manual_seed(rank)
    xs = [torch.randn(9, 64).to(dtype).float() for _ in range(3)]
    results = []
    for fused in (True, False):
        monkeypatch.setattr(ops, "LINEAR_STEP", fused)
        cache = new_cache(part, 256, 4, dtype)
        got, counts = counted(lambda: run_mixer(part, cache, xs, [[4] + [1] * 5] * 3, dtype))
        assert counts.get("linear_step", 0) == (5 if fused else 0)
        results.append((got, cache.view(0, True).rows.cpu()))
    for g, w in zip(*(r[0] for r in results)):
        assert rel_error(g, w) < (1e-5 if dtype == torch.float32 else 1e-2)
    assert rel_error(results[0][1][:3], results[1][1][:3]) < 1e-5


# --------------------------------------------- one key that stands out, anywhere
def crafted_attention(W, d, e, window, heads=1, kv_heads=1):
    """A window attention made so that a query that carries input 1 matches only a key that
    carries input 2: after the heads' norms that score is about 20, every other key's about
    +-1. Queries and keys live in the elements behind the rotated ones, so the rotation
    runs but turns zeros. Values are inputs 4..8; the biases are zero."""
    rot = d // 2
    m = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": e, "scale": 20.0 / d,
         "rot": {"dims": rot, "base": 100.0}}
    if window:
        m["mask"] = {"size": window}
    both = {"left": m, "right": {"heads": 1, "dim": 8, "vdim": 8, "tau": 2.0}}
    w = {k: v for k, v in tiny.random_tensors(tiny.mixer_shapes("a", both, W, 2), seed=1).items()
         if k.startswith("a.left.") and not k.endswith(".out")}
    q, k = torch.zeros(heads * d, W), torch.zeros(kv_heads * d, W)
    for h in range(heads):
        q[h * d + rot, 1] = 1.0
    val = torch.zeros(kv_heads * e, W)
    for g in range(kv_heads):
        k[g * d + rot, 2] = 1.0
        k[g * d + rot + 1, 0] = 1.0
        val[g * e:g * e + 4, 4:8] = torch.eye(4)
    out = torch.zeros(W, heads * e)  # the mean over the heads
    n = min(W, e)
    for h in range(heads):
        out[:n, h * e:h * e + n] += torch.eye(n) / heads
    out = out.to(torch.bfloat16).float()
    w.update({"a.left.q": q, "a.left.k": k, "a.left.v": val, "a.left.o": out,
              "a.left.q.norm": torch.ones(d), "a.left.k.norm": torch.ones(d)})
    w.update({f"a.left.{n}.b": torch.zeros_like(w[f"a.left.{n}.b"]) for n in "qkv"})
    return both, w


def marked_inputs(query_at, marker_at, width, behind=0):
    """Rows in which only the query of `query_at` (input 1) and the key of `marker_at`
    (input 2) match; ordinary rows carry input 0. The marker's value (inputs 4..8) is
    unlike every other. With query and marker at the same place the row carries both.
    `behind`: ordinary rows after the query."""
    gen = torch.Generator().manual_seed(query_at * 1000 + marker_at)
    x = torch.zeros(query_at + 1 + behind, width)
    x[:, 0] = 1.0
    x += 0.05 * torch.randn(x.shape, generator=gen)
    x[query_at] = 0.05 * torch.randn(width, generator=gen)
    x[query_at, 0] += 1.0  # (its own key is an ordinary one)
    x[query_at, 1] = 1.0
    if marker_at != query_at:
        x[marker_at] = 0.05 * torch.randn(width, generator=gen)
    x[marker_at, 2] = 1.0
    x[marker_at, 4:8] += 3.0
    return x.to(torch.bfloat16).float()


def places(window):
    """(query position, marker position, visible): the window's first key and the key in
    front of it, the first token of the sequence, the query itself and its neighbour,
    for queries at the first tokens, on both sides of page borders and far out."""
    out = []
    for q in (5, 63, 64, 129, 200, 700):
        lo = max(0, q - window + 1) if window else 0
        seen = {lo, q, max(lo, q - 1), min(q, lo + 1)}
        hidden = {lo - 1, 0, lo - 64} if lo > 0 else set()
        out += [(q, j, True) for j in sorted(seen)]
        out += [(q, j, False) for j in sorted(hidden) if j >= 0]
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 64, 65, 640, None])
@pytest.mark.parametrize("sizes", [(8, 8, 1, 1), (64, 64, 2, 1), (32, 128, 2, 2), (128, 128, 4, 1),
                                   (80, 56, 20, 1)])
def test_one_key_that_stands_out_on_both_sides_of_every_edge(sizes, window, dtype):
    """A crafted attention in which one key dominates one query. The key lies just inside
    or just outside the query's window, at the sequence's first token, on both sides of
    cache pages' borders, hundreds of tokens back, or is the query's own; the query is the
    last token of a prompt, stands in front of others in its prompt's portion, or is
    decoded alone."""
    d, e, heads, kv_heads = sizes
    W = 32
    m, weights = crafted_attention(W, d, e, window, heads, kv_heads)
    part = mixer_part(m, W, 1e-6, weights, dtype, 2, side="left")
    cache = new_cache(part, 2048, 2, dtype)
    wd = double(weights)
    for query_at, marker_at, visible in places(window):
        x = marked_inputs(query_at, marker_at, W, behind=3)
        want = plain.window_attention(m["left"], wd, "a.left", x[max(0, query_at - 700):query_at + 1].double(),
                                      1e-6)[-1]
        # the plain implementation itself sees the marker where it should and only there
        assert (float(want.norm()) > 2.0) == visible, (query_at, marker_at, float(want.norm()))
        for cut in ([query_at + 1, 3], [query_at, 1, 3], [query_at - 1, 5]):
            got = run_mixer(part, cache, [x], [cut], dtype)[0][query_at].double()
            err = float((got - want).norm()) / max(float(want.norm()), 1.0)
            assert err < bound(dtype, 5.0), (query_at, marker_at, visible, cut, err)


@pytest.mark.parametrize("window", [37, 64, 150, 1000, None])
@pytest.mark.parametrize("sizes", [(64, 64, 4, 2), (128, 128, 2, 1), (96, 64, 3, 3), (40, 120, 2, 2)])
def test_prompts_and_single_tokens_on_the_tensor_cores(sizes, window):
    """bfloat16 prompts against the plain attention and against the CUDA-core kernel on the
    same cache: windows that end inside a block of queries and inside a cache page,
    portions that begin in the middle of a page, three unequal sequences a step, then single
    tokens; and the kernels counted, so that no other path stands in for them."""
    from foundry_b200.kernels import ops
    d, e, heads, kv_heads = sizes
    left = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": e, "scale": d ** -0.5,
            "rot": {"dims": d // 2, "base": 1000.0}}
    if window:
        left["mask"] = {"size": window}
    W, eps = 64, 1e-5
    m = {"left": left, "right": {"heads": 1, "dim": 8, "vdim": 8, "tau": 2.0}}
    weights = tiny.random_tensors(tiny.mixer_shapes("a", m, W, 2), seed=d + e)
    part = mixer_part(m, W, eps, weights, torch.bfloat16, 2, side="left")
    cache = new_cache(part, 2048, 3, torch.bfloat16)
    torch.manual_seed(d)
    xs = [torch.randn(n, W).to(torch.bfloat16).float() for n in (333, 70, 129)]
    want = [plain.window_attention(left, double(weights), "a.left", x.double(), eps) for x in xs]
    results = {}
    for tc in (True, False):
        ops.WINDOW_ATTENTION_TC = tc
        try:
            for cuts in ([[333], [70], [129]], [[100, 133, 2, 97, 1], [5, 63, 1, 1], [64, 65]]):
                got, counts = counted(lambda: run_mixer(part, cache, xs, cuts, torch.bfloat16))
                prompts = counts.get("attention_prefill_tc", 0)
                assert (prompts > 0) == tc, counts
                results[tc, len(cuts[0])] = got
                for g, w in zip(got, want):
                    assert rel_error(g, w) < bound(torch.bfloat16), (sizes, window, tc, cuts)
        finally:
            ops.WINDOW_ATTENTION_TC = True
    for g, w in zip(results[True, 1], results[False, 1]):  # the two kernels agree more closely
        assert rel_error(g, w) < 0.5 * bound(torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_survives_every_cutting(dtype):
    """Decays close to one, so that the first tokens still weigh on the last: the state
    carried through portions of one and two tokens equals the whole prompt's (whose
    chunks run side by side)."""
    m = {"left": {"heads": 1, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 7}},
         "right": {"heads": 4, "dim": 24, "vdim": 16, "tau": 16.0}}
    weights = tiny.random_tensors(tiny.mixer_shapes("a", m, 48, 5), seed=3)
    weights["a.right.a2.b"] = torch.full((96,), 4.0)
    part = mixer_part(m, 48, 1e-6, weights, dtype, 5, side="right")
    cache = new_cache(part, 1024, 3, dtype)
    torch.manual_seed(4)
    xs = [torch.randn(n, 48).to(dtype).float() for n in (350, 9)]
    wd = double(weights)
    plain_of = lambda x: plain.gated_linear(m["right"], wd, "a.right", x.double(), 1e-6)
    want = [plain_of(x) for x in xs]
    moved = xs[0].clone()
    moved[0] += 1.0  # (the plain form itself: the first token still matters at the end)
    assert rel_error(plain_of(moved)[-1:], want[0][-1:]) > 1e-3
    for cuts in ([[350], [9]], [[1, 2, 1, 3, 2, 264, 2, 1] + [1] * 10 + [64], [2, 2, 2, 2, 1]]):
        got = run_mixer(part, cache, xs, cuts, dtype)
        for g, w in zip(got, want):
            assert rel_error(g, w) < bound(dtype, 2.0), cuts


def test_a_state_row_starts_at_zero_on_a_slot_that_was_used(dtype=torch.float32):
    """A sequence that opens on a slot whose last owner left a large state gives what it
    gives on a fresh cache."""
    m = tiny.CONFIGS["other"]["layers"][0]["mixer"]
    weights = tiny.random_tensors(tiny.mixer_shapes("a", m, 64, 3), seed=9)
    part = mixer_part(m, 64, 1e-6, weights, dtype, 3)
    cache = new_cache(part, 512, 1, dtype)
    torch.manual_seed(1)
    loud, x = 30.0 * torch.randn(80, 64), torch.randn(21, 64)
    want = plain.parallel_mixer(m, double(weights), "a", x.double(), 1e-6)
    run_mixer(part, cache, [loud], [[80]], dtype)
    for cut in ([21], [1] * 21):
        assert rel_error(run_mixer(part, cache, [x], [cut], dtype)[0], want) < bound(dtype)


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("tokovik")
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_model_in_every_cutting(name, dtype, folders):
    """Whole prompts alone; token by token from the first token on; portions of
    several sizes down to two tokens; a batch of unequal requests decoded
    together while the shorter ones end; all on slots and pages that the
    earlier cuttings used and gave back."""
    import foundry_b200 as fb
    folder, weights = folders[name]
    vocab = tiny.CONFIGS[name]["vocab"]
    rng = np.random.default_rng(11)
    prompts = [[int(t) for t in rng.integers(0, vocab, n)] for n in (310, 1, 3, 81)]
    want = [plain_logits(name, weights, p) for p in prompts]
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
        for g, w in zip(got, wanted[cutting]):
            assert np.isfinite(g).all()
            assert rel_error(g, w) < bound(dtype, 2.0 if dtype == "float32" else 3.0), \
                (name, dtype, cutting, len(w))
    if dtype == "float32":  # the cuttings agree with each other to rounding
        assert rel_error(results["portions"][0], results["whole, alone"][0]) < 2e-5
        assert rel_error(results["batch, then decoded together"][3], results["whole, alone"][3]) < 2e-5
    engine.cache.table.check()
    assert engine.free_slots() == 6


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_long_decoding_and_reused_slots(name, folders):
    """260 tokens decoded one by one behind a short prompt (across cache pages and far
    beyond every window), twice on the same slot with another sequence between."""
    import foundry_b200 as fb
    folder, weights = folders[name]
    vocab = tiny.CONFIGS[name]["vocab"]
    rng = np.random.default_rng(12)
    tokens = [int(t) for t in rng.integers(0, vocab, 265)]
    other = [int(t) for t in rng.integers(0, vocab, 40)]
    want = plain_logits(name, weights, tokens)
    engine = fb.Engine.from_folder(folder, dtype="float32", max_tokens=512, max_slots=2)
    first = run_cutting(engine, [tokens], [[5] + [1] * 260])[0]
    run_cutting(engine, [other], [[40]])
    again = run_cutting(engine, [tokens], [[5] + [1] * 260])[0]
    assert rel_error(first, want) < bound("float32", 2.0)
    assert np.array_equal(first, again)


def test_sizes_that_fit_no_tensor_core_product_and_layers_in_another_order(tmp_path):
    """Width 52 and inner sizes that are no multiples of 8 (in bfloat16 every product takes
    the CUDA-core kernel); the layer without feed-forward last, so that a pair of results
    meets the final norm; every layer with sizes, window and rotation of its own."""
    import foundry_b200 as fb
    left = {"heads": 3, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.3, "mask": {"size": 33},
            "rot": {"dims": 6, "base": 777.0,
                    "scaling": {"factor": 2.0, "original": 40, "fast": 3.0, "slow": 0.4}}}
    right = {"heads": 3, "dim": 5, "vdim": 6, "tau": 7.0}
    doc = {"architecture": "Tokovik", "vocab": 77, "width": 52, "norm": {"eps": 1e-5},
           "embedding": {"scale": 7.0}, "logit_scale": 2.0,
           "layers": [
               {"type": "parallel", "mixer": {"left": dict(left, heads=2, kv_heads=1, vdim=9, mask={"size": 2}),
                                              "right": dict(right, heads=4, tau=1.0)},
                "mlp": {"kind": "dense", "ff": 90}},
               {"type": "parallel", "mixer": {"left": left, "right": right},
                "mlp": {"kind": "dense", "ff": 18}},
               {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": None}]}
    weights = tiny.random_tensors(tiny.tensor_shapes(doc, [2, 9, 1]), seed=31)
    folder, _ = tiny.write_model(str(tmp_path / "odd"), doc, weights)
    rng = np.random.default_rng(3)
    prompts = [[int(t) for t in rng.integers(0, 77, n)] for n in (70, 9)]
    want = [plain.forward(doc, double(weights), p).numpy() for p in prompts]
    for dtype in ("float32", "bfloat16"):
        engine = fb.Engine.from_folder(folder, dtype=dtype, max_tokens=512, max_slots=3)
        got = run_cutting(engine, prompts, [[66, 2, 1, 1], [5, 1, 2, 1]])
        for g, w in zip(got, want):
            assert rel_error(g, w) < bound(dtype, 2.0), dtype


def test_wider_heads_through_the_serving_kernels(tmp_path):
    """One layer of each kind at sizes whose bfloat16 steps take the tensor-core products and
    attentions in prompts, in replayed short prompts and in single tokens (graphs), with
    a window that passes over decoded tokens."""
    import foundry_b200 as fb
    mixer = {"left": {"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.125,
                      "mask": {"size": 130}, "rot": {"dims": 64, "base": 10000.0}},
             "right": {"heads": 2, "dim": 128, "vdim": 128, "tau": 16.0}}
    doc = {"architecture": "Tokovik", "vocab": 320, "width": 512, "norm": {"eps": 1e-5},
           "embedding": {"scale": 2.0}, "logit_scale": 0.3,
           "layers": [{"type": "parallel", "mixer": mixer, "mlp": {"kind": "dense", "ff": 768}},
                      {"type": "parallel", "mixer": mixer, "mlp": None}]}
    weights = tiny.random_tensors(tiny.tensor_shapes(doc, [16, 16]), seed=41)
    folder, _ = tiny.write_model(str(tmp_path / "wide"), doc, weights)
    rng = np.random.default_rng(5)
    prompts = [[int(t) for t in rng.integers(0, 320, n)] for n in (700, 150, 40)]
    want = [plain.forward(doc, double(weights), p).numpy() for p in prompts]
    engine = fb.Engine.from_folder(folder, dtype="bfloat16", max_tokens=2048, max_slots=4)
    for cuts in ([[700], [150], [40]], [[600, 60] + [1] * 40, [100, 2, 8] + [1] * 40, [1, 2, 3] + [1] * 34]):
        for g, w in zip(run_cutting(engine, prompts, cuts), want):
            assert rel_error(g, w) < bound("bfloat16", 2.0), (cuts[0][:3], len(w))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(dtype, folders):
    """`Engine.generate` (the scheduler's batches, graphs, slot reuse) against the
    plain model's greedy tokens; five prompts through batches of two."""
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
        assert dtype == "bfloat16" and gap < 0.05 * float(logits.abs().max()), (g, w, gap)


def test_trace_replay_and_command_line(folders, tmp_path):
    """`bin/trace_run` on a Tokovik folder: a prompt step of two requests, then
    single tokens, one request ending early; and `foundry run` generating."""
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
    run = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "foundry"), "run", "--model",
                          folder, "--dtype", "float32", "--prompt-ids", ",".join(map(str, a)),
                          "--max-new-tokens", "4", "--ignore-eos"], capture_output=True, text=True,
                         timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    want = plain.greedy_generate(cfg, double(weights), a, 4)
    assert json.loads(run.stdout.strip().split("\n")[-1]) == want


def test_command_line_bench_on_a_tokovik_folder(folders, tmp_path):
    """`foundry bench` (prompt step, decode steps, report with bytes and operations)."""
    folder, _ = folders["mixed"]
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "foundry"), "bench", "--model",
                           folder, "--prompt-tokens", "20", "--new-tokens", "5", "--runs", "2",
                           "--batch-size", "3", "--out", str(tmp_path)],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    report = json.loads((tmp_path / "report.json").read_text())
    assert len(report["runs"]) == 2 and all(len(r) == 5 for r in report["runs"][0]["token_ids"])
    assert report["runs"][0]["token_ids"] == report["runs"][1]["token_ids"]
