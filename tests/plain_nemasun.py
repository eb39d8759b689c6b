"""The Nemasun decoder, plainly: float64, whole sequences, no cache, one function per
mechanism. It takes a decoded config.json document and a dict of tensors by their file
names, and shares no code with `foundry_b200`.

Notation: T tokens, W width, S streams, H heads, G key/value heads, d head size,
B rows of a distance table.
"""
import math

import torch

F = torch.float64


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def distance_bucket(n, rows, last):
    """The table row of the distance n >= 0: one row a distance in the first half, rows of
    growing spans up to the distance `last` in the second, the last row from there on."""
    half = rows // 2
    if n < half:
        return n
    step = math.floor(math.log(n / half) / math.log(last / half) * (rows - half))
    return min(rows - 1, half + step)


def visible(i, j, mask):
    """Whether the query at position i sees the key at position j."""
    if j > i:
        return False
    size = (mask or {}).get("size")
    return size is None or i - j < size or j < (mask.get("keep_first") or 0)


def attention(m, w, p, h, eps):
    """m: the mixer's config entry; tensors `p.q|k|g|o`, `p.q.norm`, `p.k.norm`, `p.rel`;
    h [T, W] from position 0 on. The values are the keys before their norm."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = rms_norm((h @ w[f"{p}.q"].T).view(T, H, d), w[f"{p}.q.norm"], eps)
    v = (h @ w[f"{p}.k"].T).view(T, G, d)
    k = rms_norm(v, w[f"{p}.k.norm"], eps)
    table = w[f"{p}.rel"]
    rows = torch.tensor([distance_bucket(n, table.shape[0], m["bias_max"]) for n in range(T)])
    away = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    bias = table[rows[away.clamp(min=0)]]  # [T, T, H]
    see = torch.tensor([[visible(i, j, m.get("mask")) for j in range(T)] for i in range(T)])
    heads = []
    for a in range(H):
        g = a // (H // G)
        score = (q[:, a] @ k[:, g].T) * m["scale"] + bias[:, :, a]
        score = torch.where(see, score, torch.full((), -math.inf, dtype=F))
        heads.append(torch.softmax(score, -1) @ v[:, g])
    return (torch.cat(heads, -1) * sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def dense(mlp, w, p, h):
    limit = mlp["limit"]
    g = (h @ w[f"{p}.gate"].T + w[f"{p}.gate.b"]).clamp(max=limit)
    u = (h @ w[f"{p}.up"].T + w[f"{p}.up.b"]).clamp(min=-limit, max=limit)
    y = g * sigmoid(1.702 * g) * (u + 1.0)
    return y @ w[f"{p}.down"].T + w[f"{p}.down.b"]


def expert(w, p, h):
    g = h @ w[f"{p}.gate"].T
    return (g * sigmoid(g) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def choose(z, correction, router):
    """One token's (chosen outputs, their weights) from its router logits z, the routed
    experts first and the identity experts behind them."""
    n, top = z.shape[0], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(z, -1)
    c = (s + correction).tolist()
    size = n // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(c[g * size:(g + 1) * size]))
    open_to = [e for e in range(n) if e // size in best[:groups["keep"]]]
    chosen = sorted(open_to, key=lambda e: -c[e])[:top]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return chosen, [float(s[e]) / total for e in chosen]


def routed(mlp, w, p, h):
    router = mlp["router"]
    z = h @ w[f"{p}.router"].T
    out = expert(w, f"{p}.shared", h) if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*choose(z[t], w[f"{p}.correction"], router)):
            y = expert(w, f"{p}.e{e}", h[t]) if e < router["experts"] else h[t]
            out[t] = out[t] + weight * y
    return out


def feed_forward(mlp, w, p, h):
    return dense(mlp, w, p, h) if mlp["kind"] == "dense" else routed(mlp, w, p, h)


def connect(w, p, xs, sublayer):
    """One sublayer between streams xs [S, T, W]: what it reads is a weighted sum of the
    streams, and every stream becomes a weighted sum of the old ones plus its share of the
    result; `p.mix` is indexed [from, to]."""
    u = torch.einsum("s,stw->tw", w[f"{p}.in"], xs)
    y = sublayer(u)
    return torch.einsum("sr,stw->rtw", w[f"{p}.mix"], xs) + w[f"{p}.out"][:, None, None] * y


def layer_step(cfg, w, i, xs):
    layer, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}"
    xs = connect(w, f"{p}.hc1", xs, lambda u: attention(
        layer["mixer"], w, f"{p}.mix", rms_norm(u, w[f"{p}.norm1"], eps), eps))
    if layer.get("mlp"):
        xs = connect(w, f"{p}.hc2", xs, lambda u: feed_forward(
            layer["mlp"], w, f"{p}.mlp", rms_norm(u, w[f"{p}.norm2"], eps)))
    return xs


def forward(cfg, weights, tokens, streams=None):
    """Logits [T, vocab] of the whole sequence; the sum of the streams behind every layer is
    appended to `streams` where a list is given."""
    w = {k: v.to(F) for k, v in weights.items()}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    xs = torch.stack([x] * cfg["streams"])
    for i in range(len(cfg["layers"])):
        xs = layer_step(cfg, w, i, xs)
        if streams is not None:
            streams.append(xs.sum(0))
    x = rms_norm(xs.sum(0), w["final.norm"], cfg["norm"]["eps"])
    return x @ w["head"].T


def greedy_generate(cfg, weights, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(torch.argmax(forward(cfg, weights, tokens)[-1])))
    return tokens[len(prompt):]
