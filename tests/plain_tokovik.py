"""The Tokovik decoder, plainly: float64, whole sequences, no cache, no state
carried between calls, one function per mechanism. It takes a decoded
config.json document and a dict of tensors by their file names, and shares no
code with `foundry_b200`. `gated_linear_stepwise` walks a sequence token by
token with an explicit state and guards the whole-sequence form
(tests/test_tokovik_cpu.py).

Notation: T tokens, W width, H heads, G key/value heads, d key size, e value
size, f rotation frequencies.
"""
import math

import torch

F = torch.float64


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_around_zero(x, w, eps):
    """The model's norm: the stored weight is the distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def silu(z):
    return z * torch.exp(log_sigmoid(z))


def yarn(rot):
    """(frequencies [dims / 2], the factor on cosine and sine) of a rotation entry."""
    dims, base = rot["dims"], rot["base"]
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def dim_of(turns):  # the element whose wavelength makes `turns` turns in the original span
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(s["fast"])), 0)
    hi = min(math.ceil(dim_of(s["slow"])), dims - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
                         for i in range(dims // 2)], dtype=F)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate_half(x, positions, freq, factor):
    """x [T, heads, d]: element i < n = len(freq) of a head turns with element i + n by
    the angle position * freq[i], cosine and sine times `factor`; elements from 2 n on
    pass unchanged."""
    n = freq.shape[0]
    if not n:
        return x
    angle = torch.as_tensor(positions, dtype=F)[:, None] * freq[None, :]
    cos, sin = factor * torch.cos(angle)[:, None, :], factor * torch.sin(angle)[:, None, :]
    u, v, rest = x[..., :n], x[..., n:2 * n], x[..., 2 * n:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], -1)


def window_visible(i, j, size):
    """Whether the query at position i sees the key at position j."""
    return 0 <= i - j and (size is None or i - j < size)


def window_attention(m, w, p, h, eps):
    """The left mixer. m: its config entry; tensors `p.q|k|v` with `.b`, `p.q.norm`,
    `p.k.norm`, `p.o`; h [T, W] from position 0 on."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size = (m.get("mask") or {}).get("size")
    q, k, v = (h @ w[f"{p}.{n}"].T + w[f"{p}.{n}.b"] for n in "qkv")
    q = rms_unit(q.view(T, H, d), eps) * w[f"{p}.q.norm"]
    k = rms_unit(k.view(T, G, d), eps) * w[f"{p}.k.norm"]
    v = v.view(T, G, e)
    if m.get("rot"):
        freq, factor = yarn(m["rot"])
        q, k = (rotate_half(x, range(T), freq, factor) for x in (q, k))
    see = torch.tensor([[window_visible(i, j, size) for j in range(T)] for i in range(T)])
    heads = []
    for a in range(H):
        g = a // (H // G)
        score = (q[:, a] @ k[:, g].T) * m["scale"]
        score = torch.where(see, score, torch.full((), -math.inf, dtype=F))
        heads.append(torch.softmax(score, -1) @ v[:, g])
    return torch.cat(heads, -1) @ w[f"{p}.o"].T


def _linear_inputs(m, w, p, h):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[f"{p}.q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[f"{p}.k"].T).view(T, H, d)
    v = (h @ w[f"{p}.v"].T).view(T, H, e)
    z = (h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T + w[f"{p}.a2.b"]
    return q, k, v, (log_sigmoid(z) / m["tau"]).view(T, H, d)


def _linear_output(m, w, p, o, h, eps):
    o = rms_unit(o, eps) * w[f"{p}.norm"]  # [T, H, e]
    return (o.reshape(h.shape[0], -1) * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def gated_linear(m, w, p, h, eps):
    """The right mixer in the attention-like form: the output at i is the sum over j <= i
    of (sum_c q_ic k_jc * product of channel c's decays after j up to i) v_j."""
    T = h.shape[0]
    q, k, v, log_a = _linear_inputs(m, w, p, h)
    total = torch.cumsum(log_a, 0)  # [T, H, d]
    o = torch.zeros_like(v)
    for i in range(T):
        decay = torch.exp(total[i][None] - total[:i + 1])  # [i + 1, H, d]
        weight = (q[i][None] * k[:i + 1] * decay).sum(-1)  # [i + 1, H]
        o[i] = (weight[:, :, None] * v[:i + 1]).sum(0)
    return _linear_output(m, w, p, o, h, eps)


def gated_linear_stepwise(m, w, p, h, eps):
    """The same token by token: S <- diag(alpha) S + k v^T; o = S^T q."""
    q, k, v, log_a = _linear_inputs(m, w, p, h)
    S = torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=F)
    o = torch.zeros_like(v)
    for t in range(h.shape[0]):
        for a in range(m["heads"]):
            S[a] = torch.exp(log_a[t, a])[:, None] * S[a] + torch.outer(k[t, a], v[t, a])
            o[t, a] = S[a].T @ q[t, a]
    return _linear_output(m, w, p, o, h, eps)


def parallel_mixer(m, w, p, h, eps):
    left = window_attention(m["left"], w, f"{p}.left", h, eps)
    right = gated_linear(m["right"], w, f"{p}.right", h, eps)
    return 0.5 * (rms_unit(left, eps) * w[f"{p}.left.out"] +
                  rms_unit(right, eps) * w[f"{p}.right.out"])


def feed_forward(w, p, h):
    return (silu(h @ w[f"{p}.gate"].T) * (h @ w[f"{p}.up"].T)) @ w[f"{p}.down"].T


def layer_step(cfg, w, i, x):
    layer, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}"
    x = x + rms_around_zero(parallel_mixer(layer["mixer"], w, f"{p}.mix", x, eps),
                            w[f"{p}.norm1"], eps)
    if layer.get("mlp"):
        x = x + rms_around_zero(feed_forward(w, f"{p}.mlp", x), w[f"{p}.norm2"], eps)
    return x


def forward(cfg, weights, tokens, streams=None):
    """Logits [T, vocab] of the whole sequence; the stream behind every layer is appended
    to `streams` where a list is given."""
    w = {k: v.to(F) for k, v in weights.items()}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer_step(cfg, w, i, x)
        if streams is not None:
            streams.append(x)
    x = rms_around_zero(x, w["final.norm"], cfg["norm"]["eps"])
    return (x @ w["head"].T) * cfg["logit_scale"]


def greedy_generate(cfg, weights, prompt, count):
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(torch.argmax(forward(cfg, weights, tokens)[-1])))
    return tokens[len(prompt):]
