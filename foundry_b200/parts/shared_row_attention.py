"""Grouped-query attention whose values are its keys before their norm, with a learnt bias
by distance, a sliding window that keeps the first tokens and an output gate, as a mixer.

    q = Wq h (H x dim), r = Wk h (G x dim), z = Wg h (H x dim)     (one product), no biases
    q' = q / sqrt(mean(q^2) + eps) * wq per head;   k = r f wk,  f = 1 / sqrt(mean(r^2) + eps)
    s_ij = (q'_i . k_j) * scale + rel[bucket(i - j), head]
    j visible to i iff j <= i and (i - j < window or j < keep_first)
    out = Wo [softmax(s) r side by side * sigmoid(z)]

No rotation: positions enter through the table and the mask only; a kept token counts by the
distance it really has. bucket(n) of a table of B rows: n itself below B / 2, then
B / 2 + floor(ln(n / (B / 2)) / ln(bias_max / (B / 2)) * (B - B / 2)), at most B - 1.

Because a key is its value times a number a row and a vector for all rows, a token has ONE
cached row a head: r as it was projected, read as the value, and f beside it; wk goes into
the queries' weight, (q' wk) . (r f) = q' . k. That is half the cache and half the bytes of a
single-token step of two rows. The table is laid out by distance at load time, so a kernel's
bias is one read. Every constant is a parameter. Tensor names under the mixer's prefix:
`q k g o`, `q.norm k.norm`, `rel`.

The cache keeps every row of a sequence (kept tokens stay readable for ever); the kernels
walk the kept prefix and the window only. In bfloat16 prompts run on tcgen05 (one ring of
pages for both products, the table in shared memory, the gate in the epilogue) and single
tokens on the split-range tensor-core kernel; float32 and other sizes on the CUDA cores.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np
import torch

from ..cache.store import KVRequest, KVView
from ..kernels import ops
from ..weights.loader import ExpectedTensor
from .base import Fetch, Part, register_mixer
from .products import product_f32

NO_ROTATION = ops.Rotation(None, "cpu")


def distance_buckets(rows: int, last: int) -> List[int]:
    """bucket(n) for n = 0 .. last (every distance from `last` on has the last row). The
    logarithms' floor is decided in whole numbers: floor >= k iff
    (n / half)^span >= (last / half)^k."""
    half = rows // 2
    span = rows - half
    if half < 1 or last <= half:
        raise ValueError(f"a table of {rows} rows with its last bucket at distance {last}")
    out, k = [], 0
    for n in range(last + 1):
        if n < half:
            out.append(n)
            continue
        while k < span and last ** (k + 1) * half ** span <= n ** span * half ** (k + 1):
            k += 1
        out.append(min(rows - 1, half + k))
    return out


@register_mixer("shared_row_attention")
class SharedRowAttention(Part):
    replay_safe = True

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, scale: float, eps: float,
                 bias_rows: int, bias_max: int, window: Optional[int] = None, keep_first: int = 0,
                 output_gate: bool = True, *, dtype: torch.dtype, device: torch.device):
        if kv_heads <= 0 or heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} key-value heads")
        if not 1 <= dim <= 768:
            raise ValueError(f"head size {dim} must be at most 768")
        self.width, self.heads, self.kv_heads, self.dim = width, heads, kv_heads, dim
        self.scale, self.eps = float(scale), float(eps)
        self.window, self.keep_first = (int(window) if window else 0), int(keep_first or 0)
        self.bias_rows, self.bias_max = int(bias_rows), int(bias_max)
        self.buckets = distance_buckets(self.bias_rows, self.bias_max)
        self.output_gate = bool(output_gate)
        self.dtype, self.device = dtype, device
        self.nq, self.nk = heads * dim, kv_heads * dim
        self.w_in = self.w_o = self.qk_norm = self.dist_bias = None

    def expected_tensors(self, prefix: str) -> Dict[str, ExpectedTensor]:
        W = self.width
        shapes = {"q": (self.nq, W), "k": (self.nk, W), "q.norm": (self.dim,),
                  "k.norm": (self.dim,), "rel": (self.bias_rows, self.heads), "o": (W, self.nq)}
        if self.output_gate:
            shapes["g"] = (self.nq, W)
        return {f"{prefix}.{n}": ExpectedTensor(s) for n, s in shapes.items()}

    def load(self, prefix: str, fetch: Fetch) -> None:
        names = ("q", "k", "g") if self.output_gate else ("q", "k")
        self.w_in = torch.cat([fetch(f"{prefix}.{n}") for n in names], 0).contiguous()
        self.w_o = fetch(f"{prefix}.o").contiguous()
        self.qk_norm = (fetch(f"{prefix}.q.norm").to(torch.float32)
                        * fetch(f"{prefix}.k.norm").to(torch.float32)).contiguous()
        table = fetch(f"{prefix}.rel").to(torch.float32)
        rows = torch.tensor(self.buckets, dtype=torch.long, device=table.device)
        self.dist_bias = ops.DistanceBias(table[rows].t())  # by distance, 0 .. bias_max

    def cache_request(self) -> KVRequest:
        return KVRequest(self.kv_heads, self.dim, None, 0, row_scales=True)

    def first_weight(self):
        return self.w_in

    def context_flops(self, token_counts, starts) -> float:
        pairs = 0.0
        for n, start in zip(token_counts, starts):
            seen = np.arange(start + 1, start + n + 1, dtype=np.float64)
            if self.window:
                kept = np.minimum(self.keep_first, np.maximum(0, seen - self.window))
                seen = np.minimum(seen, self.window + kept)
            pairs += float(seen.sum())
        return 4.0 * self.heads * self.dim * pairs

    def forward(self, ctx, x, cache: KVView):
        table = ctx.page_table(cache.group)
        rows = product_f32(x, self.w_in)  # [T, q | the key rows | the gate]
        q = torch.empty((x.shape[0], self.nq), dtype=x.dtype, device=x.device)
        ops.head_norm_rope_cache_write(rows, q, self.qk_norm, None, self.eps, False, ctx,
                                       NO_ROTATION, table, cache.k, cache.v, self.heads,
                                       self.kv_heads, self.dim, self.dim,
                                       write_cache=cache.writes, key_scales=cache.row_scales)
        attn = torch.empty((x.shape[0], self.nq), dtype=x.dtype, device=x.device)
        ops.attention_shared_rows(ctx, q, attn, table, cache.k, cache.row_scales, self.heads,
                                  self.kv_heads, self.dim, self.scale, window=self.window,
                                  keep_first=self.keep_first, dist_bias=self.dist_bias,
                                  gate=rows[:, self.nq + self.nk:] if self.output_gate else None,
                                  then_reads=self.w_o)
        return product_f32(attn, self.w_o)
