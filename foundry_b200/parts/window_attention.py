"""Grouped-query attention with biased projections, a norm of every query and key head,
rotation by given frequencies and a sliding window, as a mixer.

    q = Wq h + bq (H x dim), k = Wk h + bk (G x dim), v = Wv h + bv (G x vdim)  (one product)
    q, k per head:  x / sqrt(mean(x^2) + eps) * w   (w [dim], shared by the heads), then the
        first 2 n elements turned, element i with element i + n by the angle p * f_i at
        position p, cosine and sine times `rot_factor` (n = number of frequencies)
    s_ij = (q_i . k_j) * scale;   j visible to i iff 0 <= i - j < window  (None: j <= i)
    out = Wo [heads' softmax outputs side by side]

Keys have `dim` elements a head, values `vdim`; query head a reads key head
a // (H / G). Every constant is a parameter (the frequencies are float64; any
scaling of them is another vector). Tensor names under the mixer's prefix:
`q k v o`, `q.b k.b v.b`, `q.norm k.norm`.

The cache keeps every key of the sequence (a prompt may bring more tokens in one
step than a window holds); the kernels walk the window only.
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import numpy as np
import torch

from ..cache.store import KVRequest, KVView
from ..kernels import ops
from ..weights.loader import ExpectedTensor
from .base import Fetch, Part, register_mixer
from .linear import Linear
from .products import product_f32


@register_mixer("window_attention")
class WindowAttention(Part):
    replay_safe = True

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 eps: float, window: Optional[int] = None,
                 frequencies: Optional[Sequence[float]] = None, rot_factor: float = 1.0,
                 bias: bool = True, *, dtype: torch.dtype, device: torch.device):
        if kv_heads <= 0 or heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} key-value heads")
        if not 1 <= dim <= 1024 or not 1 <= vdim <= 256:
            raise ValueError(f"key size {dim} (at most 1024) and value size {vdim} (at most 256)")
        freq = np.asarray(() if frequencies is None else frequencies, dtype=np.float64)
        if 2 * freq.size > dim:
            raise ValueError(f"{2 * freq.size} rotated elements of heads of {dim}")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.scale, self.eps, self.window = float(scale), float(eps), int(window) if window else 0
        self.biased = bool(bias)
        self.dtype, self.device = dtype, device
        self.nq, self.nk, self.nv = heads * dim, kv_heads * dim, kv_heads * vdim
        self.rotation = ops.Rotation(freq, device, rot_factor)
        self.qkv = Linear(width, [("q", self.nq), ("k", self.nk), ("v", self.nv)], dtype=dtype,
                          device=device, suffix="")
        self.o = Linear(heads * vdim, [("o", width)], dtype=dtype, device=device, suffix="")
        self.q_norm = self.k_norm = self.bias = None

    def expected_tensors(self, prefix: str) -> Dict[str, ExpectedTensor]:
        out = {**self.qkv.expected_tensors(prefix), **self.o.expected_tensors(prefix),
               f"{prefix}.q.norm": ExpectedTensor((self.dim,)),
               f"{prefix}.k.norm": ExpectedTensor((self.dim,))}
        if self.biased:
            for name, n in (("q", self.nq), ("k", self.nk), ("v", self.nv)):
                out[f"{prefix}.{name}.b"] = ExpectedTensor((n,))
        return out

    def load(self, prefix: str, fetch: Fetch) -> None:
        self.qkv.load(prefix, fetch)
        self.o.load(prefix, fetch)
        self.q_norm = fetch(f"{prefix}.q.norm").to(torch.float32).contiguous()
        self.k_norm = fetch(f"{prefix}.k.norm").to(torch.float32).contiguous()
        if self.biased:  # joins the projections' 32-bit sums
            self.bias = torch.cat([fetch(f"{prefix}.{n}.b").to(torch.float32)
                                   for n in ("q", "k", "v")]).contiguous()

    def cache_request(self) -> KVRequest:
        return KVRequest(self.kv_heads, self.dim, None, self.vdim)

    def first_weight(self):
        return self.qkv.weight

    def context_flops(self, token_counts, starts) -> float:
        pairs = 0.0
        for n, start in zip(token_counts, starts):
            seen = np.arange(start + 1, start + n + 1, dtype=np.float64)
            pairs += float((np.minimum(seen, self.window) if self.window else seen).sum())
        return 2.0 * self.heads * (self.dim + self.vdim) * pairs

    # the pieces of a mixer that may stand beside another one (parts/parallel.py)
    def input_weight(self) -> torch.Tensor:
        return self.qkv.weight

    def output_weight(self) -> torch.Tensor:
        return self.o.weight

    @property
    def inner_size(self) -> int:
        return self.heads * self.vdim

    def between(self, ctx, p: torch.Tensor, cache: KVView, out: torch.Tensor,
                out_scale: float = 1.0) -> torch.Tensor:
        """From the projections `p` (float32 rows [q | k | v], biases still to be added) to the
        heads' outputs side by side in `out` (rows may lie further apart)."""
        if out_scale != 1.0:
            raise ValueError("window_attention: softmax outputs take no constant")
        table = ctx.page_table(cache.group)
        q = torch.empty((p.shape[0], self.nq), dtype=out.dtype, device=p.device)
        ops.head_norm_rope_cache_write(p, q, self.q_norm, self.k_norm, self.eps, False, ctx,
                                       self.rotation, table, cache.k, cache.v, self.heads,
                                       self.kv_heads, self.dim, self.vdim,
                                       write_cache=cache.writes, bias=self.bias)
        ops.attention_window(ctx, q, out, table, cache.k, cache.v, self.heads, self.kv_heads,
                             self.dim, self.vdim, self.scale, self.window,
                             then_reads=self.o.weight)
        return out

    def forward(self, ctx, x, cache: KVView):
        attn = torch.empty((x.shape[0], self.inner_size), dtype=x.dtype, device=x.device)
        self.between(ctx, product_f32(x, self.qkv.weight), cache, attn)
        return product_f32(attn, self.o.weight)
