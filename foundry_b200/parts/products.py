"""A product whose result feeds 32-bit arithmetic: float32 out, any shape."""
from __future__ import annotations

import torch

from ..kernels import ops
from .linear import matmul_nt

SMALL_K = 64  # below one K block of the tensor-core products the CUDA-core product runs


def product_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, K] @ w [N, K]^T accumulated and returned in float32. The operands
    are in the run's element type (bfloat16 products round nothing but their
    inputs). Low-rank projections (K below a tensor-core K block) and views
    that TMA cannot address take the CUDA-core product."""
    out = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32, device=x.device)
    if x.shape[0] == 0:
        return out
    if x.dtype == torch.float32 or x.shape[1] < SMALL_K:
        return ops.gemm_simt(ops.plain(x), w, out)
    y = matmul_nt(x, w, out)
    return y if isinstance(y, torch.Tensor) else out


def product_planes(x: torch.Tensor, w: torch.Tensor, then_reads=None):
    """`product_f32` for a consumer that sums split-K planes while it reads: float32 rows or
    `ops.Planes`."""
    if x.shape[0] == 0 or x.dtype == torch.float32 or x.shape[1] < SMALL_K:
        return product_f32(x, w)
    return matmul_nt(x, w, out_dtype=torch.float32, allow_planes=True, then_reads=then_reads)


def product_pair(x1: torch.Tensor, w1: torch.Tensor, x2: torch.Tensor, w2: torch.Tensor,
                 then_reads=None):
    """(x1 w1^T, x2 w2^T), each as `product_planes` gives it; a handful of tokens takes one
    launch for both."""
    if min(x1.shape[1], x2.shape[1]) >= SMALL_K and ops.skinny_pair_fits(x1, w1, x2, w2):
        return ops.gemm_skinny_pair(x1, w1, x2, w2, then_reads)
    return product_planes(x1, w1, then_reads=w2), product_planes(x2, w2, then_reads=then_reads)


def product_to_residual(ctx, x: torch.Tensor, w: torch.Tensor):
    """A part's last product, whose result joins the residual: float32 as
    `product_f32` gives it, or, where the block offers the next norm's sink
    (`ctx.residual_sink`, single-token steps in bfloat16), the sum and the norm's
    preparation made in the product's epilogue (an `ops.NormPending` comes back)."""
    sink = getattr(ctx, "residual_sink", None)
    if sink is None or x.dtype == torch.float32 or x.shape[1] < SMALL_K or x.shape[0] == 0:
        return product_f32(x, w)
    return matmul_nt(x, w, out_dtype=torch.float32, residual=sink,
                     then_reads=getattr(ctx, "reads_after_part", None))
