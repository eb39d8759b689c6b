"""Rotary position encodings: the frequency vector is the part.

The rotation itself runs inside the mixer's kernel, which takes the inverse
frequencies, the rotary width and the pairing as parameters (`pairing = "half"`:
frequency i turns elements i and i + width/2, the reference's; "interleaved":
elements 2i and 2i + 1); a variant of the encoding is another frequency vector
and, if it pairs otherwise, another `pairing` attribute.

inv_freq[j] = 1 / theta^(2j / D), j = 0 .. D/2, in 32-bit
(src/models/llama/rotary_emb.rs:135-160). The "llama3" scaling
(rotary_emb.rs:162-183) leaves short wavelengths as they are, divides long
ones by `factor`, and blends between the two bands:

    wavelen = 2*pi / f;  low_wl = ctx / low_freq_factor;  high_wl = ctx / high_freq_factor
    f' = f / factor if wavelen > low_wl else f
    smooth = (ctx / wavelen - low_freq_factor) / (high_freq_factor - low_freq_factor)
    f'' = (1 - smooth) * f' / factor + smooth * f'   if high_wl <= wavelen <= low_wl else f'
"""
from __future__ import annotations

import math

import numpy as np
import torch

from .base import Part, register_position_encoding

F = np.float32


def plain_inv_freq(head_dim: int, theta: float) -> np.ndarray:
    if head_dim <= 0 or head_dim % 2:
        raise ValueError(f"rotary width {head_dim} is not a positive even number")
    exponents = np.arange(0, head_dim, 2, dtype=F) / F(head_dim)
    return (F(1.0) / np.power(F(theta), exponents, dtype=F)).astype(F)


def llama3_inv_freq(head_dim: int, theta: float, factor: float, low_freq_factor: float,
                    high_freq_factor: float, original_max_position_embeddings: int) -> np.ndarray:
    f = plain_inv_freq(head_dim, theta)
    ctx = F(original_max_position_embeddings)
    factor, low, high = F(factor), F(low_freq_factor), F(high_freq_factor)
    low_wl, high_wl = ctx / low, ctx / high
    wavelen = F(2.0 * math.pi) / f
    scaled = np.where(wavelen > low_wl, f / factor, f).astype(F)
    smooth = ((ctx / wavelen - low) / (high - low)).astype(F)
    medium = (wavelen >= high_wl) & (wavelen <= low_wl)
    blended = ((F(1.0) - smooth) * scaled / factor + smooth * scaled).astype(F)
    return np.where(medium, blended, scaled).astype(F)


def banded_frequencies(dims: int, base: float, factor: float = 1.0, low: float = 1.0,
                       high: float = 1.0, original: float = 0.0) -> np.ndarray:
    """float64 frequencies f_i = base^(-2i / dims), i < dims / 2, for kernels that make the
    angle as a 64-bit product with the position. With `original` > 0 they are scaled by
    wavelength l = 2 pi / f in three bands: kept where l < original / high; f / factor
    where l > original / low; between the two blended,
    s = (original / l - low) / (high - low),  f' = (1 - s) f / factor + s f."""
    if dims < 0 or dims % 2:
        raise ValueError(f"rotary width {dims} is not an even number")
    f = np.power(np.float64(base), -2.0 * np.arange(dims // 2, dtype=np.float64) / max(1, dims))
    if not original:
        return f
    wavelength = 2.0 * math.pi / f
    with np.errstate(divide="ignore", invalid="ignore"):
        blend = (original / wavelength - low) / (high - low) if high != low else np.ones_like(f)
    mixed = (1.0 - blend) * f / factor + blend * f
    return np.where(wavelength < original / high, f,
                    np.where(wavelength > original / low, f / factor, mixed))


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float,
                     slow: float):
    """(float64 frequencies f_i, i < dims / 2; the factor on cosines and sines) of YaRN's
    scaling. An element whose wavelength makes t turns in `original` positions is number
    e(t) = dims ln(original / (2 pi t)) / (2 ln base). Elements in front of e(fast) (rounded
    down) keep base^(-2i / dims), those behind e(slow) (rounded up) are divided by `factor`,
    and between the two the frequencies are blended linearly in i."""
    f = banded_frequencies(dims, base)

    def element(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(element(fast)), 0)
    last = min(math.ceil(element(slow)), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - first) / max(last - first, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


class _Rotary(Part):
    attention_factor = 1.0
    pairing = "half"  # src/models/llama/rotary_emb.rs:76-85 (rotate_half)

    def _finish(self, inv_freq: np.ndarray, device: torch.device) -> None:
        self.rotary_dim = 2 * int(inv_freq.shape[0])
        self.inv_freq_host = inv_freq
        self.inv_freq = torch.from_numpy(inv_freq.copy()).to(device)


@register_position_encoding("rope")
class Rope(_Rotary):
    def __init__(self, head_dim: int, theta: float, *, dtype=None, device=None):
        self._finish(plain_inv_freq(head_dim, theta), device)


@register_position_encoding("rope_llama3")
class RopeLlama3(_Rotary):
    def __init__(self, head_dim: int, theta: float, factor: float, low_freq_factor: float,
                 high_freq_factor: float, original_max_position_embeddings: int, *,
                 dtype=None, device=None):
        self._finish(llama3_inv_freq(head_dim, theta, factor, low_freq_factor, high_freq_factor,
                                     original_max_position_embeddings), device)
