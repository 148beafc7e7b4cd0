"""Position encodings that act on queries and keys before the keys are cached.

``RotaryHalves`` is the reference's RoPE (edgerag/core/layers.py:63-114): ``inv_freq[j] =
1 / theta**(2j / D)`` built exactly as there (int64 arange, float32 division and power), angles
``position * inv_freq`` in float32, and the halves convention ``[-x2, x1]``.  The rotation runs in
the same kernel that writes keys and values to their cache slots, so the cache holds rotated keys
(edgerag/core/layers.py:301-306) and a key's encoding depends on its own logical position only.

``RotaryPairs`` turns neighbouring pairs ``(2i, 2i + 1)`` of the first ``rot_dim`` entries of a head by
``position * theta**(-2i / rot_dim) / factor`` (``factor``: linear scaling of positions) and leaves the rest
of the head as it is.

``NoPosition`` encodes nothing and only writes the cache; it is what a mixer uses when another
part has already put positions into the stream.
"""

from __future__ import annotations

import math

import torch

from ..ops import kernels
from .base import PositionEncoding, register_part


def rotary_frequencies(base: float, dims: int, scaling: dict | None = None) -> torch.Tensor:
    """``f_i = base^(-2i / dims)`` for ``i < dims / 2``, made in float64.  ``scaling = {factor, low, high, original}``
    stretches the long wavelengths: with ``l = 2 pi / f``, a frequency stays where ``l < original / high``, becomes
    ``f / factor`` where ``l > original / low``, and in between is the blend ``(1 - s) f / factor + s f`` with
    ``s = (original / l - low) / (high - low)``.

    ``scaling = {factor, original, fast, slow}`` (YaRN, Peng et al. 2023) tells the pairs apart by the turns they make within
    ``original`` positions: ``pair(t) = dims * ln(original / (2 pi t)) / (2 ln base)`` is the pair that makes ``t`` turns; up
    to ``lo = max(floor(pair(fast)), 0)`` a frequency stays, from ``hi = min(ceil(pair(slow)), dims - 1)`` on it becomes
    ``f / factor``, between them the two are blended linearly in ``i``.  (Its other half is ``rotary_multiplier``.)"""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / max(dims, 1))
    if scaling and "fast" in scaling:
        factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
        if not (factor > 0 and original > 0 and fast > 0 and slow > 0) or base <= 0 or base == 1:
            raise ValueError("rotary scaling needs positive factor, original, fast and slow, and a base other than 1")
        pair = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))   # noqa: E731
        lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        f = f / factor * ramp + f * (1.0 - ramp)
    elif scaling:
        factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
        if not (factor > 0 and high > low and original > 0):
            raise ValueError("rotary scaling needs factor > 0, high > low and original > 0")
        wavelength = 2.0 * math.pi / f
        s = ((original / wavelength - low) / (high - low)).clamp(0.0, 1.0)
        blend = (1.0 - s) * f / factor + s * f
        f = torch.where(wavelength < original / high, f, torch.where(wavelength > original / low, f / factor, blend))
    return f


def rotary_multiplier(scaling: dict | None) -> float:
    """What a scaled rotation multiplies cosines and sines by: ``0.1 ln(factor) + 1`` for ``{factor, original, fast, slow}``,
    1 for everything else."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and "fast" in scaling else 1.0


@register_part("position", "rope_halves")
class RotaryHalves(PositionEncoding):
    graph_safe = True
    pairs = False            # which entries make a pair: (i, i + rot_dim / 2)

    def __init__(self, head_dim: int, theta: float, dtype: torch.dtype, device: torch.device,
                 rot_dim: int | None = None, precise: bool = False) -> None:
        """``precise``: the frequencies ``theta ** (-2j / rot_dim)`` are made in float64 and rounded to float32 once
        (otherwise in float32 arithmetic, as the Llama decoder's reference does)."""
        self.head_dim = head_dim
        self.rot_dim = head_dim if rot_dim is None else rot_dim
        if self.rot_dim % 2 or not 0 < self.rot_dim <= head_dim:
            raise ValueError(f"rot_dim {self.rot_dim} must be even and at most head_dim {head_dim}")
        self.theta = float(theta)
        if precise:
            inv_freq = self.theta ** (-torch.arange(0, self.rot_dim, 2, dtype=torch.float64) / self.rot_dim)
        else:
            inv_freq = 1.0 / (self.theta ** (torch.arange(0, self.rot_dim, 2, dtype=torch.int64).float() / self.rot_dim))
        self.inv_freq = inv_freq.to(device=device, dtype=torch.float32).contiguous()

    def apply_and_store(self, qkv, ctx, n_q_heads, n_kv_heads, head_dim, pages, slots) -> None:
        k_pages, v_pages = pages if pages is not None else (None, None)
        kernels.rope_cache_write(
            qkv, ctx.positions, self.inv_freq, n_q_heads, n_kv_heads, head_dim, self.rot_dim,
            slots=slots, k_pages=k_pages, v_pages=v_pages, page_size=ctx.page_size)

    def project_apply_store(self, x, w_qkv, qkv, ctx, n_q_heads, n_kv_heads, head_dim, pages, slots) -> bool:
        """A few rows (a decode step): the rotation and the cache write ride in the product's epilogue."""
        if pages is None or slots is None or not kernels.linear_rope_store_supported(x, w_qkv, head_dim, self.rot_dim):
            return False
        kernels.linear_rope_store(x, w_qkv, qkv, ctx.positions, self.inv_freq, n_q_heads, n_kv_heads, head_dim,
                                  slots, pages[0], pages[1], ctx.page_size)
        return True


@register_part("position", "rope_pairs")
class RotaryPairs(PositionEncoding):
    graph_safe = True
    pairs = True             # (2i, 2i + 1)

    def __init__(self, head_dim: int, theta: float, dtype: torch.dtype, device: torch.device, rot_dim: int | None = None,
                 factor: float = 1.0) -> None:
        self.head_dim = head_dim
        self.rot_dim = head_dim if rot_dim is None else int(rot_dim)
        if self.rot_dim % 2 or not 0 <= self.rot_dim <= head_dim:
            raise ValueError(f"rot_dim {self.rot_dim} must be even and at most head_dim {head_dim}")
        if not factor > 0:
            raise ValueError(f"scaling factor {factor} must be positive")
        self.theta, self.factor = float(theta), float(factor)
        i = torch.arange(self.rot_dim // 2, dtype=torch.float64)
        inv_freq = self.theta ** (-2.0 * i / max(self.rot_dim, 1)) / self.factor
        self.inv_freq = inv_freq.to(device=device, dtype=torch.float32).contiguous()

    def apply_and_store(self, qkv, ctx, n_q_heads, n_kv_heads, head_dim, pages, slots) -> None:
        k_pages, v_pages = pages if pages is not None else (None, None)
        kernels.qk_prepare(qkv, ctx.positions, n_q_heads, n_kv_heads, head_dim, inv_freq=self.inv_freq, rot_dim=self.rot_dim,
                           pairs=True, slots=slots, k_pages=k_pages, v_pages=v_pages, page_size=ctx.page_size)


@register_part("position", "none")
class NoPosition(PositionEncoding):
    graph_safe = True
    pairs = False
    rot_dim = 0
    inv_freq = None

    def __init__(self, dtype: torch.dtype, device: torch.device, **_unused) -> None:
        pass

    def apply_and_store(self, qkv, ctx, n_q_heads, n_kv_heads, head_dim, pages, slots) -> None:
        if pages is None:
            return
        kernels.rope_cache_write(qkv, ctx.positions, None, n_q_heads, n_kv_heads, head_dim, 0,
                                 slots=slots, k_pages=pages[0], v_pages=pages[1], page_size=ctx.page_size)
