"""Rotary position encoding."""

from __future__ import annotations

import math
from typing import Mapping

import torch

from ..errors import KernelError
from .base import POSITION_ENCODINGS, PositionEncoding, Runtime


@POSITION_ENCODINGS.register("rope")
class RotaryEmbedding(PositionEncoding):
    """``inv_freq[i] = 1 / theta^(2i / rotary_dim)``, built in float32 on the host
    with the same expression as the reference (mini_llm/nn/rope.py:37-40); the
    angle ``float32(position) * inv_freq[i]`` and its sine and cosine are formed
    in float32 inside the fused kernel (mini_llm/nn/rope.py:74-80).  Pairs are
    ``(i, i + rotary_dim/2)`` (mini_llm/nn/rope.py:110-114).  ``rotary_dim``
    smaller than the head size leaves the remaining columns unrotated.

    ``scaling`` (``factor``, ``low``, ``high``, ``original``) stretches long wavelengths: with ``l = 2 pi / f`` a frequency
    is kept where ``l < original / high``, divided by ``factor`` where ``l > original / low``, and in between blended as
    ``(1 - s) f / factor + s f`` with ``s = (original / l - low) / (high - low)`` (formed in float64, kept in float32).

    ``scaling`` (``factor``, ``original``, ``fast``, ``slow``; YaRN): pair ``i``'s frequency goes linearly in ``i`` from itself to
    itself divided by ``factor``, between the pair at which a wavelength fits ``fast`` times into ``original`` positions (rounded down,
    at least 0) and the one at which it fits ``slow`` times (rounded up, at most ``rotary_dim - 1``); cosine and sine are
    multiplied by ``0.1 ln(factor) + 1``.  ``interleaved``: pairs are ``(2i, 2i + 1)``.  Kernels that take either of these get
    them from ``rotary_layout``."""

    graph_safe = True

    def __init__(self, head_dim: int, theta: float, rotary_dim: int | None = None,
                 scaling: Mapping[str, float] | None = None, interleaved: bool = False) -> None:
        rotary_dim = head_dim if rotary_dim is None else rotary_dim
        if head_dim <= 0 or rotary_dim <= 0 or rotary_dim % 2 or rotary_dim > head_dim:
            raise ValueError(f"rope needs an even rotary_dim in (0, head_dim], got {rotary_dim}, {head_dim}")
        if theta <= 0:
            raise ValueError(f"rope theta must be positive, got {theta}")
        self.head_dim, self.theta, self.rotary_dim = head_dim, float(theta), rotary_dim
        self.scaling, self.interleaved, self.factor = None, bool(interleaved), 1.0
        if scaling and "fast" in scaling:
            self.scaling = {k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")}
            if min(self.scaling.values()) <= 0 or self.theta <= 1:
                raise ValueError(f"rope scaling needs factor, original, fast and slow > 0 and theta > 1, got {self.scaling}, {theta}")
            self.factor = 0.1 * math.log(self.scaling["factor"]) + 1.0
        elif scaling:
            self.scaling = {k: float(scaling[k]) for k in ("factor", "low", "high", "original")}
            if self.scaling["factor"] <= 0 or self.scaling["original"] <= 0 or not 0 < self.scaling["low"] < self.scaling["high"]:
                raise ValueError(f"rope scaling needs factor > 0, original > 0 and 0 < low < high, got {self.scaling}")
        self.inv_freq: torch.Tensor | None = None

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        self.runtime = runtime
        dims = torch.arange(0, self.rotary_dim, 2, dtype=torch.float32)
        if self.scaling is None:
            self.inv_freq = (1.0 / (self.theta ** (dims / self.rotary_dim))).to(runtime.device)
            return
        s = self.scaling
        if "fast" in s:
            self.inv_freq = torch.tensor(self._ramped(), dtype=torch.float64).to(torch.float32).to(runtime.device)
            return
        f = self.theta ** (-dims.to(torch.float64) / self.rotary_dim)
        wavelength = 2.0 * math.pi / f
        blend = (s["original"] / wavelength - s["low"]) / (s["high"] - s["low"])
        blended = (1.0 - blend) * f / s["factor"] + blend * f
        f = torch.where(wavelength < s["original"] / s["high"], f,
                        torch.where(wavelength > s["original"] / s["low"], f / s["factor"], blended))
        self.inv_freq = f.to(torch.float32).to(runtime.device)

    def _ramped(self) -> list[float]:
        s, dims = self.scaling, self.rotary_dim

        def pair_of(turns: float) -> float:
            return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        lo = max(math.floor(pair_of(s["fast"])), 0)
        hi = min(math.ceil(pair_of(s["slow"])), dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
        plain = [self.theta ** (-2.0 * i / dims) for i in range(dims // 2)]
        return [f / s["factor"] * r + f * (1.0 - r) for f, r in zip(plain, ramp)]

    def rotary_parameters(self) -> tuple[torch.Tensor, int]:
        if self.interleaved or self.factor != 1.0:
            raise KernelError("this mixer's kernels rotate pairs (i, i + rotary_dim / 2) without a factor only")
        return self.inv_freq, self.rotary_dim

    def rotary_layout(self) -> tuple[torch.Tensor, int, bool, float]:
        return self.inv_freq, self.rotary_dim, self.interleaved, self.factor
