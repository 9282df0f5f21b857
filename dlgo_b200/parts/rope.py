"""Rotary position encoding: cos/sin tables built once from constants.

Reference: ``theta_i = base^(-2i/rotary_dim)``, ``angle = pos * theta_i`` in
float64, cos and sin cast to float32, one row per position
(models/llm/workers.go:147-171); only the first ``rotary_dim`` dims of a head
are rotated (workers.go:151-159).  Pairing: ``split_half`` pairs (i, i+rot/2),
``interleaved`` pairs (2i, 2i+1) (ops/rope.go:21-31); which one is right is a
property of the weight layout, so it is a parameter.

The llama3 scaling of the frequencies is not in the reference (it has no rope
scaling at all); it follows the published Llama 3.1 rule: with wavelength
``lam = 2*pi/f``, frequencies with ``lam < orig/high`` are kept, those with
``lam > orig/low`` are divided by ``factor``, and those between are blended by
``s = (orig/lam - low) / (high - low)``: ``f <- (1-s) * f/factor + s * f``.

Linear scaling (``rope_type`` "linear": ``factor``) divides every frequency: ``f_i <- f_i / factor``.

YaRN scaling (``rope_type`` "yarn": ``factor``, ``original_max_position_embeddings``, ``beta_fast``,
``beta_slow``) blends by the pair's index instead.  With ``where(t) = rot * ln(orig / (2 pi t)) / (2 ln base)`` (the
index whose pair makes t turns over the original context), ``lo = max(floor(where(beta_fast)), 0)``,
``hi = min(ceil(where(beta_slow)), rot - 1)`` and ``r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1)``:
``f_i <- r_i * f_i / factor + (1 - r_i) * f_i``; cosine and sine are multiplied by ``0.1 ln(factor) + 1``
(:func:`rotary_amplitude`).
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

from .base import PositionEncoding
from .registry import POSITION_ENCODINGS


def rotary_frequencies(rotary_dim: int, theta: float, scaling: Optional[Dict[str, Any]]) -> List[float]:
    half = rotary_dim // 2
    freqs = [1.0 / math.pow(theta, (2 * i) / rotary_dim) for i in range(half)]
    if not scaling:
        return freqs
    kind = scaling.get("rope_type", "llama3")
    if kind == "yarn":
        factor = float(scaling["factor"])
        orig = float(scaling["original_max_position_embeddings"])

        def where(turns: float) -> float:
            return rotary_dim * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
        lo = max(math.floor(where(float(scaling["beta_fast"]))), 0)
        hi = min(math.ceil(where(float(scaling["beta_slow"]))), rotary_dim - 1)
        out = []
        for i, f in enumerate(freqs):
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out.append(f / factor * r + f * (1.0 - r))
        return out
    if kind == "linear":
        return [f / float(scaling["factor"]) for f in freqs]
    if kind != "llama3":
        raise ValueError(f"rotary scaling {kind!r} is not supported")
    factor = float(scaling["factor"])
    low = float(scaling["low_freq_factor"])
    high = float(scaling["high_freq_factor"])
    orig = float(scaling["original_max_position_embeddings"])
    out = []
    for f in freqs:
        lam = 2.0 * math.pi / f
        if lam < orig / high:
            out.append(f)
        elif lam > orig / low:
            out.append(f / factor)
        else:
            s = (orig / lam - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def rotary_amplitude(scaling: Optional[Dict[str, Any]]) -> float:
    """The factor on cosine and sine that a scaling rule brings with it (YaRN: ``0.1 ln(factor) + 1``; else 1)."""
    if scaling and scaling.get("rope_type") == "yarn":
        return 0.1 * math.log(float(scaling["factor"])) + 1.0
    return 1.0


class RotaryEmbedding(PositionEncoding):
    def __init__(self, head_dim: int, rotary_dim: int, theta: float, max_positions: int,
                 pairing: str = "split_half", scaling: Optional[Dict[str, Any]] = None):
        super().__init__(head_dim=head_dim, rotary_dim=rotary_dim, theta=theta, max_positions=max_positions,
                         pairing=pairing, scaling=scaling)
        if rotary_dim % 2 or not 0 < rotary_dim <= head_dim:
            raise ValueError(f"rotary_dim must be even and in (0, head_dim], got {rotary_dim} for head_dim {head_dim}")
        if pairing not in ("split_half", "interleaved"):
            raise ValueError(f"pairing must be 'split_half' or 'interleaved', got {pairing!r}")
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim)
        self.theta = float(theta)
        self.max_positions = int(max_positions)
        self.interleaved = pairing == "interleaved"
        self.scaling = dict(scaling) if scaling else None
        self.cos: Optional[torch.Tensor] = None
        self.sin: Optional[torch.Tensor] = None

    def tables(self) -> tuple[torch.Tensor, torch.Tensor]:
        """(cos, sin), each ``[max_positions, rotary_dim/2]`` float32 on the CPU."""
        f = torch.tensor(rotary_frequencies(self.rotary_dim, self.theta, self.scaling), dtype=torch.float64)
        pos = torch.arange(self.max_positions, dtype=torch.float64)
        ang = pos[:, None] * f[None, :]
        a = rotary_amplitude(self.scaling)
        return (torch.cos(ang) * a).to(torch.float32), (torch.sin(ang) * a).to(torch.float32)

    def prepare(self, runtime: Any) -> None:
        c, s = self.tables()
        self.cos = c.contiguous().to(runtime.device)
        self.sin = s.contiguous().to(runtime.device)


class RotaryFrequencies(PositionEncoding):
    """Rotary positions without tables: only the frequencies ``f_i = theta^(-2i/rotary_dim)`` (float64, rounded
    to float32) are kept; a kernel that rotates forms the angle ``float(position) * f_i`` in fp32 and takes its
    cosine and sine itself, so no context limit is built in.  ``pairing``: ``split_half`` pairs (i, i + rotary_dim/2),
    ``interleaved`` pairs (2i, 2i + 1); a kernel takes the one it is written for.  :attr:`amplitude` is the factor
    on cosine and sine that the scaling rule brings (1 without one)."""

    def __init__(self, head_dim: int, rotary_dim: int, theta: float, scaling: Optional[Dict[str, Any]] = None,
                 pairing: str = "split_half"):
        super().__init__(head_dim=head_dim, rotary_dim=rotary_dim, theta=theta, scaling=scaling, pairing=pairing)
        if pairing not in ("split_half", "interleaved"):
            raise ValueError(f"pairing must be 'split_half' or 'interleaved', got {pairing!r}")
        if rotary_dim % 2 or not 0 < rotary_dim <= head_dim:
            raise ValueError(f"rotary_dim must be even and in (0, head_dim], got {rotary_dim} for head_dim {head_dim}")
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim)
        self.theta = float(theta)
        self.interleaved = pairing == "interleaved"
        self.scaling = dict(scaling) if scaling else None
        self.amplitude = rotary_amplitude(self.scaling)
        self.frequencies: Optional[torch.Tensor] = None

    def prepare(self, runtime: Any) -> None:
        f = torch.tensor(rotary_frequencies(self.rotary_dim, self.theta, self.scaling), dtype=torch.float64)
        self.frequencies = f.to(torch.float32).contiguous().to(runtime.device)


POSITION_ENCODINGS.register("rotary", RotaryEmbedding)
POSITION_ENCODINGS.register("rotary_frequencies", RotaryFrequencies)
