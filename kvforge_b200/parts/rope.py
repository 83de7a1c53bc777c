"""Rotary position encoding: the frequency table, with optional llama3 or YaRN scaling.

Frequencies as umarhassan-cloud/kvforge builds them (src/tokenvault/model.py:44):
``inv_freq[j] = 1 / theta^(2j/d)`` in 32-bit.  The angle ``float(pos) * inv_freq[j]`` and the
rotation of pair ``(j, j + d/2)`` (model.py:47-61) are computed in the kernel
(``csrc/elementwise.cu``), in 32-bit, from this table.

llama3 scaling is not in kvforge; Llama 3.1/3.2 checkpoints need it.  For wavelength
``lam = 2*pi/f`` and original context ``P``: ``lam < P/high`` keeps ``f``; ``lam > P/low`` gives
``f/factor``; between, ``s = (P/lam - low)/(high - low)`` blends ``(1-s)*f/factor + s*f``.

YaRN scaling ("YaRN: Efficient Context Window Extension of Large Language Models", Peng et al.) blends by the index of a pair
instead: the (fractional) pair whose wave turns ``t`` times within the original context ``P`` is ``rot ln(P / (2 pi t)) / (2 ln theta)``;
from the one of ``fast`` turns (rounded down) to the one of ``slow`` turns (rounded up) the frequencies go linearly from ``f`` to
``f/factor``.  What turns also grows by the encoding's ``magnitude``, ``1 + ln(factor) / 10``.
"""

from __future__ import annotations

import math

import torch

from .. import ops
from .base import PositionEncoding, WeightDecl, register_position_encoding


def rotary_inv_freq(rotary_dim: int, theta: float) -> torch.Tensor:
    return 1.0 / (theta ** (torch.arange(0, rotary_dim, 2, dtype=torch.float32) / rotary_dim))


def llama3_scale(inv_freq: torch.Tensor, factor: float, low_freq_factor: float, high_freq_factor: float, original_max_position: int) -> torch.Tensor:
    f = inv_freq.to(torch.float64)
    lam = 2.0 * math.pi / f
    smooth = (original_max_position / lam - low_freq_factor) / (high_freq_factor - low_freq_factor)
    blended = (1.0 - smooth) * f / factor + smooth * f
    out = torch.where(lam < original_max_position / high_freq_factor, f, blended)
    out = torch.where(lam > original_max_position / low_freq_factor, f / factor, out)
    return out.to(torch.float32)


def yarn_scale(rotary_dim: int, theta: float, factor: float, original: float, fast: float, slow: float) -> torch.Tensor:
    def pair_of(turns: float) -> float:
        return rotary_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))

    first, last = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), rotary_dim - 1)
    i = torch.arange(rotary_dim // 2, dtype=torch.float64)
    f = theta ** (-2.0 * i / rotary_dim)
    scaled = ((i - first) / max(last - first, 0.001)).clamp(0.0, 1.0)
    return (f / factor * scaled + f * (1.0 - scaled)).to(torch.float32)


@register_position_encoding("rotary")
class RotaryEmbedding(PositionEncoding):
    """params: ``head_dim``, ``theta``, optional ``rotary_dim`` (leading dims that turn;
    default all), ``scaling`` (``None``, the llama3 dict: ``factor``,
    ``low_freq_factor``, ``high_freq_factor``, ``original_max_position_embeddings``, or the YaRN dict: ``type: "yarn"``,
    ``factor``, ``original``, ``fast``, ``slow``) and
    ``interleaved`` (the pairs that turn are dims ``(2i, 2i+1)`` instead of ``(i, i + rot/2)``; a
    mixer asks ``pairs_interleaved`` and tells its kernel)."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.head_dim = int(params["head_dim"])
        self.rotary_dim = int(params.get("rotary_dim") or self.head_dim)
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.theta = float(params["theta"])
        self.scaling = params.get("scaling")
        self.pairs_interleaved = bool(params.get("interleaved", False))
        self.yarn = bool(self.scaling) and self.scaling.get("type") == "yarn"
        if self.yarn and (self.theta <= 1.0 or not all(float(self.scaling[k]) > 0 for k in ("factor", "original", "fast", "slow"))):
            raise ValueError("YaRN scaling needs a base above one and positive factor, original, fast and slow")
        if self.yarn:
            self.magnitude = 0.1 * math.log(float(self.scaling["factor"])) + 1.0

    def inv_freq_host(self) -> torch.Tensor:
        s = self.scaling
        if self.yarn:
            return yarn_scale(self.rotary_dim, self.theta, *(float(s[k]) for k in ("factor", "original", "fast", "slow")))
        inv = rotary_inv_freq(self.rotary_dim, self.theta)
        if s:
            inv = llama3_scale(
                inv,
                float(s["factor"]),
                float(s["low_freq_factor"]),
                float(s["high_freq_factor"]),
                int(s["original_max_position_embeddings"]),
            )
        return inv

    def bind(self, weights, rt):
        super().bind(weights, rt)
        self.inv_freq = self.inv_freq_host().to(rt.device).contiguous()

    def table(self) -> torch.Tensor:
        return self.inv_freq


@register_position_encoding("learned")
class LearnedPositions(PositionEncoding):
    """A learned vector per position, added to the residual stream after the embedding lookup.  params: ``rows`` (positions
    there are; a later one raises the device error flag), ``hidden_size``.  Tensor: ``weight [rows, hidden_size]``."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.rows, self.hidden = int(params["rows"]), int(params["hidden_size"])

    @classmethod
    def weight_decls(cls, params):
        return {"weight": WeightDecl((int(params["rows"]), int(params["hidden_size"])))}

    def bind(self, weights, rt):
        super().bind(weights, rt)
        self.weight = weights["weight"].contiguous()

    def embed(self, ctx, resid):
        ops.add_position_rows(resid, self.weight, ctx.positions, self.rt.err)
