"""Rotary positions: tables of cos and sin (optionally with scaled frequencies), and the per-head preparation of queries and keys (norm with
a weight, rotation, norm without one, cache write) in one launch of ``csrc/rotary.cu``.  CPU tensors run the restatement here."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Union

import torch

from .. import _native

_TABLES = {}


@dataclass(frozen=True)
class YarnScaling:
    """Frequencies of pairs that turn less than ``slow`` times within ``original`` positions are divided by ``factor``, those that turn
    more than ``fast`` times are kept, with a linear ramp over the pairs between them; cos and sin grow by ``0.1 ln(factor) + 1``."""
    factor: float
    original: float
    fast: float
    slow: float

    @staticmethod
    def from_json(c: Optional[dict]) -> Optional["YarnScaling"]:
        return YarnScaling(*(float(c[n]) for n in ("factor", "original", "fast", "slow"))) if c else None

    def pair_of(self, turns: float, base: float, dims: int) -> float:
        """(Fractional) pair that makes ``turns`` turns within the original length."""
        return dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(base))

    def apply(self, freqs: torch.Tensor, base: float, dims: int) -> torch.Tensor:
        lo = max(math.floor(self.pair_of(self.fast, base, dims)), 0)
        hi = min(math.ceil(self.pair_of(self.slow, base, dims)), dims - 1)
        ramp = ((torch.arange(freqs.numel(), dtype=freqs.dtype) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        return freqs / self.factor * ramp + freqs * (1 - ramp)

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0


@dataclass(frozen=True)
class BandScaling:
    """Frequencies whose wavelength is longer than ``original / low`` are divided by ``factor``, those below ``original / high`` are kept;
    between the two bounds the scaled and the kept frequency are mixed linearly in ``original / wavelength``.  cos and sin keep their size."""
    factor: float
    original: float
    low: float
    high: float
    amplitude = 1.0

    @staticmethod
    def from_json(c: Optional[dict]) -> Optional["BandScaling"]:
        return BandScaling(*(float(c[n]) for n in ("factor", "original", "low", "high"))) if c else None

    def apply(self, freqs: torch.Tensor, base: float, dims: int) -> torch.Tensor:
        turns = self.original * freqs / (2 * math.pi)         # within the original length
        keep = (turns > self.high).to(freqs.dtype)
        if self.high > self.low:
            keep = ((turns - self.low) / (self.high - self.low)).clamp(0, 1)
        return (1 - keep) * freqs / self.factor + keep * freqs


def rope_table(base: float, dims: int, width: int, positions: int, device,
               scaling: Union[YarnScaling, BandScaling, None] = None) -> torch.Tensor:
    """fp32 [positions, width]: cos and sin of ``p * base^(-2 i / dims)`` for pair i at columns (2 i, 2 i + 1), computed in fp64;
    columns from ``dims`` on (padding) are zero.  One table per rotation and device, grown when more positions are needed."""
    key = (float(base), int(dims), int(width), str(device), scaling)
    t = _TABLES.get(key)
    if t is None or t.shape[0] < positions:
        f = float(base) ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
        amp = 1.0
        if scaling is not None:
            f, amp = scaling.apply(f, float(base), int(dims)), scaling.amplitude
        a = torch.arange(positions, dtype=torch.float64)[:, None] * f
        t = torch.zeros(positions, width, dtype=torch.float32)
        t[:, :dims] = (torch.stack([a.cos(), a.sin()], dim=-1) * amp).reshape(positions, dims).float()
        t = _TABLES[key] = t.to(device)
    return t


def rotate_pairs(x: torch.Tensor, cs: torch.Tensor, interleaved: bool) -> torch.Tensor:
    """fp32 restatement: the leading ``cs.shape[-1]`` elements of ``x`` turn, the rest passes."""
    n = cs.shape[-1]
    c, s = cs[..., 0::2], cs[..., 1::2]
    head, rest = x[..., :n], x[..., n:]
    u, v = (head[..., 0::2], head[..., 1::2]) if interleaved else (head[..., :n // 2], head[..., n // 2:])
    a, b = u * c - v * s, v * c + u * s
    head = torch.stack([a, b], dim=-1).flatten(-2) if interleaved else torch.cat([a, b], dim=-1)
    return torch.cat([head, rest], dim=-1)


def head_prep(z: torch.Tensor, heads: int, kv_heads: int, dim: int, dim_real: int, q_w: Optional[torch.Tensor],
              k_w: Optional[torch.Tensor], unit: bool, eps: float, cos_sin: torch.Tensor, rot: int, interleaved: bool,
              pos: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
    """``z`` [T, >= (H + 2 G) D] holds q, k, v of heads padded to ``dim``.  Returns the queries [T, H, D]; keys and values go to rows
    ``rows`` (int64 [T], negative: not stored) of the caches (viewed as [rows, G, D]).  Per head of q and k: RMS norm with the fp32
    weight ``q_w`` / ``k_w`` [D] (None: no norm), rotation of the first ``rot`` elements to ``pos`` (``interleaved``: neighbours form
    the pairs, else element i and i + rot / 2), and with ``unit`` an RMS norm without a weight; means run over ``dim_real``."""
    H, G, D = int(heads), int(kv_heads), int(dim)
    if _native.use_native(z, k_cache):
        return _native.load(True).head_prep(z, H, G, D, int(dim_real), q_w, k_w, bool(unit), float(eps), cos_sin, int(rot),
                                            bool(interleaved), pos, k_cache, v_cache, rows)
    T = z.shape[0]
    q, k, v = z[:, :(H + 2 * G) * D].float().split([H * D, G * D, G * D], dim=1)
    cs = cos_sin[pos][:, None, :rot]

    def norm(x):
        return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) / dim_real + eps)

    def prep(x, n, w):
        x = x.reshape(T, n, D)
        if w is not None:
            x = norm(x) * w
        x = rotate_pairs(x, cs, interleaved)
        return (norm(x) if unit else x).to(z.dtype)

    ok = rows >= 0
    k_cache.view(-1, G, D)[rows[ok]] = prep(k, G, k_w)[ok]
    v_cache.view(-1, G, D)[rows[ok]] = v.reshape(T, G, D)[ok].to(z.dtype)
    return prep(q, H, q_w)
