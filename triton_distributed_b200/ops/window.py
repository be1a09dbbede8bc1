"""Attention over a sliding window: position i sees the positions j with ``0 <= i - j < window`` (0: every j <= i).

Two kinds of weights, each a value of its own class:

* :class:`SigmoidWeights`: ``sigmoid(scale q . k + bias[head, i - j])``, not normalised over the keys; the distance table holds whatever
  depends on the distance and the head (see :func:`distance_table`).
* :class:`DifferentialWeights`: two softmax maps over the same values, ``o = a1 - lam a2``, then ``RMSNorm(o) * out_scale``.

An output gate of one number per head may follow.  A sequence keeps its last ``min(window, max_length)`` tokens in a ring; prompts read a
packed copy (``models.kv_cache.WindowPlan``).  GPU forms: ``csrc/window_attn_sm100.cu`` (tcgen05, prompts), ``csrc/window_attn.cu``
(decode; fp32 arithmetic for 32-bit models and other head sizes), ``csrc/qkv_prep.cu``.  CPU tensors run the restatement here.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch

from .. import _native
from .attention import _PENDING_ERRORS, _decode_counters, check_attention_errors

WINDOW_DIMS = (64, 128)        # head dims (of a map) and value dims of the tensor-core kernels
WINDOW_MAX_DIM = 1024          # of the simple kernel


@dataclass
class SigmoidWeights:
    bias: torch.Tensor         # fp32 [heads, distances], added to the score
    maps = 1

    def _native(self):
        return self.bias, 0.0, 1.0, 0.0, 1


@dataclass
class DifferentialWeights:
    lam: float                 # of the second map
    out_scale: float
    eps: float
    dv_real: int               # divisor of the norm when values are padded
    maps = 2

    def _native(self):
        return None, float(self.lam), float(self.out_scale), float(self.eps), int(self.dv_real)


def distance_table(r1: torch.Tensor, r2: torch.Tensor, offset: torch.Tensor, distances: int) -> torch.Tensor:
    """fp32 [heads, distances]: ``offset_h - r1_h ln(1 + r2_h d)``, computed in fp64 on the host."""
    d = torch.arange(distances, dtype=torch.float64)
    r1, r2, off = (t.detach().double().cpu().reshape(-1, 1) for t in (r1, r2, offset))
    return (off - r1 * torch.log1p(r2 * d)).float().contiguous()


def qkv_prep(z: torch.Tensor, q_heads: int, k_heads: int, v_heads: int, dk: int, dv: int, bias: Optional[torch.Tensor],
             norms: Optional[Tuple[torch.Tensor, torch.Tensor, int, int]], eps: float, cos_sin: Optional[torch.Tensor], rot: int, pos: torch.Tensor,
             dest: Tuple[torch.Tensor, torch.Tensor, torch.Tensor], dest2: Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]] = None,
             sumsq: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``z`` [T, >= q | k | v] of heads padded to ``dk`` / ``dv``.  Adds ``bias`` (fp32, over q | k | v), norms the whole of q and the whole of k
    (``norms = (q weight, k weight, real size of q, of k)``; ``sumsq`` fp32 [T, 2]: their sums of squares when other ranks hold a part), turns the
    first ``rot`` elements of every head of q and k (element i with i + rot / 2, angles from ``cos_sin``) and returns the queries
    [T, q_heads, dk]; keys and values go to rows ``rows`` (int64, negative: not stored) of ``dest = (k, v, rows)`` and of ``dest2``."""
    Hq, Gk, G = int(q_heads), int(k_heads), int(v_heads)
    qw, kw, nq, nk = norms if norms is not None else (None, None, 1, 1)
    if _native.use_native(z, dest[0]):
        return _native.load(True).qkv_prep(z, Hq, Gk, G, int(dk), int(dv), bias, qw, kw, int(nq), int(nk), sumsq, float(eps), cos_sin, int(rot), pos, *dest,
                                           *(dest2 if dest2 is not None else (None, None, None)))
    T, n = z.shape[0], (Hq + Gk) * dk + G * dv
    x = z[:, :n].float()
    if bias is not None:
        x = x + bias
    q, k, v = x.split([Hq * dk, Gk * dk, G * dv], dim=1)
    if norms is not None:
        ss = torch.stack([q.pow(2).sum(-1), k.pow(2).sum(-1)], dim=1) if sumsq is None else sumsq
        q = q * torch.rsqrt(ss[:, :1] / nq + eps) * qw
        k = k * torch.rsqrt(ss[:, 1:] / nk + eps) * kw
    q, k, v = q.reshape(T, Hq, dk), k.reshape(T, Gk, dk), v.reshape(T, G, dv)
    if rot:
        from .rotary import rotate_pairs
        cs = cos_sin[pos][:, None, :rot]
        q, k = rotate_pairs(q, cs, False), rotate_pairs(k, cs, False)
    for place in (dest, dest2):
        if place is None:
            continue
        kc, vc, rows = place
        ok = rows >= 0
        kc.view(-1, Gk, dk)[rows[ok]] = k[ok].to(z.dtype)
        vc.view(-1, G, dv)[rows[ok]] = v[ok].to(z.dtype)
    return q.to(z.dtype)


def _restatement(q, k, v, weights, scale, gate, row0, n_keys, newest):
    T, G, dk, dv = q.shape[0], v.shape[-2], q.shape[-1], v.shape[-1]
    m = weights.maps
    H = q.shape[1] // m
    kf, vf = k.reshape(-1, G, m, dk), v.reshape(-1, G, dv)
    out = torch.empty(T, H, dv)
    for t in range(T):
        lo, n, new = int(row0[t]), int(n_keys[t]), int(newest[t])
        kk = kf[lo:lo + n].float().repeat_interleave(H // G, dim=1)
        vv = vf[lo:lo + n].float().repeat_interleave(H // G, dim=1)
        s = torch.einsum("hmd,nhmd->mhn", q[t].float().reshape(H, m, dk), kk) * scale
        if m == 1:
            dist = torch.remainder(new - torch.arange(n), n).clamp(max=weights.bias.shape[1] - 1)
            out[t] = torch.einsum("hn,nhd->hd", torch.sigmoid(s[0] + weights.bias[:, dist]), vv)
        else:
            a = torch.einsum("mhn,nhd->mhd", torch.softmax(s, dim=-1), vv)
            o = a[0] - weights.lam * a[1]
            out[t] = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / weights.dv_real + weights.eps) * weights.out_scale
    if gate is not None:
        out = out * torch.sigmoid(gate[:, :H].float()).unsqueeze(-1)
    return out.to(q.dtype)


Weights = Union[SigmoidWeights, DifferentialWeights]


def window_attention_simple(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, weights: Weights, scale: float, gate: Optional[torch.Tensor],
                            row0: torch.Tensor, n_keys: torch.Tensor, newest: torch.Tensor) -> torch.Tensor:
    """fp32 arithmetic for head dims up to ``WINDOW_MAX_DIM`` and bf16 or fp32 tensors: ``q`` [T, H maps, dk], ``k`` [.., G maps, dk], ``v``
    [.., G, dv] -> [T, H, dv].  Token t sees the rows ``row0[t] .. + n_keys[t]``; row ``row0 + newest`` is its own, rows after it are the oldest
    ones of a ring.  ``gate`` [T, >= H]: its sigmoid multiplies a head."""
    if _native.use_native(q, k, v):
        return _native.load(True).window_simple(q, k, v, float(scale), *weights._native(), gate, row0, n_keys, newest)
    return _restatement(q, k, v, weights, scale, gate, row0, n_keys, newest)


def window_tensor_cores(q: torch.Tensor, v: torch.Tensor, scale: float) -> bool:
    return q.is_cuda and q.dtype == torch.bfloat16 and q.shape[-1] in WINDOW_DIMS and v.shape[-1] in WINDOW_DIMS and scale > 0


def pick_window_splits(batch: int, units: int, rows: int, num_sms: int = 148) -> int:
    """KV splits of :func:`window_attention_decode`; ``units``: CTAs per sequence and split.  Makes the longest way of a CTA slot short, in
    64-token blocks: waves of three CTAs per SM, each with its blocks and what starting and merging cost (about one and a half blocks per
    CTA, and a little per split); at most 32."""
    blocks, ctas = max(1, (rows + 63) // 64), max(1, batch * units)

    def cost(splits):
        return math.ceil(splits * ctas / (3 * num_sms)) * (math.ceil(blocks / splits) + 1.5) + 0.15 * splits

    return min(range(1, min(blocks, 32) + 1), key=cost)


def window_attention_decode(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, weights: Weights, scale: float, gate: Optional[torch.Tensor],
                            slots: torch.Tensor, pos: torch.Tensor, splits: int = -1) -> torch.Tensor:
    """One token per sequence over the rings ``k`` [slots, R, G maps, dk] and ``v`` [slots, R, G, dv] (GPU, bf16, dims in ``WINDOW_DIMS``): the token at
    ``pos`` (int64) of slot ``slots`` (int32) sees the last ``min(pos + 1, R)`` positions, position p at row ``p % R``."""
    lib = _native.load(True)
    G = v.shape[2]
    units = G * lib.window_head_chunks(q.shape[1] // weights.maps, G, weights.maps)
    if splits < 1:
        splits = pick_window_splits(q.shape[0], units, v.shape[1])
    return lib.window_decode(q, k, v, float(scale), *weights._native(), gate, slots, pos, int(splits), _decode_counters(q.device, q.shape[0] * units))


def window_attention_prompt(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, weights: Weights, scale: float, gate: Optional[torch.Tensor],
                            cu: torch.Tensor, q_pos0: torch.Tensor, shift: torch.Tensor, max_q: int, window: int) -> torch.Tensor:
    """Prompts over packed rows ``k`` [rows, G maps, dk] and ``v`` [rows, G, dv] (GPU, bf16, dims in ``WINDOW_DIMS``, positive scale): the queries of sequence b are
    tokens ``cu[b] .. cu[b + 1]`` at positions from ``q_pos0[b]`` on, position p lies at row ``p + shift[b]``."""
    out, err = _native.load(True).window_prompt(q, k, v, float(scale), *weights._native(), gate, cu, q_pos0, shift, int(max_q), int(window))
    _PENDING_ERRORS.append(err)
    if len(_PENDING_ERRORS) > 64:
        check_attention_errors()
    return out
