"""fp32 residual stream of layered decoders: embedding, ``x += RMSNorm(y) * w`` (norm on a sublayer's output), sublayers between two norms or ``x += mixer +
feed-forward`` with the next layer's norms (parallel layers), the norm before the head, and the whole-projection q / k norm that
writes a tied KV cache.

The stream ``x`` [T, W] stays in fp32 for every activation dtype; ``xb`` is its bf16 copy that the next sublayer's GEMMs
read (for fp32 models ``xb`` IS ``x``).  W may be padded: columns from ``n_real`` on are zero and do not count in means.
GPU tensors run ``csrc/stream_ops.cu`` / ``csrc/tied_kv.cu``; CPU tensors run the torch restatement here.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .. import _native


def _rms_factor(x: torch.Tensor, n_real: int, eps: float) -> torch.Tensor:
    return torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n_real + eps)


def _token_sum(y, T, rows, shared, shared_gate):
    s = y.float().reshape(T, rows, -1).sum(1)
    if shared is not None:
        g = 1.0 if shared_gate is None else shared_gate.float().reshape(T, 1)
        s = s + g * shared.float()
    return s


def embed_stream(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0, copy: bool = True):
    """``(x, xb)`` of token ids [T]: ``x = scale * table[ids]`` in fp32 (without ``copy``, ``xb`` is None)."""
    ids = ids.reshape(-1)
    if _native.use_native(ids, table):
        x = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
        xb = None if not copy else x if table.dtype == torch.float32 else torch.empty_like(x, dtype=table.dtype)
        _native.load(True).embed_stream(ids.to(torch.int64).contiguous(), table, x, None if xb is x else xb, float(scale))
        return x, xb
    x = table[ids.long()].float() * scale
    return x, (None if not copy else x if table.dtype == torch.float32 else x.to(table.dtype))


def postnorm_add(x: torch.Tensor, xb: torch.Tensor, y: torch.Tensor, w: torch.Tensor, n_real: int, eps: float,
                 rows_per_token: int = 1, shared: Optional[torch.Tensor] = None,
                 shared_gate: Optional[torch.Tensor] = None) -> None:
    """In place: ``x += RMSNorm(s) * w`` and ``xb = x`` with ``s[t]`` the sum of the token's ``rows_per_token`` rows of
    ``y`` (plus ``shared_gate[t] * shared[t]``).  ``w`` fp32 [W]."""
    if _native.use_native(x, y):
        _native.load(True).postnorm_add(x, None if xb is x else xb, y.contiguous(), w, int(rows_per_token), int(n_real),
                                        float(eps), shared, shared_gate)
        return
    s = _token_sum(y, x.shape[0], rows_per_token, shared, shared_gate)
    x += s * _rms_factor(s, n_real, eps) * w
    if xb is not x:
        xb.copy_(x)


@dataclass
class FeedForward:
    """What a feed-forward adds to the stream, left in pieces for :func:`parallel_add` to sum: ``rows`` rows of ``y`` per token,
    of which those of an expert id outside [0, ``experts``) stand for ``weight * hin`` (identity experts; ``hin`` None: nothing),
    a shared expert's rows and a bias."""
    y: torch.Tensor
    rows: int = 1
    ids: Optional[torch.Tensor] = None
    weights: Optional[torch.Tensor] = None
    experts: int = 0
    hin: Optional[torch.Tensor] = None
    shared: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None


def parallel_sum(x: torch.Tensor, mix: Optional[torch.Tensor], ff: Optional[FeedForward]) -> torch.Tensor:
    """fp32 [T, W]: what :func:`parallel_add` would add to the stream (what tensor-parallel ranks exchange)."""
    return _parallel(x, mix, ff, None, None, 1, 0.0, torch.float32 if mix is None else mix.dtype, True)[0]


def parallel_add(x: torch.Tensor, mix: Optional[torch.Tensor], ff: Optional[FeedForward], w1: Optional[torch.Tensor],
                 w2: Optional[torch.Tensor], n_real: int, eps: float, dtype: torch.dtype):
    """In place ``x += mix + ff``; returns ``(RMSNorm(x) * w1, RMSNorm(x) * w2)`` in ``dtype``, None where the weight is None."""
    out = _parallel(x, mix, ff, w1, w2, n_real, eps, dtype, False)
    return tuple(out) + (None,) * (2 - len(out))


def _parallel(x, mix, ff, w1, w2, n_real, eps, dtype, sum_only):
    f = ff if ff is not None else FeedForward(None)
    if _native.use_native(x):
        return _native.load(True).parallel_add(x, mix, f.y, int(f.rows), f.ids, f.weights, int(f.experts), f.hin, f.shared, f.bias,
                                               w1, w2, int(n_real), float(eps), dtype == torch.float32, sum_only)
    s = torch.zeros_like(x)
    if mix is not None:
        s += mix.float()
    if f.y is not None:
        y = f.y.float().reshape(x.shape[0], f.rows, -1)
        if f.ids is not None:
            own = (f.ids >= 0) & (f.ids < f.experts)
            y = torch.where(own.unsqueeze(-1), y, torch.zeros_like(y))
            if f.hin is not None:
                y = y + (~own).unsqueeze(-1) * f.weights.unsqueeze(-1) * f.hin.float().unsqueeze(1)
        s += y.sum(1)
    for t in (f.shared, f.bias):
        if t is not None:
            s += t.float()
    if sum_only:
        return [s]
    x += s
    r = x * _rms_factor(x, n_real, eps)
    return [(r * w).to(dtype) for w in (w1, w2) if w is not None]


# ------------------------------------------------------------------ several streams
@dataclass
class HyperWeights:
    """What joins a sublayer to S streams, fp32: its input is ``sum_s inp[s] x_s``; then ``x_t <- sum_s mix[s, t] x_s + out[t] y``."""
    inp: torch.Tensor
    out: torch.Tensor
    mix: torch.Tensor


@dataclass
class SublayerOutput:
    """``y``, or with a second branch ``(RMSNorm(y) * y_w + RMSNorm(y2) * y2_w) / 2`` (weights fp32)."""
    y: torch.Tensor
    y2: Optional[torch.Tensor] = None
    y_w: Optional[torch.Tensor] = None
    y2_w: Optional[torch.Tensor] = None


def hyper_step(x: torch.Tensor, last: Optional[Tuple[HyperWeights, SublayerOutput]], nxt: Optional[Tuple[torch.Tensor, torch.Tensor]],
               n_real: int, eps: float, dtype: torch.dtype, rows: Optional[torch.Tensor] = None,
               start: Optional[Tuple[torch.Tensor, torch.Tensor]] = None) -> Optional[torch.Tensor]:
    """One pass over the streams ``x`` [T, S, W] (fp32, in place) between two sublayers: adds the output of the ``last`` one and
    returns the normed input ``RMSNorm(sum_s inp[s] x_s) * w`` of the next, ``nxt = (inp, w)``, in ``dtype``.  ``start = (ids, table)``
    sets all streams to the tokens' rows first.  With ``rows`` (int64) only these tokens are computed and ``x`` stays as it is."""
    if _native.use_native(x):
        ids, table = start if start is not None else (None, None)
        hw, o = last if last is not None else (None, None)
        h = _native.load(True).hyper_step(x, ids, table, *((o.y, o.y2, o.y_w, o.y2_w, hw.mix, hw.out) if o is not None else (None,) * 6),
                                          *(nxt if nxt is not None else (None, None)), rows, int(n_real), float(eps), dtype == torch.float32)
        return h if nxt is not None else None
    if start is not None:
        x.copy_(start[1][start[0].long()].float().unsqueeze(1).expand_as(x))
    v = x if rows is None else x[rows]
    if last is not None:
        hw, o = last
        y, y2 = (t if t is None or rows is None else t[rows] for t in (o.y, o.y2))
        y = y.float()
        if y2 is not None:
            y2 = y2.float()
            y = 0.5 * (y * _rms_factor(y, n_real, eps) * o.y_w + y2 * _rms_factor(y2, n_real, eps) * o.y2_w)
        v = torch.einsum("st,nsw->ntw", hw.mix, v) + hw.out[:, None] * y.unsqueeze(1)
        if rows is None:
            x.copy_(v)
    if nxt is None:
        return None
    u = torch.einsum("s,nsw->nw", nxt[0], v)
    return (u * _rms_factor(u, n_real, eps) * nxt[1]).to(dtype)


# ------------------------------------------------------------------ a sublayer between two norms
def sandwich_step(x: torch.Tensor, last: Optional[Tuple[torch.Tensor, torch.Tensor]], pre: Optional[torch.Tensor], n_real: int, eps: float,
                  dtype: torch.dtype, rows: Optional[torch.Tensor] = None,
                  start: Optional[Tuple[torch.Tensor, torch.Tensor, float]] = None) -> Optional[torch.Tensor]:
    """One pass over the stream ``x`` [T, W] (fp32, in place) between two sublayers: ``x += RMSNorm(y) * post`` with ``last = (y, post)``,
    then the next one's input ``RMSNorm(x) * pre`` in ``dtype``.  ``post`` and ``pre`` are fp32 weights, one number for all coordinates
    or one each.  ``start = (ids, table, scale)`` sets x to the tokens' scaled rows first.  With ``rows`` (int64) only these tokens
    are computed and ``x`` stays as it is."""
    if _native.use_native(x):
        ids, table, scale = start if start is not None else (None, None, 1.0)
        h = _native.load(True).sandwich(x, ids, table, float(scale), *(last if last is not None else (None, None)), pre, rows, int(n_real), float(eps),
                                        dtype == torch.float32)
        return h if pre is not None else None
    if start is not None:
        x.copy_(start[1][start[0].long()].float() * start[2])
    v = x if rows is None else x[rows]
    if last is not None:
        y = (last[0] if rows is None else last[0][rows]).float()
        v = v + y * _rms_factor(y, n_real, eps) * last[1]
        if rows is None:
            x.copy_(v)
    return None if pre is None else (v * _rms_factor(v, n_real, eps) * pre).to(dtype)


def combine_rows(y: torch.Tensor, T: int, rows_per_token: int, shared: Optional[torch.Tensor] = None,
                 shared_gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The sum of :func:`postnorm_add` alone, [T, W] in the dtype of ``y`` (what tensor-parallel ranks exchange)."""
    if _native.use_native(y):
        return _native.load(True).combine_rows(y.contiguous(), int(T), int(rows_per_token), shared, shared_gate)
    return _token_sum(y, T, rows_per_token, shared, shared_gate).to(y.dtype)


def stream_norm(x: torch.Tensor, w: torch.Tensor, n_real: int, eps: float, dtype: torch.dtype,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``RMSNorm(x[rows]) * w`` in ``dtype`` (``rows`` int64, None: every row)."""
    if _native.use_native(x):
        n = x.shape[0] if rows is None else rows.numel()
        out = torch.empty(n, x.shape[1], dtype=dtype, device=x.device)
        _native.load(True).stream_norm(x, rows, w, out, int(n_real), float(eps))
        return out
    xr = x if rows is None else x[rows]
    return (xr * _rms_factor(xr, n_real, eps) * w).to(dtype)


def qk_sumsq(qk: torch.Tensor, n_q: int, n_k: int) -> torch.Tensor:
    """fp32 [T, 2]: sums of squares of the q columns and of the k columns (to be summed over ranks)."""
    if _native.use_native(qk):
        return _native.load(True).qk_sumsq(qk, int(n_q), int(n_k))
    f = qk.float()
    return torch.stack([f[:, :n_q].pow(2).sum(-1), f[:, n_q:n_q + n_k].pow(2).sum(-1)], dim=1).contiguous()


def qk_norm_tied(qk: torch.Tensor, q_weight: torch.Tensor, n_k: int, nq_real: int, nk_real: int, eps: float,
                 dest: Tuple[torch.Tensor, torch.Tensor, torch.Tensor],
                 dest2: Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]] = None,
                 sumsq: Optional[torch.Tensor] = None) -> torch.Tensor:
    """RMS norms of q and of k, each over its whole projection, for a tied cache.  ``qk`` [T, >= Nq + Nk] holds q then k.

    Returns the query [T, Nq] = ``q / rms(q) * q_weight``, where ``q_weight`` (fp32) carries the query norm's weight, the
    KEY norm's weight and the score scale; the raw key rows and their factors ``1 / rms(k)`` go to rows ``rows`` of
    ``dest = (k, scale, rows)`` (and ``dest2``); negative rows are not stored."""
    n_q = q_weight.numel()
    if _native.use_native(qk, dest[0]):
        d2 = dest2 if dest2 is not None else (None, None, None)
        return _native.load(True).qk_norm_tied(qk, q_weight, int(n_k), int(nq_real), int(nk_real), float(eps), *dest, *d2, sumsq)
    if sumsq is None:
        sumsq = qk_sumsq(qk, n_q, n_k)
    q, k = qk[:, :n_q].float(), qk[:, n_q:n_q + n_k]
    fq = torch.rsqrt(sumsq[:, :1] / nq_real + eps)
    fk = torch.rsqrt(sumsq[:, 1] / nk_real + eps)
    for d in (dest, dest2):
        if d is None:
            continue
        kc, sc, rows = d
        ok = rows >= 0
        kc.view(-1, n_k)[rows[ok]] = k[ok]
        sc.view(-1)[rows[ok]] = fk[ok]
    return (q * fq * q_weight).to(qk.dtype)
