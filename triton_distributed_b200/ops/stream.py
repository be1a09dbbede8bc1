"""fp32 residual stream of decoders that norm a sublayer's output: embedding, ``x += RMSNorm(y) * w``, the norm before
the head, and the whole-projection q / k norm that writes a tied KV cache.

The stream ``x`` [T, W] stays in fp32 for every activation dtype; ``xb`` is its bf16 copy that the next sublayer's GEMMs
read (for fp32 models ``xb`` IS ``x``).  W may be padded: columns from ``n_real`` on are zero and do not count in means.
GPU tensors run ``csrc/stream_ops.cu`` / ``csrc/tied_kv.cu``; CPU tensors run the torch restatement here.
"""
from __future__ import annotations

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


def embed_stream(ids: torch.Tensor, table: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """``(x, xb)`` of token ids [T]."""
    ids = ids.reshape(-1)
    if _native.use_native(ids, table):
        x = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
        xb = x if table.dtype == torch.float32 else torch.empty_like(x, dtype=table.dtype)
        _native.load(True).embed_stream(ids.to(torch.int64).contiguous(), table, x, None if xb is x else xb)
        return x, xb
    rows = table[ids.long()]
    x = rows.float().clone()
    return x, (x if table.dtype == torch.float32 else rows.clone())


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
