"""Gated linear attention with a per-channel decay (forward, with carried state).

Per head the fp32 state ``S`` [dk, dv] follows ``S <- diag(alpha_t) S + k_t v_t^T``, ``o_t = q_scale S^T q_t``; the decay is
``alpha_t = sigmoid(a2^T a_t + b)^(1 / tau)`` with the low-rank input ``a_t``; the output is ``RMSNorm(o) * w * silu(g)``.
GPU forms: ``csrc/gla.cu`` (fused one-token decode; token recurrence for fp32) and ``csrc/gla_chunk.cu`` (64-token chunks in
parallel, bf16).  CPU tensors run the torch restatement.  The gated delta rule, a different recurrence with one decay per
head, is in ``ops/gdn.py``.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from .. import _native

GLA_CHUNK = 64


def gla_chunk_tables(cu: List[int], device, chunk: int = GLA_CHUNK) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """Sequence and first token of every chunk, first chunk of every sequence (int32, on ``device``)."""
    seq_of, t0_of, first = [], [], [0]
    for s in range(len(cu) - 1):
        for t in range(cu[s], cu[s + 1], chunk):
            seq_of.append(s)
            t0_of.append(t)
        first.append(len(seq_of))
    flat = torch.tensor(seq_of + t0_of + first, dtype=torch.int32).to(device)
    n = len(seq_of)
    return flat[:n], flat[n:2 * n], flat[2 * n:]


def _restatement(qkvg, lowrank, a2, a2_b, inv_tau, norm_w, state, slots, pos0, cu, dv_real, q_scale, eps):
    T = qkvg.shape[0]
    _, H, dk, dv = state.shape
    q, k, v, g = qkvg[:, :2 * H * (dk + dv)].float().split([H * dk, H * dk, H * dv, H * dv], dim=1)
    q, k, v = q.reshape(T, H, dk) * q_scale, k.reshape(T, H, dk), v.reshape(T, H, dv)
    alpha = torch.exp(torch.nn.functional.logsigmoid(lowrank @ a2 + a2_b) * inv_tau).reshape(T, H, dk)
    o = torch.empty(T, H, dv)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for n in range(len(bounds) - 1):
        slot = int(slots[n])
        S = torch.zeros(H, dk, dv) if int(pos0[n]) == 0 else state[slot].clone()
        for t in range(bounds[n], bounds[n + 1]):
            S = S * alpha[t].unsqueeze(-1) + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
            o[t] = torch.einsum("hkv,hk->hv", S, q[t])
        state[slot] = S
    o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / dv_real + eps) * norm_w
    return (o.reshape(T, H * dv) * torch.nn.functional.silu(g)).to(qkvg.dtype)


def gated_linear_attention(qkvg: torch.Tensor, lowrank: torch.Tensor, a2: torch.Tensor, a2_b: torch.Tensor, tau: float,
                           norm_w: torch.Tensor, state: torch.Tensor, slots: torch.Tensor, pos0: torch.Tensor,
                           cu: Optional[torch.Tensor], dv_real: int, q_scale: float, eps: float, chunk_tables=None,
                           impl: str = "auto") -> torch.Tensor:
    """``qkvg`` [T, 2 H dk + 2 H dv] (q, k, v, output gate), ``lowrank`` fp32 [T, R], ``a2`` fp32 [R, H dk], ``state`` fp32
    [slots, H, dk, dv] updated in place at ``slots`` [N] (int32).  Sequence n owns tokens ``cu[n] .. cu[n + 1]`` (``cu`` None:
    one token per sequence, the decode form); ``pos0[n] == 0`` starts it from a zero state.  ``dv_real`` is the divisor of
    the head norm when dv is padded.  ``impl``: "auto", "decode", "recurrent" or "chunk" (bf16, needs ``chunk_tables``)."""
    inv_tau = 1.0 / float(tau)
    if not _native.use_native(qkvg, state):
        return _restatement(qkvg, lowrank, a2, a2_b, inv_tau, norm_w, state, slots, pos0, cu, dv_real, q_scale, eps)
    lib = _native.load(True)
    if impl == "auto":
        if cu is None:
            impl = "decode"
        else:
            ok = qkvg.dtype == torch.bfloat16 and lib.gla_chunk_supported(state.shape[2], state.shape[3]) and chunk_tables is not None
            impl = "chunk" if ok else "recurrent"
    form = {"decode": 0, "recurrent": 1, "chunk": 2}[impl]
    tabs = chunk_tables if form == 2 else (None, None, None)
    return lib.gla_forward(qkvg, lowrank, a2, a2_b, inv_tau, norm_w, state, slots, pos0, cu, int(dv_real), float(q_scale),
                           float(eps), form, *tabs)
