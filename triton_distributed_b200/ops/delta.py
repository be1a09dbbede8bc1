"""Gated delta rule in its serving form (forward, with carried state): short convolutions, unit norms, decay, recurrence, head norm
and output gate.

Per value head the fp32 state ``S`` [dk, dv] follows ``S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q`` with unit
``k`` and ``q`` (``q`` times ``q_scale``), ``g = exp(-exp(a_log) softplus(a + dt_bias))``, ``beta = sigmoid(b)``; q, k and v come out
of a causal convolution per channel and silu; the output is ``RMSNorm(o) * w * silu(gate)``.  Value head h uses key head
``h // (H / G)``.  GPU forms: ``csrc/delta.cu`` (fused one-token decode; token recurrence) and ``csrc/delta_chunk.cu`` (64-token
chunks in parallel, bf16).  CPU tensors run the restatement.  ``ops/gdn.py`` has the bare recurrence as a library call, with inputs
that are prepared already.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native

UNIT_EPS = 1e-6        # inside the root of the unit norms of q and k
DELTA_MAX_DIM = 256    # head dims the kernels take


def _restatement(z, ab, conv_w, a_log, dt_bias, norm_w, state, conv, slots, pos0, cu, G, dv_real, q_scale, eps):
    T = z.shape[0]
    _, H, dk, dv = state.shape
    C, taps = conv_w.shape
    F = torch.nn.functional
    x, gate = z[:, :C], z[:, C:C + H * dv].float()
    g = torch.exp(-torch.exp(a_log) * F.softplus(ab[:, :H] + dt_bias))
    beta = torch.sigmoid(ab[:, H:])
    o = torch.empty(T, H, dv)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for n in range(len(bounds) - 1):
        lo, hi, slot, p0 = bounds[n], bounds[n + 1], int(slots[n]), int(pos0[n])
        before = [conv[slot, p % taps].float() if p >= 0 else torch.zeros(C) for p in range(p0 - taps + 1, p0)]
        seq = torch.cat([torch.stack(before) if before else x.new_zeros(0, C).float(), x[lo:hi].float()])
        y = F.silu(sum(seq[j:j + hi - lo] * conv_w[:, j] for j in range(taps)))
        for p in range(max(p0, p0 + hi - lo - taps + 1), p0 + hi - lo):
            conv[slot, p % taps] = x[lo + p - p0]
        q, k, v = y.split([G * dk, G * dk, H * dv], dim=1)
        q, k = (t.reshape(-1, G, dk) for t in (q, k))
        q, k = ((t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + UNIT_EPS)).repeat_interleave(H // G, dim=1) for t in (q, k))
        v = v.reshape(-1, H, dv)
        S = torch.zeros(H, dk, dv) if p0 == 0 else state[slot].clone()
        for t in range(hi - lo):
            S = S * g[lo + t, :, None, None]
            u = beta[lo + t, :, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
            S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
            o[lo + t] = torch.einsum("hkv,hk->hv", S, q[t] * q_scale)
        state[slot] = S
    o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / dv_real + eps) * norm_w
    return (o.reshape(T, H * dv) * F.silu(gate)).to(z.dtype)


def gated_delta_rule(z: torch.Tensor, ab: torch.Tensor, conv_w: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor,
                     norm_w: torch.Tensor, state: torch.Tensor, conv: torch.Tensor, slots: torch.Tensor, pos0: torch.Tensor,
                     cu: Optional[torch.Tensor], kv_heads: int, dv_real: int, q_scale: float, eps: float, chunk_tables=None,
                     impl: str = "auto") -> torch.Tensor:
    """``z`` [T, 2 G dk + 2 H dv] (q, k, v, output gate), ``ab`` fp32 [T, 2 H] (decay input, step-size input), ``conv_w`` fp32
    [C, taps] over the q, k, v columns, ``state`` fp32 [slots, H, dk, dv] and ``conv`` [slots, taps, C] (the convolutions' inputs,
    position p at row ``p % taps``) updated in place at ``slots`` [N] (int32).  Sequence n owns tokens ``cu[n] .. cu[n + 1]``
    (``cu`` None: one token per sequence, the decode form) from position ``pos0[n]`` on; nothing before position 0 is read.
    ``impl``: "auto", "decode", "recurrent" or "chunk"; prompts need ``chunk_tables`` on a GPU."""
    if not _native.use_native(z, state):
        return _restatement(z, ab, conv_w, a_log, dt_bias, norm_w, state, conv, slots, pos0, cu, int(kv_heads), dv_real, q_scale, eps)
    lib = _native.load(True)
    if impl == "auto":
        chunk = z.dtype == torch.bfloat16 and lib.delta_chunk_supported(state.shape[2], state.shape[3])
        impl = "decode" if cu is None else "chunk" if chunk else "recurrent"
    form = {"decode": 0, "recurrent": 1, "chunk": 2}[impl]
    tabs = chunk_tables if form else (None, None, None)
    return lib.delta_forward(z, ab, conv_w, a_log, dt_bias, norm_w, state, conv, slots, pos0, cu, int(kv_heads), int(dv_real),
                             float(q_scale), UNIT_EPS, float(eps), form, *tabs)
