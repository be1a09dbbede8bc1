"""State space layer with one decay per head and token (Mamba-2's recurrence) in its serving form (forward, with carried state), and the
gated norm over groups behind it.

Per head the fp32 state ``S`` [dk, dv] follows ``S <- exp(-exp(a_log) dt) S + dt B x^T``, ``y = S^T C + D x`` with ``dt = softplus(dt_in +
dt_bias)``; x, B and C come out of a causal convolution per channel with a bias and silu, B and C are shared by the heads of a group.
GPU forms: ``csrc/ssd.cu`` (fused one-token decode; token recurrence) and ``csrc/ssd_chunk.cu`` (64-token chunks in parallel, bf16).
CPU tensors run the restatement.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import _native

SSD_MAX_DIM = 256      # state and head sizes the kernels take


@dataclass
class SsdWeights:
    """fp32: ``conv_w`` [channels, taps] and ``conv_b`` over x | B | C, and per head the logarithm of the decay rate, the step size's bias, the skip."""
    conv_w: torch.Tensor
    conv_b: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    skip: torch.Tensor


def _restatement(z, dt_col, w, state, conv, slots, pos0, cu, G):
    T = z.shape[0]
    _, H, dk, dv = state.shape
    C, taps = w.conv_w.shape
    F = torch.nn.functional
    x = z[:, :C]
    dt = F.softplus(z[:, dt_col:dt_col + H].float() + w.dt_bias)
    a = torch.exp(-torch.exp(w.a_log) * dt)
    y = torch.empty(T, H, dv)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for n in range(len(bounds) - 1):
        lo, hi, slot, p0 = bounds[n], bounds[n + 1], int(slots[n]), int(pos0[n])
        before = [conv[slot, p % taps].float() if p >= 0 else torch.zeros(C) for p in range(p0 - taps + 1, p0)]
        seq = torch.cat([torch.stack(before) if before else x.new_zeros(0, C).float(), x[lo:hi].float()])
        u = F.silu(sum(seq[j:j + hi - lo] * w.conv_w[:, j] for j in range(taps)) + w.conv_b)
        for p in range(max(p0, p0 + hi - lo - taps + 1), p0 + hi - lo):
            conv[slot, p % taps] = x[lo + p - p0]
        xs, B, Cc = u.to(z.dtype).float().split([H * dv, G * dk, G * dk], dim=1)
        xs = xs.reshape(-1, H, dv)
        B, Cc = (t.reshape(-1, G, dk).repeat_interleave(H // G, dim=1) for t in (B, Cc))
        S = torch.zeros(H, dk, dv) if p0 == 0 else state[slot].clone()
        for t in range(hi - lo):
            S = S * a[lo + t, :, None, None] + B[t].unsqueeze(-1) * (dt[lo + t, :, None] * xs[t]).unsqueeze(1)
            y[lo + t] = torch.einsum("hkv,hk->hv", S, Cc[t]) + w.skip[:, None] * xs[t]
        state[slot] = S
    return y.reshape(T, H * dv).to(z.dtype)


def state_space(z: torch.Tensor, dt_col: int, w: SsdWeights, state: torch.Tensor, conv: torch.Tensor, slots: torch.Tensor, pos0: torch.Tensor,
                cu: Optional[torch.Tensor], groups: int, chunk_tables=None, impl: str = "auto") -> torch.Tensor:
    """``z`` [T, ..]: x [H, dv], B [G, dk], C [G, dk] from column 0, the step sizes' input [H] from column ``dt_col``.  ``state`` fp32
    [slots, H, dk, dv] and ``conv`` [slots, taps, channels] (the convolutions' inputs, position p at row ``p % taps``) are updated in place at
    ``slots`` [N] (int32).  Sequence n owns tokens ``cu[n] .. cu[n + 1]`` (``cu`` None: one token per sequence, the decode form) from position
    ``pos0[n]`` on; nothing before position 0 is read.  Returns y [T, H dv].  ``impl``: "auto", "decode", "recurrent" or "chunk"; prompts
    need ``chunk_tables`` on a GPU."""
    if not _native.use_native(z, state):
        return _restatement(z, dt_col, w, state, conv, slots, pos0, cu, int(groups))
    lib = _native.load(True)
    if impl == "auto":
        chunk = z.dtype == torch.bfloat16 and lib.ssd_chunk_supported(state.shape[2], state.shape[3])
        impl = "decode" if cu is None else "chunk" if chunk else "recurrent"
    form = {"decode": 0, "recurrent": 1, "chunk": 2}[impl]
    tabs = chunk_tables if form else (None, None, None)
    return lib.ssd_forward(z, int(dt_col), w.conv_w, w.conv_b, w.a_log, w.dt_bias, w.skip, state, conv, slots, pos0, cu, int(groups), form, *tabs)


def gated_group_norm(y: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, heads: int, dv_real: int, parts: int, eps: float) -> torch.Tensor:
    """``y * silu(gate)``, then every one of ``parts`` equal parts of a row divided by its own root mean square, times ``w`` (fp32).  ``y``
    [T, heads dv], ``gate`` [T, >= heads dv]; of a head's dv columns ``dv_real`` are real, the parts are cut over the real ones."""
    H, D = int(heads), int(dv_real)
    if _native.use_native(y, gate):
        return _native.load(True).gated_norm(y, gate, w, H, D, int(parts), float(eps))
    T, dv = y.shape[0], y.shape[1] // H
    g = gate[:, :H * dv].float()
    v = (y.float() * torch.nn.functional.silu(g)).reshape(T, H, dv)[..., :D].reshape(T, parts, -1)
    v = (v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, H, D)
    return (torch.nn.functional.pad(v, (0, dv - D)).reshape(T, H * dv) * w).to(y.dtype)
