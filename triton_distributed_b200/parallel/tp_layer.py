"""Common part of the tensor-parallel mixers / feed-forwards of layered decoders: padding of weights at load time, the
projection and all-reduce calls of the execution modes, shared communication contexts.

Padding happens once, on the weights, so that no kernel needs ragged edges: zero rows and columns bring every dimension to
what the kernels take (multiples of eight; head dims to a kernel's tile), produce zeros, and never count in a norm's mean.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.distributed as dist

from .. import ops

AR_MODES = ("triton_dist", "ag_rs", "triton_dist_AR", "allreduce")
GEMM_AR_MODES = ("triton_dist_gemm_ar", "gemm_ar")


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad_rows(t: torch.Tensor, *sizes: int) -> torch.Tensor:
    """``t`` with zeros appended up to ``sizes`` (leading dimensions first; missing sizes stay)."""
    pads = []
    for d in range(t.dim() - 1, -1, -1):
        pads += [0, (sizes[d] - t.shape[d]) if d < len(sizes) else 0]
    return torch.nn.functional.pad(t, pads) if any(pads) else t


def pad_heads(t: torch.Tensor, heads: int, dim: int, to: int) -> torch.Tensor:
    """Rows grouped by head, [heads * dim, ...] -> [heads * to, ...] with every head padded."""
    return pad_rows(t.reshape(heads, dim, *t.shape[1:]), heads, to).reshape(heads * to, *t.shape[1:])


def shard(t: torch.Tensor, rank: int, world: int, dim: int = 0) -> torch.Tensor:
    if t.shape[dim] % world:
        raise ValueError(f"dimension of {t.shape[dim]} cannot be split over {world} ranks")
    n = t.shape[dim] // world
    return t.narrow(dim, rank * n, n)


class TPLayer:
    def __init__(self, rank: int = 0, world_size: int = 1, group=None):
        self.rank, self.world_size, self.group = rank, world_size, group
        self.mode = "torch"
        self.ar_ctx = self.gemm_ar_ctx = None

    def set_fwd(self, mode: str):
        if mode != "torch" and mode not in AR_MODES and mode not in GEMM_AR_MODES:
            raise KeyError(mode)
        self.mode = mode

    def init_ctx(self, mode: str, max_M: int, hidden: int):
        """fp32 all-reduce buffer, and in the gemm_ar modes the fused GEMM + all-reduce of the output projection."""
        self.ar_ctx = ops.create_allreduce_ctx(max(4 * max_M * hidden * 4, 1 << 20))
        if mode in GEMM_AR_MODES:
            self.gemm_ar_ctx = ops.create_gemm_ar_context(max_M=max_M, N=hidden, dtype=torch.bfloat16)

    def finalize(self):
        for c in (self.ar_ctx, self.gemm_ar_ctx):
            if c is not None:
                c.finalize()
        self.ar_ctx = self.gemm_ar_ctx = None

    def linear(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return torch.matmul(x, w.t()) if self.mode == "torch" else ops.gemm(x, w)

    def reduce(self, y: torch.Tensor) -> torch.Tensor:
        """Sum of the ranks' partial outputs."""
        if self.world_size == 1:
            return y
        if self.mode != "torch" and self.ar_ctx is not None and y.is_cuda:
            return ops.all_reduce(y, ctx=self.ar_ctx)
        dist.all_reduce(y, group=self.group)
        return y

    def out_linear(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """Row-parallel projection: partial products summed over the ranks."""
        if self.world_size > 1 and self.mode in GEMM_AR_MODES and self.gemm_ar_ctx is not None and x.dtype == torch.bfloat16:
            return ops.gemm_allreduce_op(self.gemm_ar_ctx, x, w)
        return self.reduce(self.linear(x, w))
