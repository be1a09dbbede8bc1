"""Tensor-parallel mixture of squared-ReLU experts with sigmoid scores and a gated shared expert (intermediate dimension
split over the ranks, router replicated).

The routing weight scales an expert's INPUT; its up projection has no bias, so the weight is applied to that projection's
output inside the activation.  Few tokens (and fp32) stream the chosen experts pair by pair; longer inputs sort the (token,
expert) pairs and run the grouped tcgen05 GEMMs with the row gather inside the kernel.
"""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_rows, shard


class TP_SigmoidMoE(TPLayer):
    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        self.spec = spec

    def load(self, get, prefix: str, width: int, dtype, device):
        s, w8 = self.spec, pad8(width)

        def expert(p):
            up = shard(get(prefix + p + "up"), self.rank, self.world_size)
            down = shard(get(prefix + p + "down"), self.rank, self.world_size, 1)
            ff = pad8(up.shape[0])
            return pad_rows(up, ff, w8).to(dtype).to(device), pad_rows(down, w8, ff).to(dtype).to(device)

        pairs = [expert(f"e{e}.") for e in range(s.experts)]
        self.up = torch.stack([u for u, _ in pairs]).contiguous()
        self.down = torch.stack([d for _, d in pairs]).contiguous()
        router = get(prefix + "router")
        self.shared_up = self.shared_down = None
        if s.shared_ff:
            self.shared_up, self.shared_down = (t.contiguous() for t in expert("shared."))
            router = torch.cat([router, get(prefix + "shared.sg").reshape(1, -1)])      # its gate is one more column
        self.router = pad_rows(router, router.shape[0], w8).to(dtype).to(device).contiguous()

    def __call__(self, x: torch.Tensor):
        """``(y, rows per token, shared, shared gate)``: contributions for the stream's norm to sum (already summed, with
        rows = 1 and no shared part, on several ranks)."""
        s = self.spec
        T = x.shape[0]
        ids, w, gate = ops.sigmoid_router(x, self.router, s.top, bool(s.shared_ff))
        if not x.is_cuda or x.dtype == torch.float32 or T <= ops.EXPERT_GEMV_MAX_T:
            y = ops.relu2_experts_gemv(x, self.up, self.down, ids, w, self.shared_up, self.shared_down, gate)
            return self.reduce(y), 1, None, None
        srt = ops.sort_topk_ids_align_block_size(ids, s.experts)
        h = ops.group_gemm_gather(x, self.up, srt, a_row_div=s.top, scatter_out=True)
        h = ops.relu2(h, w.reshape(-1))
        y = ops.group_gemm_gather(h, self.down, srt, a_row_div=1, scatter_out=True)
        shared = None
        if self.shared_up is not None:
            shared = self.linear(ops.relu2(self.linear(x, self.shared_up)), self.shared_down)
        if self.world_size > 1:
            return self.reduce(ops.combine_rows(y, T, s.top, shared, gate)), 1, None, None
        return y, s.top, shared, gate
