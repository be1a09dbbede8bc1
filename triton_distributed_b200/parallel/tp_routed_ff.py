"""Tensor-parallel feed-forwards of layered decoders: dense gated; and of parallel layers: dense squared-ReLU with biases, and a mixture of gated (SiLU) experts with a
softmax router, a choice correction, expert groups, identity experts and a shared expert.  Intermediate dimensions are split over
the ranks, the router is replicated.

The latter two return their contribution in pieces (``ops.FeedForward``): the layer's one addition to the stream sums them together with
the mixer's.  What is not split (biases, identity experts) is added by rank 0 alone.
"""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_rows, shard


class TP_DenseFF(TPLayer):
    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        self.spec = spec

    def load(self, get, prefix: str, width: int, dtype, device):
        w8 = pad8(width)
        up = shard(get(prefix + "up"), self.rank, self.world_size)
        ff = pad8(up.shape[0])
        self.up = pad_rows(up, ff, w8).to(dtype).to(device).contiguous()
        self.up_b = pad_rows(shard(get(prefix + "up.b"), self.rank, self.world_size).float(), ff).to(device)
        self.down = pad_rows(shard(get(prefix + "down"), self.rank, self.world_size, 1), w8, ff).to(dtype).to(device).contiguous()
        self.down_b = pad_rows(get(prefix + "down.b").float(), w8).to(device) if self.rank == 0 else None

    def __call__(self, x: torch.Tensor) -> ops.FeedForward:
        y = self.linear(ops.relu2(self.linear(x, self.up), None, self.up_b), self.down)
        return ops.FeedForward(y, bias=self.down_b)


class TP_GatedFF(TPLayer):
    """``W_down (act(W_gate x) * W_up x)`` with ``act`` one of ``ops.GATED_ACTS``; ``spec.ff`` is the intermediate size.  Decode steps of
    a few tokens apply the activation inside the down projection's launch."""

    def __init__(self, spec, act: str, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        self.spec, self.act = spec, act

    def load(self, get, prefix: str, width: int, dtype, device):
        w8 = pad8(width)
        gate, up = (shard(get(prefix + n), self.rank, self.world_size) for n in ("gate", "up"))
        ff = pad8(up.shape[0])
        self.gate_up = torch.cat([pad_rows(gate, ff, w8), pad_rows(up, ff, w8)]).to(dtype).to(device).contiguous()
        self.down = pad_rows(shard(get(prefix + "down"), self.rank, self.world_size, 1), w8, ff).to(dtype).to(device).contiguous()

    def __call__(self, x: torch.Tensor) -> ops.SublayerOutput:
        h = self.linear(x, self.gate_up)
        few = x.shape[0] <= ops.GEMV_FAST_M and ops.gemv_supported(x.shape[0], self.down.shape[1])
        if few and self.mode != "torch" and self.world_size == 1 and x.is_cuda and x.dtype == torch.bfloat16:
            return ops.SublayerOutput(ops.gemv_fused(h, self.down, silu_mul=True, act=self.act))
        return ops.SublayerOutput(self.out_linear(ops.gated_act(h, self.act), self.down))


class TP_RoutedMoE(TPLayer):
    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        self.spec = spec

    def load(self, get, prefix: str, width: int, dtype, device):
        s, w8 = self.spec, pad8(width)

        def expert(p):
            gate, up = (shard(get(prefix + p + n), self.rank, self.world_size) for n in ("gate", "up"))
            ff = pad8(up.shape[0])
            down = shard(get(prefix + p + "down"), self.rank, self.world_size, 1)
            both = torch.cat([pad_rows(gate, ff, w8), pad_rows(up, ff, w8)])
            return both.to(dtype).to(device), pad_rows(down, w8, ff).to(dtype).to(device)

        pairs = [expert(f"e{e}.") for e in range(s.experts)]
        self.gate_up = torch.stack([u for u, _ in pairs]).contiguous()
        self.down = torch.stack([d for _, d in pairs]).contiguous()
        self.shared_gate_up = self.shared_down = None
        if s.shared_ff:
            self.shared_gate_up, self.shared_down = (t.contiguous() for t in expert("shared."))
        router = get(prefix + "router")
        self.router = pad_rows(router, router.shape[0], w8).to(dtype).to(device).contiguous()
        self.correction = get(prefix + "correction").float().to(device).contiguous()

    def __call__(self, x: torch.Tensor) -> ops.FeedForward:
        s, T = self.spec, x.shape[0]
        ids, w = ops.softmax_router(x, self.router, self.correction, s.top, s.groups, s.keep)
        if not x.is_cuda or x.dtype == torch.float32 or T <= ops.EXPERT_GEMV_MAX_T:
            return ops.FeedForward(ops.gated_experts_gemv(x, self.gate_up, self.down, ids, w, self.shared_gate_up, self.shared_down,
                                                          s.identity, self.rank != 0))
        # pairs of identity experts have ids beyond the experts: the sort leaves them out and their rows stay unwritten
        srt = ops.sort_topk_ids_align_block_size(ids, s.experts)
        h = ops.silu_mul(ops.group_gemm_gather(x, self.gate_up, srt, a_row_div=s.top, scatter_out=True))
        y = ops.group_gemm_gather(h, self.down, srt, a_row_div=1, scatter_out=True, row_weight=w)
        shared = None
        if self.shared_gate_up is not None:
            shared = self.linear(ops.silu_mul(self.linear(x, self.shared_gate_up)), self.shared_down)
        return ops.FeedForward(y, s.top, ids, w, s.experts, x if self.rank == 0 else None, shared)
