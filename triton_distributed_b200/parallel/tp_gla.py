"""Tensor-parallel gated linear attention (heads split over the ranks): one GEMM for q | k | v | gate, the low-rank decay
input in fp32, the recurrence with its norm and gate (``ops.gated_linear_attention``), output projection."""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


class TP_GLA(TPLayer):
    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.heads % world_size:
            raise ValueError(f"{spec.heads} heads cannot be split over {world_size} ranks")
        self.spec, self.heads = spec, spec.heads // world_size
        self.dk, self.dv = pad16(spec.dim), pad16(spec.vdim)

    def cache_spec(self):
        from ..models.kv_cache import StateSpec
        return StateSpec(self.heads, self.dk, self.dv)

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, H, w8 = self.spec, self.heads, pad8(width)
        self.eps = eps

        def heads(name, dim, to):
            return pad_heads(shard(get(prefix + name), self.rank, self.world_size), H, dim, to)

        w = torch.cat([heads("q", s.dim, self.dk), heads("k", s.dim, self.dk), heads("v", s.vdim, self.dv), heads("g", s.vdim, self.dv)])
        self.wqkvg = pad_rows(w, w.shape[0], w8).to(dtype).to(device).contiguous()
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), H, s.vdim, self.dv).t(), w8, H * self.dv).to(dtype).to(device).contiguous()
        a1 = get(prefix + "a1")
        self.a1 = pad_rows(a1, a1.shape[0], w8).to(dtype).to(device).contiguous()
        self.a2 = heads("a2", s.dim, self.dk).float().t().contiguous().to(device)
        self.a2_b = heads("a2.b", s.dim, self.dk).float().contiguous().to(device)
        self.norm_w = pad_rows(get(prefix + "norm").float(), self.dv).to(device)

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        s = self.spec
        qkvg = self.linear(x, self.wqkvg)
        lowrank = ops.narrow_linear(x, self.a1)
        o = ops.gated_linear_attention(qkvg, lowrank, self.a2, self.a2_b, s.tau, self.norm_w, storage["state"], plan.slots,
                                       plan.pos0, plan.cu, s.vdim, s.dim ** -0.5, self.eps, plan.chunk_tables())
        return self.out_linear(o, self.wo)
