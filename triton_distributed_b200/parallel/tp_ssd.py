"""Tensor-parallel state space layer (heads and groups split over the ranks): one GEMM for gate | x | B | C | step sizes, convolutions and
recurrence in ``ops.state_space``, gate and norm over groups, output projection."""
from __future__ import annotations

import torch

from .. import ops
from .tp_delta import pad_key_dim
from .tp_gla import pad16
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


class TP_StateSpace(TPLayer):
    """``spec``: heads, groups, state, vdim, conv (taps), norm_groups."""

    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.groups % world_size or spec.norm_groups % world_size:
            raise ValueError(f"{spec.groups} groups and {spec.norm_groups} norm groups cannot be split over {world_size} ranks")
        self.spec = spec
        self.heads, self.groups, self.parts = (n // world_size for n in (spec.heads, spec.groups, spec.norm_groups))
        self.dk, self.dv = pad_key_dim(spec.state), pad16(spec.vdim)
        if max(self.dk, self.dv) > ops.SSD_MAX_DIM:
            raise ValueError(f"state space layer: states and heads of at most {ops.SSD_MAX_DIM} elements")
        self.inner = self.heads * self.dv
        self.channels = self.inner + 2 * self.groups * self.dk

    def cache_spec(self):
        from ..models.kv_cache import DeltaSpec
        return DeltaSpec(self.heads, self.dk, self.dv, self.channels, self.spec.conv)

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, w8 = self.spec, pad8(width)
        self.eps = eps
        inner, shared = s.heads * s.vdim, s.groups * s.state
        head, state = (self.heads, s.vdim, self.dv), (self.groups, s.state, self.dk)

        def cut(t, sizes, pads):
            """Consecutive parts of ``t``, each sharded and padded head by head (None: as it is)."""
            out = [shard(p, self.rank, self.world_size) for p in t.split(sizes)]
            return torch.cat([p if pad is None else pad_heads(p, *pad) for p, pad in zip(out, pads)])

        def fp32(t):
            return t.float().to(device).contiguous()

        w = cut(get(prefix + "in"), [inner, inner, shared, shared, s.heads], [head, head, state, state, None])
        self.dt_col = self.channels                                  # counted from x on
        self.w_in = pad_rows(w, pad8(w.shape[0]), w8).to(dtype).to(device).contiguous()
        conv = [cut(get(prefix + n), [inner, shared, shared], [head, state, state]) for n in ("conv", "conv.b")]
        per_head = (shard(get(prefix + n), self.rank, self.world_size) for n in ("A_log", "dt_bias", "D"))
        self.w = ops.SsdWeights(*(fp32(t) for t in (*conv, *per_head)))
        self.norm_w = fp32(cut(get(prefix + "norm"), [inner], [head]))
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), *head).t(), w8, self.inner).to(dtype).to(device).contiguous()

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        z = self.linear(x, self.w_in)
        y = ops.state_space(z[:, self.inner:], self.dt_col, self.w, storage["state"], storage["conv"], plan.slots, plan.pos0, plan.cu, self.groups,
                            plan.chunk_tables())
        return self.out_linear(ops.gated_group_norm(y, z, self.norm_w, self.heads, self.spec.vdim, self.parts, self.eps), self.wo)
