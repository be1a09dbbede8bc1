"""Tensor-parallel gated delta rule with short convolutions (heads split over the ranks): one GEMM for q | k | v | gate, decay and
step-size inputs in fp32, everything up to the gate in ``ops.gated_delta_rule``, output projection."""
from __future__ import annotations

import torch

from .. import ops
from .tp_gla import pad16
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


def pad_key_dim(n: int) -> int:
    """Key dim the weights are padded to: one the chunk kernels are compiled for."""
    return next((d for d in (16, 32, 48, 64, 80, 96, 128, 192, 256) if d >= n), pad16(n))


class TP_DeltaRule(TPLayer):
    """``spec``: heads, kv_heads (of q and k), dim, vdim, conv (taps)."""

    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.kv_heads % world_size:
            raise ValueError(f"{spec.kv_heads} key heads cannot be split over {world_size} ranks")
        self.spec = spec
        self.heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.dk, self.dv = pad_key_dim(spec.dim), pad16(spec.vdim)
        if max(self.dk, self.dv) > ops.DELTA_MAX_DIM:
            raise ValueError(f"delta rule: heads of at most {ops.DELTA_MAX_DIM} elements")
        self.channels = 2 * self.kv_heads * self.dk + self.heads * self.dv

    def cache_spec(self):
        from ..models.kv_cache import DeltaSpec
        return DeltaSpec(self.heads, self.dk, self.dv, self.channels, self.spec.conv)

    @property
    def columns(self) -> int:
        return self.channels + self.heads * self.dv

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, w8 = self.spec, pad8(width)
        self.eps = eps
        dims = {"q": (self.kv_heads, s.dim, self.dk), "k": (self.kv_heads, s.dim, self.dk), "v": (self.heads, s.vdim, self.dv),
                "g": (self.heads, s.vdim, self.dv)}

        def part(name):
            return shard(get(prefix + name), self.rank, self.world_size)

        w = torch.cat([pad_heads(part(n), *dims[n]) for n in "qkvg"])
        self.w_in = pad_rows(w, w.shape[0], w8).to(dtype).to(device).contiguous()
        self.conv_w = torch.cat([pad_heads(part(n + ".conv").float(), *dims[n]) for n in "qkv"]).to(device).contiguous()
        ab = torch.cat([part("a"), part("b")])
        self.ab = pad_rows(ab, ab.shape[0], w8).to(dtype).to(device).contiguous()
        self.a_log, self.dt_bias = (part(n).float().to(device).contiguous() for n in ("A_log", "dt_bias"))
        self.norm_w = pad_rows(get(prefix + "norm").float(), self.dv).to(device)
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), self.heads, s.vdim, self.dv).t(), w8, self.heads * self.dv).to(dtype).to(device).contiguous()

    def mix(self, x: torch.Tensor, z: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        """Input ``x`` and its projection ``z`` (q | k | v | gate) -> gated heads [T, H dv]."""
        s = self.spec
        return ops.gated_delta_rule(z, ops.narrow_linear(x, self.ab), self.conv_w, self.a_log, self.dt_bias, self.norm_w, storage["state"],
                                    storage["conv"], plan.slots, plan.pos0, plan.cu, self.kv_heads, s.vdim, s.dim ** -0.5, self.eps,
                                    plan.chunk_tables())

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> ops.SublayerOutput:
        return ops.SublayerOutput(self.out_linear(self.mix(x, self.linear(x, self.w_in), plan, storage), self.wo))
