"""Tensor-parallel causal attention with rotary positions on (part of) a head and the usual options, each a parameter: per-head q / k
norms with a weight before the rotation, weightless ones after it, either pairing, YaRN frequencies, value heads of another size, a
soft cap on the scores, a sink (learned per head, or one fixed number).

Per step: one GEMM for q | k | v, one launch that norms, rotates and writes the cache rows (``ops.head_prep``), attention over the
cache, output projection.  Prompts read the cache as well, so a prompt may come in portions of any size.  Query / key and value heads
are padded to one head dim that the tensor-core kernels take; beyond them, and in fp32, the simple kernel runs.
"""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


def padded_head_dim(dim: int, vdim: int) -> int:
    """Common head dim of keys and values in the cache."""
    d = max(dim, vdim)
    for p in ops.TENSOR_CORE_DIMS + (512, 1024):
        if p >= d:
            return p
    raise ValueError(f"attention: heads of {d} elements (at most 1024)")


class TP_RotaryAttn(TPLayer):
    """``spec``: heads, kv_heads, dim, vdim, scale, softcap (0: none), rot_base, rot_dims, scaling (``ops.YarnScaling`` or None),
    interleaved, qk_norm, unit, sink ("learned", a number, or None)."""

    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.kv_heads % world_size:
            raise ValueError(f"{spec.kv_heads} KV heads cannot be split over {world_size} ranks")
        self.spec = spec
        self.q_heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.head_dim = padded_head_dim(spec.dim, spec.vdim)

    def cache_spec(self):
        from ..models.kv_cache import KVSpec
        return KVSpec(self.kv_heads, self.head_dim)

    @property
    def columns(self) -> int:
        return (self.q_heads + 2 * self.kv_heads) * self.head_dim

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, D, w8 = self.spec, self.head_dim, pad8(width)
        self.eps = eps

        def heads(name, n, dim):
            return pad_heads(shard(get(prefix + name), self.rank, self.world_size), n, dim, D)

        w = torch.cat([heads("q", self.q_heads, s.dim), heads("k", self.kv_heads, s.dim), heads("v", self.kv_heads, s.vdim)])
        self.w_in = pad_rows(w, w.shape[0], w8).to(dtype).to(device).contiguous()
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), self.q_heads, s.vdim, D).t(), w8, self.q_heads * D).to(dtype).to(device).contiguous()
        self.q_w = self.k_w = self.sink = None
        if s.qk_norm:
            self.q_w, self.k_w = (pad_rows(get(prefix + n).float(), D).to(device) for n in ("q.norm", "k.norm"))
        if s.sink == "learned":
            self.sink = shard(get(prefix + "sink"), self.rank, self.world_size).float().to(device).contiguous()
        elif s.sink is not None:
            self.sink = torch.full((self.q_heads,), float(s.sink), device=device)

    def mix(self, z: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        """Projected tokens (q | k | v in the first columns) -> concatenated heads [T, H D]."""
        s, D, T, kp = self.spec, self.head_dim, z.shape[0], plan.kv()
        k, v = storage["k"], storage["v"]
        table = ops.rope_table(s.rot_base, s.rot_dims, s.rot_dims, plan.cache.max_length, z.device, s.scaling)
        q = ops.head_prep(z, self.q_heads, self.kv_heads, D, s.dim, self.q_w, self.k_w, s.unit, self.eps, table, s.rot_dims, s.interleaved,
                          plan.positions, k, v, kp.home_rows)
        if z.is_cuda and z.dtype == torch.bfloat16 and D in ops.TENSOR_CORE_DIMS:
            if plan.decode:
                o = ops.gqa_fwd_batch_decode(q, k, v, None, None, kp.kv_lens, kp.block_table, s.scale, s.softcap, sink=self.sink)
            else:
                o = ops.flash_attn_varlen(q, k, v, kp.block_table, plan.cu, kp.kv_lens, kp.max_q, kp.q_pos0, True, s.scale, s.softcap,
                                          max_kv_len=kp.max_kv, sink=self.sink)
        else:
            o = ops.attention_simple(q, k, v, kp.row0, kp.n_keys, self.sink, s.scale, s.softcap)
        return o.reshape(T, self.q_heads * D)

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> ops.SublayerOutput:
        return ops.SublayerOutput(self.out_linear(self.mix(self.linear(x, self.w_in), plan, storage), self.wo))
