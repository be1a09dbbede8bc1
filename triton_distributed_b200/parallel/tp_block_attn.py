"""Tensor-parallel block-local attention with a sink per head, an output gate, whole-projection q / k norms and values tied
to the raw keys.  Positions do not enter the scores except through the mask.

Per step: one GEMM for q | k | gate, one kernel that norms q, stores the raw keys with their norm factors
(``ops.qk_norm_tied``; the key norm's weight and the score scale ride on the query), attention with sink and gate in its
epilogue, output projection.  A query of block b sees positions of block b only, so a prompt is cut into (sequence, block)
pairs that the var-len kernels take as sequences of their own, and the cache keeps one block per sequence.
"""
from __future__ import annotations

import torch
import torch.distributed as dist

from .. import ops
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


def padded_head_dim(dim: int) -> int:
    """Head dim the weights are padded to: that of the next tensor-core kernel, beyond them a multiple of eight."""
    return next((d for d in ops.TIED_TENSOR_CORE_DIMS if d >= dim), pad8(dim))


class TP_BlockAttn(TPLayer):
    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.kv_heads % world_size:
            raise ValueError(f"{spec.kv_heads} KV heads cannot be split over {world_size} ranks")
        self.spec = spec
        self.q_heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.head_dim = padded_head_dim(spec.dim)

    def cache_spec(self):
        from ..models.kv_cache import TiedKVSpec
        return TiedKVSpec(self.kv_heads, self.head_dim, self.spec.block)

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, D, w8 = self.spec, self.head_dim, pad8(width)
        self.eps = eps
        self.n_q, self.n_k = self.q_heads * D, self.kv_heads * D

        def heads(name, n):
            t = shard(get(prefix + name), self.rank, self.world_size)
            return pad_heads(t, n, s.dim, D)

        wq, wk, wg = heads("q", self.q_heads), heads("k", self.kv_heads), heads("g", self.q_heads)
        self.wqkg = pad_rows(torch.cat([wq, wk, wg]), self.n_q * 2 + self.n_k, w8).to(dtype).to(device).contiguous()
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), self.q_heads, s.dim, D).t(), w8, self.n_q).to(dtype).to(device).contiguous()
        qn = heads("q.norm", self.q_heads).float().reshape(self.kv_heads, -1, D)
        kn = heads("k.norm", self.kv_heads).float().reshape(self.kv_heads, 1, D)
        self.q_weight = (qn * kn * s.scale).reshape(-1).to(device).contiguous()
        self.sink = shard(get(prefix + "sink"), self.rank, self.world_size).float().to(device).contiguous()

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        s, D = self.spec, self.head_dim
        T = x.shape[0]
        bp = plan.blocks(self.cache_spec())
        qkg = self.linear(x, self.wqkg)
        gate = qkg[:, self.n_q + self.n_k:]
        sumsq = None
        if self.world_size > 1:
            sumsq = ops.qk_sumsq(qkg, self.n_q, self.n_k)
            dist.all_reduce(sumsq, group=self.group)
        home = (storage["k"], storage["scale"], bp.home_rows)
        norm = (qkg, self.q_weight, self.n_k, s.heads * s.dim, s.kv_heads * s.dim, self.eps)
        tensor_cores = x.is_cuda and x.dtype == torch.bfloat16 and D in ops.TIED_TENSOR_CORE_DIMS
        if plan.decode:
            q = ops.qk_norm_tied(*norm, home, None, sumsq).reshape(T, self.q_heads, D)
            if tensor_cores:
                rows = storage["k"].shape[1]
                splits = ops.pick_tied_splits(T, self.kv_heads, (self.q_heads // self.kv_heads + 15) // 16, rows)
                o = ops.tied_attn_decode(q, storage["k"], storage["scale"], bp.block_table, bp.kv_lens, rows, splits, self.sink, gate)
            else:
                o = ops.tied_attention_simple(q, storage["k"], storage["scale"], bp.row0, bp.n_keys, self.sink, gate)
        else:
            k = torch.empty(bp.pages, bp.page_rows, self.kv_heads, D, dtype=x.dtype, device=x.device)
            scale = torch.empty(bp.pages, bp.page_rows, dtype=torch.float32, device=x.device)
            if bp.carry_src is not None:     # before the new keys may take the place of the old block's
                k.view(-1, self.n_k)[bp.carry_dst] = storage["k"].view(-1, self.n_k)[bp.carry_src]
                scale.view(-1)[bp.carry_dst] = storage["scale"].view(-1)[bp.carry_src]
            q = ops.qk_norm_tied(*norm, (k, scale, bp.scratch_rows), home, sumsq).reshape(T, self.q_heads, D)
            if tensor_cores:
                o = ops.tied_attn_varlen(q, k, scale, bp.block_table, bp.cu, bp.q_pos0, bp.kv_lens, bp.max_q, bp.max_kv,
                                         self.sink, gate)
            else:
                o = ops.tied_attention_simple(q, k, scale, bp.row0, bp.n_keys, self.sink, gate)
        return self.out_linear(o.reshape(T, self.n_q), self.wo)
