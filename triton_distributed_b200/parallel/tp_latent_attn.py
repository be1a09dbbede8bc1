"""Tensor-parallel latent attention with an output gate: heads split over the ranks, the latent projection and its cache row
replicated.  A layer may use the rows of an earlier layer (``kv_from``) in place of its own.

Decoding (and fp32, and sizes the prompt kernel does not take) runs the absorbed form: one GEMM for q | latent | gate, one launch
for W_uk^T q, rotations, latent norm and cache write, attention over the cached rows, one launch for the merge of its splits, W_uv
and the gate.  bf16 prompts run the expanded form: keys and transposed values of the visible tokens by two GEMMs over the packed
rows, then the tcgen05 kernel with the gate in its epilogue.  Returns the output projection's partial sums: parallel layers add
the feed-forward's before the ranks' sum.
"""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


class TP_LatentAttn(TPLayer):
    def __init__(self, spec, index: int, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.heads % world_size:
            raise ValueError(f"{spec.heads} heads cannot be split over {world_size} ranks")
        self.spec, self.index, self.heads = spec, index, spec.heads // world_size
        self.d, self.r, self.dv, self.R = pad8(spec.dim), pad8(spec.rot_dim), pad8(spec.vdim), pad8(spec.kv_rank)
        if self.R + self.r > 1024:
            raise ValueError("latent attention: rows of more than 1024 elements")
        self.own_kv = spec.kv_from is None
        self.source = index if self.own_kv else spec.kv_from     # layer whose rows are read
        self.shared = False                                      # another layer reads this one's rows

    def cache_spec(self):
        from ..models.kv_cache import LatentSpec, SharedSpec
        return LatentSpec(self.R, self.r) if self.own_kv else SharedSpec(self.source)

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s, H, w8 = self.spec, self.heads, pad8(width)
        self.eps = eps

        def heads(name, dim, to):
            return pad_heads(shard(get(prefix + name), self.rank, self.world_size), H, dim, to)

        def final(t):
            return t.to(dtype).to(device).contiguous()

        q = shard(get(prefix + "q"), self.rank, self.world_size).reshape(H, s.dim + s.rot_dim, -1)
        parts = [torch.cat([pad_rows(q[:, :s.dim], H, self.d), pad_rows(q[:, s.dim:], H, self.r)], dim=1).flatten(0, 1)]
        self.norm_w = None
        if self.own_kv:
            dkv = get(prefix + "dkv")
            parts += [pad_rows(dkv[:s.kv_rank], self.R), pad_rows(dkv[s.kv_rank:], self.r)]
            self.norm_w = pad_rows(get(prefix + "dkv.norm").float(), self.R).to(device)
        self.n_q = H * (self.d + self.r)
        self.gate0 = sum(p.shape[0] for p in parts)
        parts.append(heads("g", s.vdim, self.dv))
        w = torch.cat(parts)
        self.w_in = final(pad_rows(w, w.shape[0], w8))
        uk = pad_rows(heads("uk", s.dim, self.d), H * self.d, self.R)
        self.uk = final(uk)                                                       # [H d, R]
        self.uk_t = final(uk.reshape(H, self.d, self.R).transpose(1, 2))          # [H, R, d]
        self.uv = final(pad_rows(heads("uv", s.vdim, self.dv), H * self.dv, self.R)).view(H, self.dv, self.R)
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = final(pad_rows(pad_heads(wo.t(), H, s.vdim, self.dv).t(), w8, H * self.dv))

    def _table(self, plan):
        return ops.rope_table(self.spec.rot_base, self.spec.rot_dim, self.r, plan.cache.max_length, plan.positions.device)

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        s, lp, rows = self.spec, plan.latent(), storage["latent"]
        z = self.linear(x, self.w_in)
        gate = z[:, self.gate0:]
        home = (rows, lp.home_rows) if self.own_kv else None
        norm = (self.norm_w, s.kv_rank, self.eps, self._table(plan), plan.positions)
        tensor_cores = x.is_cuda and x.dtype == torch.bfloat16
        if not plan.decode and tensor_cores and ops.latent_prefill_supported(self.d, self.r, self.dv, s.scale):
            return self.linear(self._expanded(z, gate, plan, lp, rows, home, norm), self.wo)
        q = ops.latent_absorb(z, self.uk_t, self.r, *norm, home)
        if plan.decode and tensor_cores and ops.latent_decode_supported(self.R, self.r, s.scale):
            o, ml = ops.latent_decode(q, rows, plan.slots, lp.kv_lens, self.R, s.scale)
        else:
            o, ml = ops.latent_attention(q, rows, lp.row0, lp.n_keys, self.R, s.scale), None
        return self.linear(ops.latent_out(o, ml, self.uv, gate), self.wo)

    def _expanded(self, z, gate, plan, lp, rows, home, norm):
        norm_w, R_real, eps, table, pos = norm
        W = self.R + self.r
        ctx = None if self.own_kv else plan.contexts.get(self.source)
        fresh = ctx is None
        if fresh:
            ctx = torch.zeros(lp.ctx_len, W, dtype=z.dtype, device=z.device)
            if lp.carry_src is not None:
                ctx[lp.carry_dst] = rows.view(-1, W)[lp.carry_src]
            if self.shared or not self.own_kv:
                plan.contexts[self.source] = ctx
        ops.latent_rotate(z, self.heads, self.d, self.r, norm_w, self.R, R_real, eps, table, pos, home,
                          (ctx, lp.ctx_rows) if self.own_kv else None)
        if fresh and not self.own_kv:              # the layer that owns the rows ran in the other form
            ctx[lp.ctx_rows] = rows.view(-1, W)[lp.home_rows]
        k = self.linear(ctx[:, :self.R], self.uk)
        vt = self.linear(self.uv.view(-1, self.R), ctx[:, :self.R])
        return ops.latent_prefill(z, k, ctx, vt, plan.cu, lp.q_pos0, lp.kv_lens, lp.ctx0, lp.max_q, self.heads, self.d, self.r,
                                  self.dv, self.spec.scale, gate)
