"""Tensor-parallel attention over a sliding window (heads split over the ranks), in two kinds that share projections, cache and kernels:

* :class:`TP_SigmoidAttn`: independent sigmoid weights with a distance term and an offset per head, no positions besides; projections
  with biases, RMS norms over the whole of q and of k.
* :class:`TP_DifferentialAttn`: rotary positions, two softmax maps per head, the second taken off, a norm of the difference, one gate
  per head.

Per step: one GEMM for q | k | v (and the gates), one launch that prepares them and writes the cache rows (``ops.qkv_prep``), attention,
output projection.  Rings keep as many rows as the window; prompts read packed rows (``WindowPlan``), so a prompt may come in
portions of any size.  Keys and values are padded to what the tensor-core kernels take; beyond that, and in fp32, the simple kernel runs.
"""
from __future__ import annotations

import math

import torch
import torch.distributed as dist

from .. import ops
from .tp_layer import TPLayer, pad8, pad_heads, pad_rows, shard


def padded_window_dims(dk: int, dv: int):
    """Key and value sizes in the cache."""
    if max(dk, dv) > ops.WINDOW_MAX_DIM:
        raise ValueError(f"attention: heads of {max(dk, dv)} elements (at most {ops.WINDOW_MAX_DIM})")
    if max(dk, dv) <= ops.WINDOW_DIMS[-1]:
        return tuple(next(d for d in ops.WINDOW_DIMS if d >= n) for n in (dk, dv))
    return pad8(dk), pad8(dv)


class TP_WindowAttn(TPLayer):
    """``spec``: heads, kv_heads, dim (of a map), vdim, scale, window (0: none)."""
    maps = 1

    def __init__(self, spec, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        if spec.kv_heads % world_size:
            raise ValueError(f"{spec.kv_heads} KV heads cannot be split over {world_size} ranks")
        self.spec = spec
        self.q_heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.dk, self.dv = padded_window_dims(spec.dim, spec.vdim)
        self.columns = (self.q_heads + self.kv_heads) * self.maps * self.dk + self.kv_heads * self.dv
        self.bias = self.norms = self.gate_col = None
        self.rot = 0

    def cache_spec(self):
        from ..models.kv_cache import WindowKVSpec
        return WindowKVSpec(self.kv_heads, self.maps * self.dk, self.dv, self.spec.window)

    def part(self, get, name: str) -> torch.Tensor:
        return shard(get(name), self.rank, self.world_size)

    def qkv_rows(self, get, prefix: str, suffix: str = "") -> torch.Tensor:
        """Rows of q | k | v, every head padded."""
        s, m = self.spec, self.maps
        sizes = {"q": (self.q_heads * m, s.dim, self.dk), "k": (self.kv_heads * m, s.dim, self.dk), "v": (self.kv_heads, s.vdim, self.dv)}
        return torch.cat([pad_heads(self.part(get, prefix + n + suffix), *sizes[n]) for n in "qkv"])

    def load_projections(self, get, prefix: str, width: int, eps: float, dtype, device, extra: torch.Tensor = None):
        """``extra``: further rows of the input projection."""
        w8 = pad8(width)
        self.eps = eps
        w = self.qkv_rows(get, prefix)
        if extra is not None:
            w = torch.cat([w, pad_rows(extra, pad8(extra.shape[0]))])
        self.w_in = pad_rows(w, w.shape[0], w8).to(dtype).to(device).contiguous()
        wo = shard(get(prefix + "o"), self.rank, self.world_size, 1)
        self.wo = pad_rows(pad_heads(wo.t(), self.q_heads, self.spec.vdim, self.dv).t(), w8, self.q_heads * self.dv).to(dtype).to(device).contiguous()

    def weights(self, plan, device):
        """What turns scores into weights (``ops.SigmoidWeights`` or ``ops.DifferentialWeights``)."""
        raise NotImplementedError

    def rotation(self, plan, device):
        return None

    def mix(self, z: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        """Projected tokens -> concatenated heads [T, H dv]."""
        s, m, T, G = self.spec, self.maps, z.shape[0], self.kv_heads
        wp = plan.window(self.cache_spec())
        ring = (storage["k"], storage["v"], wp.home_rows)
        if plan.decode:
            places = (ring, None)
        else:
            k = torch.empty(wp.total, G, m * self.dk, dtype=z.dtype, device=z.device)
            v = torch.empty(wp.total, G, self.dv, dtype=z.dtype, device=z.device)
            if wp.carry_src is not None:     # before the new tokens may take the place of the old ones
                for new, old in ((k, storage["k"]), (v, storage["v"])):
                    new[wp.carry_dst] = old.view(-1, *new.shape[1:])[wp.carry_src]
            places = ((k, v, wp.packed_rows), ring)
        bias, norms, sumsq = self.bias, self.norms, None
        if norms is not None and self.world_size > 1:       # the norms run over all ranks' heads
            if bias is not None:
                z, bias = z.clone(), None
                z[:, :self.columns] += self.bias.to(z.dtype)
            sumsq = ops.qk_sumsq(z, self.q_heads * m * self.dk, G * m * self.dk)
            dist.all_reduce(sumsq, group=self.group)
        q = ops.qkv_prep(z, self.q_heads * m, G * m, G, self.dk, self.dv, bias, norms, self.eps, self.rotation(plan, z.device), self.rot, plan.positions,
                         *places, sumsq)
        k, v, _ = places[0]
        k = k.view(*k.shape[:-2], G * m, self.dk)
        gate = None if self.gate_col is None else z[:, self.gate_col:]
        args = (q, k, v, self.weights(plan, z.device), s.scale, gate)
        if not ops.window_tensor_cores(q, v, s.scale):
            o = ops.window_attention_simple(*args, *wp.visible())
        elif plan.decode:
            o = ops.window_attention_decode(*args, plan.slots, plan.positions)
        else:
            o = ops.window_attention_prompt(*args, plan.cu, wp.q_pos0, wp.shift, wp.max_q, s.window)
        return o.reshape(T, self.q_heads * self.dv)

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> torch.Tensor:
        return self.out_linear(self.mix(self.linear(x, self.w_in), plan, storage), self.wo)


class TP_SigmoidAttn(TP_WindowAttn):
    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s = self.spec
        self.load_projections(get, prefix, width, eps, dtype, device)
        self.bias = self.qkv_rows(get, prefix, ".b").float().to(device).contiguous()
        qn, kn = (pad_heads(self.part(get, prefix + n + ".norm").float(), h, s.dim, self.dk).to(device).contiguous()
                  for n, h in (("q", self.q_heads), ("k", self.kv_heads)))
        self.norms = (qn, kn, s.heads * s.dim, s.kv_heads * s.dim)
        self.decay = [self.part(get, prefix + n).float() for n in ("r1", "r2", "pb")]
        self.table = None

    def weights(self, plan, device):
        n = self.cache_spec().rows(plan.cache.max_length)
        if self.table is None or self.table.shape[1] < n:
            self.table = ops.distance_table(*self.decay, n).to(device)
        return ops.SigmoidWeights(self.table)


class TP_DifferentialAttn(TP_WindowAttn):
    """``spec`` adds: diff, rot_base, rot_dims, scaling (``ops.BandScaling`` or None)."""
    maps = 2

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        s = self.spec
        self.load_projections(get, prefix, width, eps, dtype, device, self.part(get, prefix + "g"))
        self.gate_col, self.rot = self.columns, s.rot_dims
        one, two = (float((get(prefix + f"lq{i}").double() * get(prefix + f"lk{i}").double()).sum()) for i in (1, 2))
        self.form = ops.DifferentialWeights(math.exp(one) - math.exp(two) + s.diff, 1.0 - s.diff, eps, s.vdim)

    def weights(self, plan, device):
        return self.form

    def rotation(self, plan, device):
        s = self.spec
        return None if not s.rot_dims else ops.rope_table(s.rot_base, s.rot_dims, s.rot_dims, plan.cache.max_length, device, s.scaling)
