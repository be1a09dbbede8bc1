"""Two tensor-parallel mixers side by side on the same input.  Their projections are one GEMM; the sublayer's output is half the sum
of the two outputs, each normed over the model width, which the pass over the residual streams computes (``ops.SublayerOutput`` with
two branches).  In decode steps on one rank the branches run on two streams."""
from __future__ import annotations

import torch

from .. import ops
from .tp_layer import TPLayer, pad8, pad_rows


class TP_TwinMixer(TPLayer):
    """``left``: a mixer with ``mix(z, plan, storage)``; ``right``: one with ``mix(x, z, plan, storage)``."""

    _side = {}          # second stream per device

    def __init__(self, left: TPLayer, right: TPLayer, rank: int = 0, world_size: int = 1, group=None):
        super().__init__(rank, world_size, group)
        self.left, self.right = left, right

    def cache_spec(self):
        from ..models.kv_cache import GroupSpec
        return GroupSpec((self.left.cache_spec(), self.right.cache_spec()))

    def load(self, get, prefix: str, width: int, eps: float, dtype, device):
        for part, name in ((self.left, "left."), (self.right, "right.")):
            part.load(get, prefix + name, width, eps, dtype, device)
        self.w_in = torch.cat([self.left.w_in, self.right.w_in]).contiguous()
        n = self.left.columns
        self.left.w_in, self.right.w_in = self.w_in[:n], self.w_in[n:]
        self.left_w, self.right_w = (pad_rows(get(prefix + f"{s}.out").float(), pad8(width)).to(device) for s in ("left", "right"))

    def _left(self, z, plan, storage):
        return self.left.out_linear(self.left.mix(z, plan, storage), self.left.wo)

    def _right(self, x, z, plan, storage):
        return self.right.out_linear(self.right.mix(x, z[:, self.left.columns:], plan, storage), self.right.wo)

    def __call__(self, x: torch.Tensor, plan, storage: dict) -> ops.SublayerOutput:
        z = self.linear(x, self.w_in)
        if not (plan.decode and x.is_cuda and self.world_size == 1):
            a, b = self._left(z, plan, storage), self._right(x, z, plan, storage)
        else:
            side = self._side.get(x.device)
            if side is None:
                side = self._side[x.device] = torch.cuda.Stream(device=x.device)
            # a tensor of one stream's pool is reused by that stream alone, which has waited for the other by then: each waits for
            # the other once per call
            main = torch.cuda.current_stream()
            side.wait_stream(main)
            with torch.cuda.stream(side), ops.scratch_lane(1):
                b = self._right(x, z, plan, storage)
            a = self._left(z, plan, storage)
            main.wait_stream(side)
        return ops.SublayerOutput(a, b, self.left_w, self.right_w)
