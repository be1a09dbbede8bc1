"""Common part of the decoders whose configuration lists the layers one by one (Vasolix, Lisenex, Tazitar, Bagasun): loading, execution modes,
cache, packed steps, the engine's rectangular interface, random weights by tensor name.

A model is a list of layers with ``parts()`` (tensor-parallel mixers / feed-forwards) and ``load``; a subclass builds them and runs
the tokens of a step through them (``hidden``) on an fp32 residual stream.
"""
from __future__ import annotations

import dataclasses
import json
import os
from typing import List, Optional, Sequence

import torch

from .. import ops
from ..parallel.tp_layer import pad8, pad_rows
from ..runtime import get_runtime
from .config import ModelConfig
from .kv_cache import HybridCache, StepPlan
from .safetensors_io import ShardedCheckpoint


def read_config(path: str) -> dict:
    """``config.json`` of a checkpoint directory (or the file itself)."""
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        return json.load(f)


class LayeredConfig:
    """What the configurations (frozen dataclasses with a tuple ``layers``) have in common."""

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def with_num_layers(self, n: int):
        """The first ``n`` layers (the list is repeated when it is shorter)."""
        return dataclasses.replace(self, layers=tuple(self.layers[i % len(self.layers)] for i in range(n)))


class LayeredLLM:
    """Same interface as :class:`DenseLLM` (``set_fwd``, ``init_ctx_for``, ``inference``, ``finalize``), plus packed steps
    (``forward_step``) over a :class:`HybridCache` made by ``new_cache``."""

    random_weights = None       # class of the random tensors

    def __init__(self, model_config: ModelConfig, group=None):
        self.rt = get_runtime()
        self.model_config = model_config
        self.arch = model_config.arch()
        self.rank, self.world_size = self.rt.rank, self.rt.world_size
        self.group = group if group is not None else self.rt.group
        self.dtype, self.device = model_config.dtype, self.rt.device
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"{type(self).__name__} runs in bfloat16 or float32")
        if self.dtype == torch.float32 and self.rt.is_cuda:
            torch.backends.cuda.matmul.allow_tf32 = False      # 32-bit means 32-bit
        self.mode = "torch"
        self.layers = self.make_layers()
        self.init_parameters()
        self.set_fwd("torch")

    def make_layers(self) -> list:
        raise NotImplementedError

    def hidden(self, ids: torch.Tensor, plan: StepPlan, streams: Optional[List[torch.Tensor]]):
        """The residual stream [T, W] after the last layer (or what ``final_hidden`` takes); ``streams`` collects it after every layer."""
        raise NotImplementedError

    def final_hidden(self, x, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """What the output projection reads: the normed rows of what ``hidden`` returned."""
        return ops.stream_norm(x, self.final_norm_w, self.arch.hidden_size, self.arch.rms_norm_eps, self.dtype, rows)

    def cache_specs(self) -> list:
        """Storage of every layer in the order in which they run."""
        return [l.mixer.cache_spec() for l in self.layers]

    # -- parameters -------------------------------------------------------------------------------------------
    def table(self, get, name: str) -> torch.Tensor:
        """[vocab, width] tensor, padded."""
        return pad_rows(get(name), pad8(self.arch.vocab_size), pad8(self.arch.hidden_size)).to(self.dtype).to(self.device).contiguous()

    def load_head(self, get):
        """Embedding table and output projection."""
        raise NotImplementedError

    def final_norm(self, get) -> torch.Tensor:
        """fp32 weight of the norm before the output projection."""
        return pad_rows(get("final.norm").float(), pad8(self.arch.hidden_size)).to(self.device)

    def init_parameters(self):
        a, mc = self.arch, self.model_config
        if mc.checkpoint_dir:
            ckpt = ShardedCheckpoint(mc.checkpoint_dir)
            get = ckpt.get
        else:
            ckpt, get = None, self.random_weights(a, mc.seed, self.device)
        self.load_head(get)
        self.final_norm_w = self.final_norm(get)
        for l in self.layers:
            l.load(get, a.hidden_size, a.rms_norm_eps, self.dtype, self.device)
        if ckpt is not None:
            ckpt.close()

    # -- modes ------------------------------------------------------------------------------------------------
    def set_fwd(self, mode: str = "torch"):
        self.mode = mode
        for l in self.layers:
            for part in l.parts():
                part.set_fwd(mode)

    def init_ctx_for(self, mode: str, max_M: int):
        """Communication contexts of the row-parallel projections, one set for all layers (nothing to do on one rank).
        The batch-sharded mode of the dense models runs as the all-reduce mode here."""
        if mode == "torch" or self.world_size == 1:
            return
        w8 = pad8(self.arch.hidden_size)
        first = self.layers[0].mixer
        first.init_ctx(mode, max_M, w8)
        for l in self.layers:
            for part in l.parts():
                part.ar_ctx, part.gemm_ar_ctx = first.ar_ctx, first.gemm_ar_ctx

    def finalize(self):
        self.layers[0].mixer.finalize()
        for l in self.layers:
            for part in l.parts():
                part.ar_ctx = part.gemm_ar_ctx = None

    def new_cache(self, batch_size: int, max_length: int, allocate: bool = True) -> HybridCache:
        return HybridCache(self.cache_specs(), batch_size, max_length, self.dtype, self.device, allocate)

    # -- forward ----------------------------------------------------------------------------------------------
    @torch.no_grad()
    def forward_step(self, ids: torch.Tensor, plan: StepPlan, rows: Optional[torch.Tensor] = None,
                     wo_lm_head: bool = False, streams: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """One step over packed tokens ``ids`` [T]: fp32 logits [len(rows), vocab] of the given token rows (None: all), or
        the normed hidden rows.  The caller advances the cache.  ``streams`` collects the residual stream after every
        layer (a debugging aid)."""
        h = self.final_hidden(self.hidden(ids, plan, streams), rows)
        if wo_lm_head:
            return h
        logits = torch.matmul(h, self.lm_head.t()) if self.mode == "torch" else ops.gemm(h, self.lm_head)
        return logits[:, :self.arch.vocab_size].float()

    def inference(self, input_ids: torch.Tensor, position_ids: torch.Tensor, kv_cache: HybridCache, wo_lm_head: bool = False,
                  seq_lens: Optional[Sequence[int]] = None) -> torch.Tensor:
        """``input_ids`` [B, S] -> fp32 logits [B, vocab] of every sequence's last token.  S = 1 is a decode step at
        ``position_ids`` (device values, graph-capturable); longer inputs continue every sequence where the cache stands,
        right-padded to S when ``seq_lens`` gives their lengths (padding is dropped before the first layer)."""
        B, S = input_ids.shape
        if S == 1:
            return self.forward_step(input_ids.reshape(-1), kv_cache.decode_plan(position_ids), None, wo_lm_head)
        lens = [S] * B if seq_lens is None else [int(n) for n in seq_lens]
        ids = input_ids.reshape(-1) if min(lens) == S else torch.cat([input_ids[b, :n] for b, n in enumerate(lens)])
        plan = kv_cache.plan(range(B), lens)
        return self.forward_step(ids, plan, None if plan.decode else plan.last_rows, wo_lm_head)


class RandomWeights:
    """Random tensors with the shapes of the checkpoint format (weights ~ N(0, 1/fan_in), norms near 1)."""

    def __init__(self, arch, seed: int, device):
        self.arch, self.device = arch, device
        self.gen = torch.Generator(device=device).manual_seed(seed)

    def shape(self, name: str):
        raise NotImplementedError

    def value(self, name: str, t: torch.Tensor) -> torch.Tensor:
        """Standard normal ``t`` -> the tensor ``name``."""
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            return 1.0 + 0.1 * t
        if name == "embed":
            return t
        return t * t.shape[-1] ** -0.5

    def __call__(self, name: str) -> torch.Tensor:
        t = torch.randn(*self.shape(name), generator=self.gen, device=self.device)
        return self.value(name, t).to(torch.bfloat16)
