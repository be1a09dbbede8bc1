"""Vasolix: a decoder whose layers are listed one by one, each with its own mixer and feed-forward.

Mixers: block-local attention with a sink, an output gate, whole-projection q / k norms and values tied to the raw keys
(``parallel.TP_BlockAttn``), and gated linear attention with a per-channel decay (``parallel.TP_GLA``).  Feed-forward: a
mixture of experts with independent sigmoid scores, squared-ReLU experts and a gated shared expert
(``parallel.TP_SigmoidMoE``), or none.  Norms act on the sublayers' outputs; the residual stream is fp32.

The configuration is a ``config.json`` with ``"architecture": "Vasolix"``: ``vocab``, ``width``, ``norm.eps`` and ``layers``, a
list of ``{type, mixer, mlp}``.  Tensors are named ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.mlp.*``,
``final.norm``, ``head``.  Activations are bf16 (with everything sensitive in fp32) or, with ``ModelConfig.dtype =
torch.float32``, fp32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from .. import ops
from ..parallel.tp_block_attn import TP_BlockAttn
from ..parallel.tp_gla import TP_GLA
from ..parallel.tp_layer import pad8, pad_rows
from ..parallel.tp_sigmoid_moe import TP_SigmoidMoE
from .kv_cache import StepPlan
from .layered import LayeredConfig, LayeredLLM, RandomWeights, read_config


# ------------------------------------------------------------------ configuration
@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    block: int = 0               # 0 = plain causal attention

    @staticmethod
    def from_json(c: dict) -> "AttentionSpec":
        if c.get("vdim", c["dim"]) != c["dim"]:
            raise ValueError("attention: the values are the keys, so vdim must equal dim")
        if c["heads"] % c["kv_heads"]:
            raise ValueError("attention: heads must be a multiple of kv_heads")
        mask = c.get("mask") or {}
        return AttentionSpec(c["heads"], c["kv_heads"], c["dim"], float(c["scale"]), int(mask.get("size", 0)))


@dataclass(frozen=True)
class GLASpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16               # of the decay's low-rank input; a checkpoint's tensors decide

    @staticmethod
    def from_json(c: dict) -> "GLASpec":
        return GLASpec(c["heads"], c["dim"], c["vdim"], float(c["tau"]))


@dataclass(frozen=True)
class MoESpec:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0           # 0 = no shared expert

    @staticmethod
    def from_json(c: Optional[dict]) -> Optional["MoESpec"]:
        if c is None:
            return None
        if c.get("kind", "moe") != "moe":
            raise ValueError(f"unknown feed-forward kind {c['kind']!r}")
        shared = c.get("shared")
        return MoESpec(c["router"]["experts"], c["router"]["top"], c["expert"]["ff"], shared["ff"] if shared else 0)


MIXERS = {"attention": (AttentionSpec, TP_BlockAttn), "gla": (GLASpec, TP_GLA)}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: Optional[MoESpec]

    @staticmethod
    def from_json(c: dict) -> "LayerSpec":
        if c["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {c['type']!r}; known: {sorted(MIXERS)}")
        return LayerSpec(c["type"], MIXERS[c["type"]][0].from_json(c["mixer"]), MoESpec.from_json(c.get("mlp")))


@dataclass(frozen=True)
class VasolixConfig(LayeredConfig):
    name: str
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    layers: Tuple[LayerSpec, ...]

    @property
    def is_moe(self) -> bool:
        return any(l.mlp is not None for l in self.layers)

    @staticmethod
    def from_json(path: str) -> "VasolixConfig":
        c = read_config(path)
        return VasolixConfig(c["architecture"], c["vocab"], c["width"], float(c["norm"]["eps"]),
                             tuple(LayerSpec.from_json(l) for l in c["layers"]))


def hybrid_stack(name: str, vocab: int, width: int, pattern: str, attention: AttentionSpec, gla: GLASpec, moe: Optional[MoESpec],
                 eps: float = 1e-5) -> VasolixConfig:
    """A configuration from a pattern string: "A" = attention layer, "G" = gated-linear-attention layer."""
    kinds = {"A": ("attention", attention), "G": ("gla", gla)}
    return VasolixConfig(name, vocab, width, eps, tuple(LayerSpec(*kinds[k], moe) for k in pattern))


VASOLIX_PRESETS = {
    # layers of the size of Qwen3-30B-A3B's (width, heads, experts)
    "vasolix-30b-a3b": hybrid_stack("vasolix-30b-a3b", 151936, 2048, "GA" * 24, AttentionSpec(32, 4, 128, 128 ** -0.5, 4096),
                                    GLASpec(16, 128, 128, 16.0), MoESpec(128, 8, 768, 768)),
    # layers of the size of a small dense model's, head dim 64
    "vasolix-1b": hybrid_stack("vasolix-1b", 65536, 1536, "GA" * 12, AttentionSpec(24, 4, 64, 0.125, 1024),
                               GLASpec(12, 64, 128, 16.0), MoESpec(32, 4, 512, 512)),
    "tiny-vasolix": hybrid_stack("tiny-vasolix", 1000, 192, "AGA", AttentionSpec(6, 2, 64, 0.11, 40),
                                 GLASpec(3, 48, 32, 8.0, rank=8), MoESpec(6, 2, 80, 112)),
}


# ------------------------------------------------------------------ model
class VasolixLayer:
    def __init__(self, index: int, spec: LayerSpec, rank: int, world_size: int, group):
        self.index, self.spec = index, spec
        self.mixer = MIXERS[spec.type][1](spec.mixer, rank, world_size, group)
        self.mlp = TP_SigmoidMoE(spec.mlp, rank, world_size, group) if spec.mlp is not None else None
        self.norm1 = self.norm2 = None

    def parts(self):
        return [self.mixer] + ([self.mlp] if self.mlp is not None else [])

    def load(self, get, width: int, eps: float, dtype, device):
        p = f"l{self.index}."
        w8 = pad8(width)
        self.width, self.eps = width, eps
        self.norm1 = pad_rows(get(p + "norm1").float(), w8).to(device)
        self.mixer.load(get, p + "mix.", width, eps, dtype, device)
        if self.mlp is not None:
            self.norm2 = pad_rows(get(p + "norm2").float(), w8).to(device)
            self.mlp.load(get, p + "mlp.", width, dtype, device)

    def fwd(self, x: torch.Tensor, xb: torch.Tensor, plan: StepPlan, storage: dict):
        """Both sublayers read the stream itself; a sublayer's output is normed on its way into it."""
        y = self.mixer(xb, plan, storage)
        ops.postnorm_add(x, xb, y, self.norm1, self.width, self.eps)
        if self.mlp is not None:
            y, rows, shared, gate = self.mlp(xb)
            ops.postnorm_add(x, xb, y, self.norm2, self.width, self.eps, rows, shared, gate)


class VasolixLLM(LayeredLLM):
    def make_layers(self):
        return [VasolixLayer(i, s, self.rank, self.world_size, self.group) for i, s in enumerate(self.arch.layers)]

    def load_head(self, get):
        self.embed_tokens, self.lm_head = self.table(get, "embed"), self.table(get, "head")

    def hidden(self, ids, plan, streams):
        x, xb = ops.embed_stream(ids, self.embed_tokens)
        for l, storage in zip(self.layers, plan.cache.layers):
            l.fwd(x, xb, plan, storage)
            if streams is not None:
                streams.append(x[:, :self.arch.hidden_size].clone())
        return x


class VasolixRandomWeights(RandomWeights):
    def shape(self, name: str):
        a = self.arch
        if name in ("embed", "head"):
            return (a.vocab_size, a.hidden_size)
        if name == "final.norm" or name.split(".", 1)[-1] in ("norm1", "norm2"):
            return (a.hidden_size,)
        layer, part, rest = name.split(".", 2)
        spec, W = a.layers[int(layer[1:])], a.hidden_size
        m = spec.mixer
        if part == "mix" and spec.type == "attention":
            nq, nk = m.heads * m.dim, m.kv_heads * m.dim
            return {"q": (nq, W), "k": (nk, W), "g": (nq, W), "o": (W, nq), "q.norm": (nq,), "k.norm": (nk,), "sink": (m.heads,)}[rest]
        if part == "mix":
            nk, nv = m.heads * m.dim, m.heads * m.vdim
            return {"q": (nk, W), "k": (nk, W), "v": (nv, W), "g": (nv, W), "o": (W, nv), "norm": (m.vdim,), "a1": (m.rank, W),
                    "a2": (nk, m.rank), "a2.b": (nk,)}[rest]
        if rest == "router":
            return (spec.mlp.experts, W)
        if rest == "shared.sg":
            return (1, W)
        ff = spec.mlp.shared_ff if rest.startswith("shared.") else spec.mlp.ff
        return (ff, W) if rest.endswith(".up") else (W, ff)

    def value(self, name, t):
        if name.endswith("a2.b"):
            return t + 2.0
        return t if name.endswith("sink") else super().value(name, t)


VasolixLLM.random_weights = VasolixRandomWeights
