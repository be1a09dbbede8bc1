"""Bagasun: a decoder whose layers are listed one by one, each sublayer between two norms; a layer may use the weights of an earlier one.

Mixers: attention over a sliding window with independent sigmoid weights and a distance term (``parallel.TP_SigmoidAttn``), differential
attention over a sliding window with rotary positions (``parallel.TP_DifferentialAttn``), and a state space layer with short convolutions
(``parallel.TP_StateSpace``).  Feed-forward: dense gated GELU (``parallel.TP_GatedFF``), or none.  Norms have one number for all
coordinates; one pass over the fp32 stream between two sublayers adds the normed output of the last and norms the input of the next
(``ops.sandwich_step``).  Layers that share weights share the tensors on the device as well, and have caches of their own.

The configuration is a ``config.json`` with ``"architecture": "Bagasun"``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and
``layers``, a list of ``{type, mixer, mlp, weights_of}``.  Tensors are named ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.mix.*``,
``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mlp.*``, ``final.norm``, ``head``.  Activations are bf16 (with everything sensitive in fp32) or,
with ``ModelConfig.dtype = torch.float32``, fp32 throughout.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch

from .. import ops
from ..parallel.tp_routed_ff import TP_GatedFF
from ..parallel.tp_ssd import TP_StateSpace
from ..parallel.tp_window_attn import TP_DifferentialAttn, TP_SigmoidAttn
from .layered import LayeredConfig, LayeredLLM, RandomWeights, read_config


# ------------------------------------------------------------------ configuration
def _window(c: dict) -> int:
    size = (c.get("mask") or {}).get("size")
    if size is not None and int(size) < 1:
        raise ValueError("attention: a window holds at least the position itself")
    return int(size or 0)


def _check_heads(s):
    if s.heads % s.kv_heads:
        raise ValueError("attention: heads must be a multiple of kv_heads")


@dataclass(frozen=True)
class SigmoidAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0              # 0 = every earlier position

    def __post_init__(self):
        _check_heads(self)

    @staticmethod
    def from_json(c: dict) -> "SigmoidAttnSpec":
        return SigmoidAttnSpec(c["heads"], c["kv_heads"], c["dim"], c["vdim"], float(c["scale"]), _window(c))


@dataclass(frozen=True)
class DifferentialAttnSpec:
    heads: int
    kv_heads: int
    dim: int                     # of a map
    vdim: int
    scale: float
    diff: float
    rot_base: float
    rot_dims: int                # leading elements of a map that turn
    scaling: Optional[ops.BandScaling] = None
    window: int = 0

    def __post_init__(self):
        _check_heads(self)
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            raise ValueError("attention: the rotation covers an even number of a map's dimensions")

    @staticmethod
    def from_json(c: dict) -> "DifferentialAttnSpec":
        rot = c["rot"]
        return DifferentialAttnSpec(c["heads"], c["kv_heads"], c["dim"], c["vdim"], float(c["scale"]), float(c["diff"]), float(rot["base"]),
                                    int(rot["dims"]), ops.BandScaling.from_json(rot.get("scaling")), _window(c))


@dataclass(frozen=True)
class StateSpaceSpec:
    heads: int
    groups: int                  # of B and C
    state: int
    vdim: int
    conv: int                    # taps of the short convolution
    norm_groups: int

    def __post_init__(self):
        if self.heads % self.groups or self.conv < 1 or (self.heads * self.vdim) % self.norm_groups:
            raise ValueError("state space layer: heads must be a multiple of groups, the inner width of norm_groups, convolutions have a tap")

    @staticmethod
    def from_json(c: dict) -> "StateSpaceSpec":
        return StateSpaceSpec(c["heads"], c["groups"], c["state"], c["vdim"], c["conv"], c["norm_groups"])


@dataclass(frozen=True)
class GatedFFSpec:
    ff: int


MIXERS = {"attention": (SigmoidAttnSpec, TP_SigmoidAttn), "attention_2": (DifferentialAttnSpec, TP_DifferentialAttn),
          "mamba2": (StateSpaceSpec, TP_StateSpace)}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Union[SigmoidAttnSpec, DifferentialAttnSpec, StateSpaceSpec]
    mlp: Optional[GatedFFSpec]
    weights_of: Optional[int] = None       # layer whose tensors this one uses

    @staticmethod
    def from_json(c: dict) -> "LayerSpec":
        if c["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {c['type']!r}; known: {sorted(MIXERS)}")
        f, of = c.get("mlp"), c.get("weights_of")
        if f is not None and f["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
        return LayerSpec(c["type"], MIXERS[c["type"]][0].from_json(c["mixer"]), None if f is None else GatedFFSpec(f["ff"]), None if of is None else int(of))


@dataclass(frozen=True)
class BagasunConfig(LayeredConfig):
    name: str
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    embed_scale: float
    layers: Tuple[LayerSpec, ...]
    is_moe = False

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            j = self.source(i)
            if dataclasses.replace(l, weights_of=None) != dataclasses.replace(self.layers[j], weights_of=None):
                raise ValueError(f"layer {i} cannot use the weights of layer {j}: their sizes differ")

    def source(self, i: int) -> int:
        """Layer whose tensors layer i uses."""
        seen = [i]
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError(f"weights_of {i} does not lead to a layer with tensors")
            seen.append(i)
        return i

    def with_num_layers(self, n: int) -> "BagasunConfig":
        """The first ``n`` layers (the list is repeated when it is shorter); a shared layer beyond them keeps weights of its own."""
        layers = [self.layers[i % len(self.layers)] for i in range(n)]
        return dataclasses.replace(self, layers=tuple(l if (l.weights_of or 0) < n else dataclasses.replace(l, weights_of=None) for l in layers))

    @staticmethod
    def from_json(path: str) -> "BagasunConfig":
        c = read_config(path)
        return BagasunConfig(c["architecture"], c["vocab"], c["width"], float(c["norm"]["eps"]), float(c["embedding"]["scale"]),
                             tuple(LayerSpec.from_json(l) for l in c["layers"]))


def sandwich_stack(name: str, vocab: int, width: int, pattern: str, attention: SigmoidAttnSpec, attention_2: DifferentialAttnSpec, mamba2: StateSpaceSpec,
                   ff: Optional[int], repeats: int = 1, embed_scale: float = 1.0, eps: float = 1e-5) -> BagasunConfig:
    """A configuration from a pattern string: "A" and "D" for sigmoid and differential attention, "M" for a state space layer; lower case:
    without a feed-forward.  The pattern runs ``repeats`` times with the same weights."""
    kinds = {"A": ("attention", attention), "D": ("attention_2", attention_2), "M": ("mamba2", mamba2)}
    layers = tuple(LayerSpec(*kinds[k.upper()], GatedFFSpec(ff) if k.isupper() else None, i if r else None)
                   for r in range(repeats) for i, k in enumerate(pattern))
    return BagasunConfig(name, vocab, width, eps, embed_scale, layers)


BAGASUN_PRESETS = {
    # layers of the size of Qwen3-8B's (width, heads, feed-forward)
    "bagasun-8b": sandwich_stack("bagasun-8b", 151936, 4096, "MDMA" * 9, SigmoidAttnSpec(32, 8, 128, 128, 128 ** -0.5, 4096),
                                 DifferentialAttnSpec(32, 8, 64, 128, 0.125, 0.8, 1e6, 64, ops.BandScaling(4.0, 8192, 1.0, 4.0), 4096),
                                 StateSpaceSpec(128, 8, 128, 64, 4, 8), 12288),
    "bagasun-1b": sandwich_stack("bagasun-1b", 65536, 1536, "MDMA" * 3, SigmoidAttnSpec(24, 4, 64, 64, 0.125, 1024),
                                 DifferentialAttnSpec(12, 4, 64, 128, 0.125, 0.5, 1e5, 32, ops.BandScaling(8.0, 4096, 1.0, 4.0), 1024),
                                 StateSpaceSpec(48, 1, 128, 64, 4, 1), 4096, repeats=2, embed_scale=8.0),
    "tiny-bagasun": sandwich_stack("tiny-bagasun", 1000, 192, "MDaA", SigmoidAttnSpec(6, 2, 40, 24, 0.2, 20),
                                   DifferentialAttnSpec(4, 2, 24, 56, 0.2, 0.4, 1e4, 12, ops.BandScaling(2.0, 64, 1.0, 3.0), 24),
                                   StateSpaceSpec(6, 2, 24, 40, 3, 3), 232, repeats=2, embed_scale=3.0),
}


# ------------------------------------------------------------------ model
class BagasunLayer:
    """``source``: the layer whose tensors this one uses, itself or another one that has been built."""

    def __init__(self, index: int, spec: LayerSpec, source: Optional["BagasunLayer"], rank: int, world_size: int, group):
        self.index, self.spec, self.source = index, spec, source
        if source is not None:
            self.mixer, self.mlp = source.mixer, source.mlp
            return
        tp = (rank, world_size, group)
        self.mixer = MIXERS[spec.type][1](spec.mixer, *tp)
        self.mlp = TP_GatedFF(spec.mlp, "gelu", *tp) if spec.mlp is not None else None

    def parts(self):
        return [self.mixer] + ([self.mlp] if self.mlp is not None else [])

    def load(self, get, width: int, eps: float, dtype, device):
        if self.source is not None:
            return
        p = f"l{self.index}."

        def norms(q):
            return tuple(get(f"{p}norm{q}{e}").float().reshape(1).to(device) for e in ("", "b"))

        self.norm1 = norms(1)                   # before the mixer, behind it
        self.mixer.load(get, p + "mix.", width, eps, dtype, device)
        if self.mlp is not None:
            self.norm2 = norms(2)
            self.mlp.load(get, p + "mlp.", width, dtype, device)

    @property
    def weights(self) -> "BagasunLayer":
        return self if self.source is None else self.source


class BagasunLLM(LayeredLLM):
    """See :class:`LayeredLLM`.  A sublayer's output waits until the next pass over the stream, which norms and adds it."""

    def make_layers(self):
        layers = {}

        def layer(i):
            if i not in layers:
                j = self.arch.source(i)
                layers[i] = BagasunLayer(i, self.arch.layers[i], None if j == i else layer(j), self.rank, self.world_size, self.group)
            return layers[i]

        return [layer(i) for i in range(len(self.arch.layers))]

    def load_head(self, get):
        self.embed_tokens, self.lm_head = self.table(get, "embed"), self.table(get, "head")

    def final_norm(self, get):
        return get("final.norm").float().reshape(1).to(self.device)

    def _step(self, x, last, pre, rows=None, start=None):
        a = self.arch
        return ops.sandwich_step(x, last, pre, a.hidden_size, a.rms_norm_eps, self.dtype, rows, start)

    def hidden(self, ids, plan, streams):
        x = torch.empty(ids.numel(), self.embed_tokens.shape[1], dtype=torch.float32, device=ids.device)
        last, start = None, (ids.reshape(-1), self.embed_tokens, self.arch.embed_scale)
        for l, storage in zip(self.layers, plan.cache.layers):
            w = l.weights
            h = self._step(x, last, w.norm1[0], start=start)
            last, start = (l.mixer(h, plan, storage), w.norm1[1]), None
            if l.mlp is not None:
                h = self._step(x, last, w.norm2[0])
                last = (l.mlp(h).y, w.norm2[1])
            if streams is not None:
                self._step(x, last, None)
                last = None
                streams.append(x[:, :self.arch.hidden_size].clone())
        return x, last

    def final_hidden(self, x, rows):
        return self._step(*x, self.final_norm_w, rows)


class BagasunRandomWeights(RandomWeights):
    def shape(self, name: str):
        a = self.arch
        W = a.hidden_size
        if name in ("embed", "head"):
            return (a.vocab_size, W)
        layer, part, *rest = name.split(".", 2)
        if layer == "final" or part.startswith("norm"):
            return (1,)
        spec = a.layers[int(layer[1:])]
        m, rest = spec.mixer, rest[0]
        if part == "mlp":
            return (W, spec.mlp.ff) if rest == "down" else (spec.mlp.ff, W)
        if spec.type == "mamba2":
            inner, shared = m.heads * m.vdim, 2 * m.groups * m.state
            return {"in": (2 * inner + shared + m.heads, W), "conv": (inner + shared, m.conv), "conv.b": (inner + shared,), "norm": (inner,),
                    "o": (W, inner)}.get(rest, (m.heads,))
        maps = 2 if spec.type == "attention_2" else 1
        rows = {"q": m.heads * maps * m.dim, "k": m.kv_heads * maps * m.dim, "v": m.kv_heads * m.vdim, "g": m.heads}
        if rest == "o":
            return (W, m.heads * m.vdim)
        if rest in rows:
            return (rows[rest], W)
        if rest.endswith((".b", ".norm")):
            return (rows[rest[0]],)
        return (m.dim,) if rest[0] == "l" else (m.heads,)

    def value(self, name, t):
        rest = name.rsplit(".", 1)[-1]
        if "norm" in rest:
            return 1.0 + 0.1 * t
        if name.endswith((".b", ".lq1", ".lq2", ".lk1", ".lk2")):
            return 0.1 * t
        if rest in ("r1", "r2"):
            return 0.5 * t.abs()
        if rest in ("dt_bias", "pb"):
            return t - 2.0
        return t if rest in ("A_log", "D") else super().value(name, t)


BagasunLLM.random_weights = BagasunRandomWeights
