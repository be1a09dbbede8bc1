"""Tazitar: a decoder with several residual streams whose layers are listed one by one; a range of layers may run more than once.

Hyper-connections join a sublayer to the streams: its input is a mixture of them, its output goes to all of them
(``ops.hyper_step``, one pass over the fp32 streams between two sublayers).  Mixers: causal attention with rotary positions in three
forms (``parallel.TP_RotaryAttn``; two are layer types, one is a branch), and a layer of two branches, attention and a gated delta rule
(``parallel.TP_DeltaRule``), each normed before half their sum is taken (``parallel.TP_TwinMixer``).  Feed-forward: dense gated GELU
(``parallel.TP_GatedFF``), or none.  A looped layer runs with the same weights and a cache of its own in every pass.

The configuration is a ``config.json`` with ``"architecture": "Tazitar"``: ``vocab``, ``width``, ``norm.eps``, ``streams``, ``loop``
(``start``, ``stop``, ``times``) and ``layers``, a list of ``{type, mixer, mlp}``.  Tensors are named ``embed``, ``l<i>.norm1``,
``l<i>.hc1.*``, ``l<i>.mix.*``, ``l<i>.norm2``, ``l<i>.hc2.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.  Activations are bf16 (with
everything sensitive in fp32) or, with ``ModelConfig.dtype = torch.float32``, fp32 throughout.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch

from .. import ops
from ..parallel.tp_delta import TP_DeltaRule
from ..parallel.tp_layer import pad8, pad_rows
from ..parallel.tp_rotary_attn import TP_RotaryAttn
from ..parallel.tp_routed_ff import TP_GatedFF
from ..parallel.tp_twin import TP_TwinMixer
from .layered import LayeredConfig, LayeredLLM, RandomWeights, read_config

MAX_STREAMS = 16


# ------------------------------------------------------------------ configuration
@dataclass(frozen=True)
class RotaryAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int                # leading elements of a head that turn
    scaling: Optional[ops.YarnScaling] = None
    softcap: float = 0.0         # 0 = none
    # what the kind of attention fixes
    qk_norm: bool = False        # per-head norms with a weight before the rotation
    unit: bool = False           # weightless ones after it
    interleaved: bool = False    # neighbours turn together, else element i and i + rot_dims / 2
    sink: Union[None, float, str] = None     # one more score in the denominator: a number, or "learned" per head

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("attention: heads must be a multiple of kv_heads")
        if self.rot_dims % 2 or not 0 < self.rot_dims <= self.dim:
            raise ValueError("attention: the rotation covers an even number of a head's dimensions")

    @staticmethod
    def from_json(c: dict, **kind) -> "RotaryAttnSpec":
        rot = c["rot"]
        return RotaryAttnSpec(c["heads"], c["kv_heads"], c["dim"], c["vdim"], float(c["scale"]), float(rot["base"]), int(rot["dims"]),
                              ops.YarnScaling.from_json(rot.get("scaling")), float(c.get("softcap") or 0.0), **kind)


@dataclass(frozen=True)
class DeltaRuleSpec:
    heads: int
    kv_heads: int                # of q and k
    dim: int
    vdim: int
    conv: int                    # taps of the short convolutions

    def __post_init__(self):
        if self.heads % self.kv_heads or self.conv < 1:
            raise ValueError("delta rule: heads must be a multiple of kv_heads, convolutions have at least one tap")

    @staticmethod
    def from_json(c: dict) -> "DeltaRuleSpec":
        return DeltaRuleSpec(c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["conv"])


@dataclass(frozen=True)
class TwinSpec:
    left: RotaryAttnSpec
    right: DeltaRuleSpec


@dataclass(frozen=True)
class GatedFFSpec:
    ff: int


KINDS = {"attention": dict(qk_norm=True), "left": dict(unit=True, sink=0.0), "attention_2": dict(unit=True, interleaved=True, sink="learned")}


def mixer_from_json(kind: str, c: dict) -> Union[RotaryAttnSpec, TwinSpec]:
    if kind == "parallel":
        return TwinSpec(RotaryAttnSpec.from_json(c["left"], **KINDS["left"]), DeltaRuleSpec.from_json(c["right"]))
    if kind not in ("attention", "attention_2"):
        raise ValueError(f"unknown mixer {kind!r}; known: attention, attention_2, parallel")
    return RotaryAttnSpec.from_json(c, **KINDS[kind])


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: Union[RotaryAttnSpec, TwinSpec]
    mlp: Optional[GatedFFSpec]

    @staticmethod
    def from_json(c: dict) -> "LayerSpec":
        f = c.get("mlp")
        if f is not None and f["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {f['kind']!r}")
        return LayerSpec(c["type"], mixer_from_json(c["type"], c["mixer"]), None if f is None else GatedFFSpec(f["ff"]))


@dataclass(frozen=True)
class TazitarConfig(LayeredConfig):
    name: str
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    streams: int
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    is_moe = False

    def __post_init__(self):
        if not 1 <= self.streams <= MAX_STREAMS:
            raise ValueError(f"{self.streams} residual streams (1 to {MAX_STREAMS})")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")

    @property
    def passes(self) -> Tuple[int, ...]:
        """Layer numbers in the order in which they run."""
        n = len(self.layers)
        start, stop, times = self.loop or (0, 0, 1)
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, n))

    def with_num_layers(self, n: int) -> "TazitarConfig":
        """The first ``n`` layers (the list is repeated when it is shorter); the loop ends with them."""
        loop = self.loop
        if loop is not None:
            loop = (loop[0], min(loop[1], n), loop[2]) if loop[0] < n else None
        return dataclasses.replace(self, loop=loop, layers=tuple(self.layers[i % len(self.layers)] for i in range(n)))

    @staticmethod
    def from_json(path: str) -> "TazitarConfig":
        c = read_config(path)
        loop = c.get("loop")
        return TazitarConfig(c["architecture"], c["vocab"], c["width"], float(c["norm"]["eps"]), c["streams"],
                             tuple(LayerSpec.from_json(l) for l in c["layers"]), (loop["start"], loop["stop"], loop["times"]) if loop else None)


def stream_stack(name: str, vocab: int, width: int, pattern: str, attention: RotaryAttnSpec, twin: TwinSpec, attention_2: RotaryAttnSpec,
                 ff: Optional[int], streams: int = 4, loop=None, eps: float = 1e-5) -> TazitarConfig:
    """A configuration from a pattern string: "A" and "B" for the two attention layers, "P" for a layer of two branches; lower case:
    without a feed-forward."""
    kinds = {"A": ("attention", attention), "B": ("attention_2", attention_2), "P": ("parallel", twin)}
    layers = tuple(LayerSpec(*kinds[k.upper()], GatedFFSpec(ff) if k.isupper() else None) for k in pattern)
    return TazitarConfig(name, vocab, width, eps, streams, layers, loop)


def _sizes(heads, kv_heads, dim, vdim, rot, base, scaling, cap, delta_heads, delta_kv, dk, dv, taps):
    scale = dim ** -0.5
    return (RotaryAttnSpec(heads, kv_heads, dim, vdim, scale, base, dim, None, cap, **KINDS["attention"]),
            TwinSpec(RotaryAttnSpec(heads, kv_heads, dim, vdim, scale, base, rot, **KINDS["left"]), DeltaRuleSpec(delta_heads, delta_kv, dk, dv, taps)),
            RotaryAttnSpec(heads, kv_heads, dim, vdim, scale, base, dim, scaling, **KINDS["attention_2"]))


TAZITAR_PRESETS = {
    # layers of the size of Qwen3-8B's (width, heads, feed-forward)
    "tazitar-8b": stream_stack("tazitar-8b", 151936, 4096, "APPB" * 9, *_sizes(32, 8, 128, 128, 32, 1e6, ops.YarnScaling(4.0, 8192, 32.0, 1.0), 50.0,
                                                                              32, 16, 128, 128, 4), 12288),
    "tazitar-1b": stream_stack("tazitar-1b", 65536, 1536, "APPB" * 6, *_sizes(24, 4, 64, 64, 16, 1e5, ops.YarnScaling(8.0, 4096, 32.0, 1.0), 30.0,
                                                                             12, 6, 64, 128, 4), 4096, loop=(4, 20, 2)),
    "tiny-tazitar": stream_stack("tiny-tazitar", 1000, 192, "APbA", *_sizes(6, 2, 40, 56, 24, 1e4, ops.YarnScaling(4.0, 64, 8.0, 1.0), 20.0,
                                                                           4, 2, 24, 40, 4), 232, 3, (1, 3, 2)),
}


# ------------------------------------------------------------------ model
class TazitarLayer:
    def __init__(self, index: int, spec: LayerSpec, rank: int, world_size: int, group):
        self.index, self.spec = index, spec
        tp = (rank, world_size, group)
        m = spec.mixer
        self.mixer = TP_TwinMixer(TP_RotaryAttn(m.left, *tp), TP_DeltaRule(m.right, *tp), *tp) if isinstance(m, TwinSpec) else TP_RotaryAttn(m, *tp)
        self.mlp = TP_GatedFF(spec.mlp, "gelu", *tp) if spec.mlp is not None else None

    def parts(self):
        twin = [self.mixer.left, self.mixer.right] if isinstance(self.mixer, TP_TwinMixer) else []
        return [self.mixer] + twin + ([self.mlp] if self.mlp is not None else [])

    def load(self, get, width: int, eps: float, dtype, device):
        p = f"l{self.index}."

        def sublayer(q):
            hc = ops.HyperWeights(*(get(f"{p}hc{q}.{n}").float().to(device).contiguous() for n in ("in", "out", "mix")))
            return pad_rows(get(f"{p}norm{q}").float(), pad8(width)).to(device), hc

        self.norm1, self.hc1 = sublayer(1)
        self.mixer.load(get, p + "mix.", width, eps, dtype, device)
        if self.mlp is not None:
            self.norm2, self.hc2 = sublayer(2)
            self.mlp.load(get, p + "mlp.", width, dtype, device)


class TazitarLLM(LayeredLLM):
    """See :class:`LayeredLLM`.  A sublayer's output waits until the next pass over the streams, which adds it."""

    def make_layers(self):
        return [TazitarLayer(i, s, self.rank, self.world_size, self.group) for i, s in enumerate(self.arch.layers)]

    def cache_specs(self):
        return [self.layers[i].mixer.cache_spec() for i in self.arch.passes]

    def load_head(self, get):
        self.embed_tokens, self.lm_head = self.table(get, "embed"), self.table(get, "head")
        self.sum_weights = torch.ones(self.arch.streams, device=self.device)

    def _step(self, x, last, nxt, rows=None, start=None):
        a = self.arch
        return ops.hyper_step(x, last, nxt, a.hidden_size, a.rms_norm_eps, self.dtype, rows, start)

    def hidden(self, ids, plan, streams):
        x = torch.empty(ids.numel(), self.arch.streams, self.embed_tokens.shape[1], dtype=torch.float32, device=ids.device)
        last, start = None, (ids.reshape(-1), self.embed_tokens)
        for run, i in enumerate(self.arch.passes):
            l = self.layers[i]
            h = self._step(x, last, (l.hc1.inp, l.norm1), start=start)
            last, start = (l.hc1, l.mixer(h, plan, plan.cache.layers[run])), None
            if l.mlp is not None:
                h = self._step(x, last, (l.hc2.inp, l.norm2))
                last = (l.hc2, l.mlp(h))
            if streams is not None:
                self._step(x, last, None)
                last = None
                streams.append(x.sum(1)[:, :self.arch.hidden_size])
        return x, last

    def final_hidden(self, x, rows):
        return self._step(*x, (self.sum_weights, self.final_norm_w), rows)


class TazitarRandomWeights(RandomWeights):
    def attention(self, m: RotaryAttnSpec, rest: str):
        W = self.arch.hidden_size
        return {"q": (m.heads * m.dim, W), "k": (m.kv_heads * m.dim, W), "v": (m.kv_heads * m.vdim, W), "o": (W, m.heads * m.vdim),
                "q.norm": (m.dim,), "k.norm": (m.dim,), "sink": (m.heads,)}[rest]

    def delta(self, m: DeltaRuleSpec, rest: str):
        W, nk, nv = self.arch.hidden_size, m.kv_heads * m.dim, m.heads * m.vdim
        return {"q": (nk, W), "k": (nk, W), "v": (nv, W), "g": (nv, W), "o": (W, nv), "a": (m.heads, W), "b": (m.heads, W), "A_log": (m.heads,),
                "dt_bias": (m.heads,), "norm": (m.vdim,), "q.conv": (nk, m.conv), "k.conv": (nk, m.conv), "v.conv": (nv, m.conv)}[rest]

    def shape(self, name: str):
        a = self.arch
        W, S = a.hidden_size, a.streams
        if name in ("embed", "head"):
            return (a.vocab_size, W)
        if name == "final.norm":
            return (W,)
        layer, part, *rest = name.split(".", 2)
        spec = a.layers[int(layer[1:])]
        if part.startswith("norm"):
            return (W,)
        if part.startswith("hc"):
            return (S, S) if rest[0] == "mix" else (S,)
        if part == "mlp":
            return (W, spec.mlp.ff) if rest[0] == "down" else (spec.mlp.ff, W)
        if not isinstance(spec.mixer, TwinSpec):
            return self.attention(spec.mixer, rest[0])
        side, rest = rest[0].split(".", 1)
        if rest == "out":
            return (W,)
        return self.attention(spec.mixer.left, rest) if side == "left" else self.delta(spec.mixer.right, rest)

    def value(self, name, t):
        S = self.arch.streams
        if ".hc" in name:
            base = torch.eye(S, device=t.device) if name.endswith("mix") else 1.0 / S if name.endswith("in") else 1.0
            return base + 0.1 / S * t
        if name.endswith((".left.out", ".right.out")):
            return 1.0 + 0.1 * t
        if name.endswith(("sink", "A_log")):
            return t
        return t - 2.0 if name.endswith("dt_bias") else super().value(name, t)


TazitarLLM.random_weights = TazitarRandomWeights
