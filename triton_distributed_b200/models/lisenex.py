"""Lisenex: a decoder whose layers are listed one by one; every layer adds its mixer and its feed-forward to the stream at once.

Layer: ``x += mixer(RMSNorm(x) * norm1) + ff(RMSNorm(x) * norm2)``.  Mixer: latent attention with an output gate, with cached rows
of its own or those of an earlier layer (``parallel.TP_LatentAttn``).  Feed-forward: dense squared ReLU with biases, a mixture of
SiLU-gated experts behind a softmax router with choice correction, groups, identity experts and a shared expert
(``parallel.tp_routed_ff``), or none.  The head is the embedding table.  The residual stream is fp32.

The configuration is a ``config.json`` with ``"architecture": "Lisenex"``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and
``layers``, a list of ``{type, mixer, mlp}``.  Tensors are named ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.norm2``,
``l<i>.mlp.*``, ``final.norm``.  Activations are bf16 (with everything sensitive in fp32) or, with ``ModelConfig.dtype =
torch.float32``, fp32 throughout.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch

from .. import ops
from ..parallel.tp_latent_attn import TP_LatentAttn
from ..parallel.tp_layer import pad8, pad_rows
from ..parallel.tp_routed_ff import TP_DenseFF, TP_RoutedMoE
from .layered import LayeredConfig, LayeredLLM, RandomWeights, read_config


# ------------------------------------------------------------------ configuration
@dataclass(frozen=True)
class LatentAttnSpec:
    heads: int
    dim: int                     # unrotated query / key dimensions of a head
    rot_dim: int                 # rotated ones (the key's are shared by all heads)
    vdim: int
    kv_rank: int                 # size of the latent
    scale: float
    rot_base: float
    kv_from: Optional[int] = None    # layer whose cached rows are used in place of own ones

    @staticmethod
    def from_json(c: dict) -> "LatentAttnSpec":
        rot = c["rot"]
        if rot.get("dims", c["rot_dim"]) != c["rot_dim"] or c["rot_dim"] % 2:
            raise ValueError("latent attention: the rotation covers the whole rotated part, an even number of dimensions")
        return LatentAttnSpec(c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"], float(c["scale"]), float(rot["base"]),
                              c.get("kv_from"))


@dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclass(frozen=True)
class RoutedSpec:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0           # 0 = no shared expert
    identity: int = 0            # router outputs beyond the experts: identity experts
    groups: int = 0              # equal groups of neighbours over experts and identity experts (0 = none), ...
    keep: int = 0                # ... of which this many can be chosen from

    def __post_init__(self):
        n = self.experts + self.identity
        if self.groups and (n % self.groups or not 1 <= self.keep <= self.groups):
            raise ValueError(f"{n} router outputs cannot form {self.groups} groups of which {self.keep} are kept")
        if not 1 <= self.top <= (n // self.groups * self.keep if self.groups else n):
            raise ValueError(f"{self.top} experts per token cannot be chosen")


def ff_from_json(c: Optional[dict]) -> Union[None, DenseSpec, RoutedSpec]:
    if c is None:
        return None
    if c["kind"] == "dense":
        return DenseSpec(c["ff"])
    if c["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {c['kind']!r}")
    r, shared, groups = c["router"], c.get("shared"), c["router"].get("groups")
    return RoutedSpec(r["experts"], r["top"], c["expert"]["ff"], shared["ff"] if shared else 0, r.get("identity") or 0,
                      groups["count"] if groups else 0, groups["keep"] if groups else 0)


MIXERS = {"latent_attention": (LatentAttnSpec, TP_LatentAttn)}
FEED_FORWARDS = {DenseSpec: TP_DenseFF, RoutedSpec: TP_RoutedMoE}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: LatentAttnSpec
    mlp: Union[None, DenseSpec, RoutedSpec]

    @staticmethod
    def from_json(c: dict) -> "LayerSpec":
        if c["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {c['type']!r}; known: {sorted(MIXERS)}")
        return LayerSpec(c["type"], MIXERS[c["type"]][0].from_json(c["mixer"]), ff_from_json(c.get("mlp")))


@dataclass(frozen=True)
class LisenexConfig(LayeredConfig):
    name: str
    vocab_size: int
    hidden_size: int
    rms_norm_eps: float
    embedding_scale: float
    layers: Tuple[LayerSpec, ...]

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            m = l.mixer
            if m.kv_from is None:
                continue
            if not 0 <= m.kv_from < i or self.layers[m.kv_from].mixer.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from must name an earlier layer with rows of its own")
            o = self.layers[m.kv_from].mixer
            if (o.kv_rank, o.rot_dim, o.rot_base) != (m.kv_rank, m.rot_dim, m.rot_base):
                raise ValueError(f"layer {i}: rank and rotation differ from those of layer {m.kv_from}")

    @property
    def is_moe(self) -> bool:
        return any(isinstance(l.mlp, RoutedSpec) for l in self.layers)

    def with_num_layers(self, n: int) -> "LisenexConfig":
        """The first ``n`` layers; when the list is shorter it is repeated, every repetition sharing rows inside itself."""
        L = len(self.layers)

        def moved(i):
            l = self.layers[i % L]
            if l.mixer.kv_from is None:
                return l
            return dataclasses.replace(l, mixer=dataclasses.replace(l.mixer, kv_from=l.mixer.kv_from + i // L * L))

        return dataclasses.replace(self, layers=tuple(moved(i) for i in range(n)))

    @staticmethod
    def from_json(path: str) -> "LisenexConfig":
        c = read_config(path)
        return LisenexConfig(c["architecture"], c["vocab"], c["width"], float(c["norm"]["eps"]), float(c["embedding"]["scale"]),
                             tuple(LayerSpec.from_json(l) for l in c["layers"]))


def latent_stack(name: str, vocab: int, width: int, pattern: str, attn: LatentAttnSpec, dense: Optional[DenseSpec],
                 moe: Optional[RoutedSpec], eps: float = 1e-5, scale: float = 1.0) -> LisenexConfig:
    """A configuration from a pattern string, one letter per layer: "D" dense, "M" mixture of experts, "N" no feed-forward; lower
    case: the layer uses the rows of the last upper-case one."""
    layers, own = [], None
    for i, k in enumerate(pattern):
        own = i if k.isupper() else own
        layers.append(LayerSpec("latent_attention", dataclasses.replace(attn, kv_from=None if k.isupper() else own),
                                {"D": dense, "M": moe, "N": None}[k.upper()]))
    return LisenexConfig(name, vocab, width, eps, scale, tuple(layers))


LISENEX_PRESETS = {
    # layers of the size of Qwen3-30B-A3B's (width, heads, experts), latent rows as in large latent-attention models
    "lisenex-30b-a3b": latent_stack("lisenex-30b-a3b", 151936, 2048, "D" + "mM" * 23 + "m",
                                    LatentAttnSpec(32, 128, 64, 128, 512, 192 ** -0.5, 1e6), DenseSpec(6144),
                                    RoutedSpec(120, 8, 768, 768, 8, 8, 4)),
    "lisenex-1b": latent_stack("lisenex-1b", 65536, 1536, "D" + "mM" * 11 + "m",
                               LatentAttnSpec(24, 64, 32, 64, 256, 96 ** -0.5, 1e5), DenseSpec(4096), RoutedSpec(28, 4, 512, 512, 4, 4, 2)),
    "tiny-lisenex": latent_stack("tiny-lisenex", 1000, 192, "DmMn", LatentAttnSpec(6, 40, 24, 48, 72, 0.13, 1e4), DenseSpec(232),
                                 RoutedSpec(7, 2, 80, 112, 2, 3, 2), scale=0.7),
}


# ------------------------------------------------------------------ model
class LisenexLayer:
    def __init__(self, index: int, spec: LayerSpec, rank: int, world_size: int, group):
        self.index, self.spec = index, spec
        self.rank, self.world_size = rank, world_size
        self.mixer = MIXERS[spec.type][1](spec.mixer, index, rank, world_size, group)
        self.mlp = FEED_FORWARDS[type(spec.mlp)](spec.mlp, rank, world_size, group) if spec.mlp is not None else None
        self.norm1 = self.norm2 = None

    def parts(self):
        return [self.mixer] + ([self.mlp] if self.mlp is not None else [])

    def load(self, get, width: int, eps: float, dtype, device):
        p = f"l{self.index}."
        w8 = pad8(width)
        self.norm1 = pad_rows(get(p + "norm1").float(), w8).to(device)
        self.mixer.load(get, p + "mix.", width, eps, dtype, device)
        if self.mlp is not None:
            self.norm2 = pad_rows(get(p + "norm2").float(), w8).to(device)
            self.mlp.load(get, p + "mlp.", width, dtype, device)

    def sublayers(self, h1, h2, plan, storage, side=None):
        """(mixer output, feed-forward pieces or None): what this rank's part of the layer adds to the stream.  Neither reads the
        other: with ``side`` (a stream) the feed-forward runs beside the mixer."""
        if self.mlp is None or side is None:
            return self.mixer(h1, plan, storage), (self.mlp(h2) if self.mlp is not None else None)
        # Tensors of either stream's pool are only reused by that stream, which has waited for the other by then: both wait for
        # each other once a layer.
        main = torch.cuda.current_stream()
        side.wait_stream(main)
        with torch.cuda.stream(side), ops.scratch_lane(1):
            ff = self.mlp(h2)
        mix = self.mixer(h1, plan, storage)
        main.wait_stream(side)
        return mix, ff


class LisenexLLM(LayeredLLM):
    """See :class:`LayeredLLM`.  On several ranks a layer costs one all-reduce: the partial sums of mixer and feed-forward travel
    together, in fp32."""

    _side = None

    def make_layers(self):
        layers = [LisenexLayer(i, s, self.rank, self.world_size, self.group) for i, s in enumerate(self.arch.layers)]
        for l in layers:
            if not l.mixer.own_kv:
                layers[l.mixer.source].mixer.shared = True
        return layers

    def side_stream(self):
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.device)
        return self._side

    def load_head(self, get):
        self.embed_tokens = self.lm_head = self.table(get, "embed")

    def hidden(self, ids, plan, streams):
        a = self.arch
        x, _ = ops.embed_stream(ids, self.embed_tokens, a.embedding_scale, copy=False)

        def add(mix, ff, nxt):
            """Adds to the stream and norms it for layer ``nxt`` (None: the last one has run)."""
            w = (None, None) if nxt is None else (nxt.norm1, nxt.norm2)
            return ops.parallel_add(x, mix, ff, *w, a.hidden_size, a.rms_norm_eps, self.dtype)

        # decode steps are bound by latency and weight streaming: mixer and feed-forward overlap
        side = self.side_stream() if plan.decode and x.is_cuda else None
        h1, h2 = add(None, None, self.layers[0])
        for i, l in enumerate(self.layers):
            mix, ff = l.sublayers(h1, h2, plan, plan.cache.layers[i], side)
            if self.world_size > 1:
                mix, ff = None, ops.FeedForward(l.mixer.reduce(ops.parallel_sum(x, mix, ff)))
            h1, h2 = add(mix, ff, self.layers[i + 1] if i + 1 < len(self.layers) else None)
            if streams is not None:
                streams.append(x[:, :a.hidden_size].clone())
        return x


class LisenexRandomWeights(RandomWeights):
    def shape(self, name: str):
        a = self.arch
        if name == "embed":
            return (a.vocab_size, a.hidden_size)
        if name == "final.norm" or name.split(".", 1)[-1] in ("norm1", "norm2"):
            return (a.hidden_size,)
        layer, part, rest = name.split(".", 2)
        spec, W = a.layers[int(layer[1:])], a.hidden_size
        if part == "mix":
            m = spec.mixer
            nv = m.heads * m.vdim
            return {"q": (m.heads * (m.dim + m.rot_dim), W), "dkv": (m.kv_rank + m.rot_dim, W), "dkv.norm": (m.kv_rank,),
                    "uk": (m.heads * m.dim, m.kv_rank), "uv": (nv, m.kv_rank), "g": (nv, W), "o": (W, nv)}[rest]
        f = spec.mlp
        if isinstance(f, DenseSpec):
            return {"up": (f.ff, W), "up.b": (f.ff,), "down": (W, f.ff), "down.b": (W,)}[rest]
        if rest in ("router", "correction"):
            return (f.experts + f.identity, W) if rest == "router" else (f.experts + f.identity,)
        ff = f.shared_ff if rest.startswith("shared.") else f.ff
        return (W, ff) if rest.endswith(".down") else (ff, W)

    def value(self, name, t):
        if name.endswith((".b", "correction")):
            return 0.02 * t
        return super().value(name, t)


LisenexLLM.random_weights = LisenexRandomWeights
