"""Small random Tazitar models for the tests, as (config, weights) in the checkpoint format; the helpers around a model are those
of ``vasolix_cases``."""
import torch

import tazitar_oracle as oracle
from vasolix_cases import engine, prompt, rel, run_portions, write  # noqa: F401


def rot(dims, base=500.0, **scaling):
    return {"base": base, "dims": dims, **({"scaling": scaling} if scaling else {})}


def attn(heads=4, kv_heads=2, dim=16, vdim=24, rot_dims=12, scale=None, cap=None, base=500.0, **scaling):
    """``scaling``: factor, original, fast, slow."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot(rot_dims, base, **scaling),
         "scale": scale if scale is not None else 1.7 * dim ** -0.5}
    if cap:
        m["softcap"] = cap
    return m


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=4):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def config(layers, width=64, vocab=101, eps=1e-5, streams=3, loop=None):
    """``layers``: list of (type, mixer, ff or None); ``loop``: (start, stop, times)."""
    c = {"architecture": "Tazitar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
         "layers": [{"type": t, "mixer": m, "mlp": None if f is None else {"kind": "dense", "ff": f}} for t, m, f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


YARN = dict(factor=4.0, original=48, fast=6.0, slow=0.8)
# every branch, and sizes that are no multiples of anything in particular: partial rotations, head groups of different sizes, one KV
# head for all, no feed-forward, convolutions of several lengths, a loop over a part of the layers
MIXED = config([("attention", attn(6, 3, 20, 28, 14, cap=3.0), 50),
                ("parallel", {"left": attn(4, 2, 18, 26, 10, scale=0.4), "right": delta(4, 2, 12, 20, 4)}, 42),
                ("attention_2", attn(5, 1, 16, 10, 12, scale=0.35, base=60.0, **YARN), None),
                ("parallel", {"left": attn(3, 3, 12, 12, 12, scale=0.5), "right": delta(6, 2, 20, 10, 2)}, None),
                ("attention", attn(2, 1, 8, 8, 8, cap=1.5), 24)], width=60, vocab=101, eps=2e-3, streams=3, loop=(1, 4, 2))
PLAIN = config([("parallel", {"left": attn(), "right": delta(conv=3)}, 40), ("attention", attn(cap=6.0), 56),
                ("attention_2", attn(factor=2.0, original=32, fast=4.0, slow=1.0), 32)], width=64, vocab=96, eps=1e-3, streams=2)


def weights(cfg, seed=0, dtype=torch.bfloat16, sharp=2.0, uneven=1.0, gain=1.0):
    """Random weights.  Queries and keys give scores of which single ones win the softmax, sinks and soft caps are of the scores' size,
    decays reach from almost 1 to strong, norm weights differ from 1 and the streams are mixed unevenly (``uneven``: by how
    much; ``gain``: how much a sublayer adds).  Strongly mixed streams and large gains let a looped model amplify rounding."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5)

    def attention(p, m, kind):
        H, G, d, dv = (m[n] for n in ("heads", "kv_heads", "dim", "vdim"))
        t.update({p + "q": r(H * d, W), p + "k": r(G * d, W), p + "v": r(G * dv, W), p + "o": r(W, H * dv)})
        if kind == "attention":
            t.update({p + "q.norm": sharp * (1 + r(d, std=0.3)), p + "k.norm": 1 + r(d, std=0.3)})
        if kind == "attention_2":
            t[p + "sink"] = 2.0 + r(H, std=1.5)

    def delta_rule(p, m):
        H, nk, nv = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
        t.update({p + "q": r(nk, W), p + "k": r(nk, W), p + "v": r(nv, W), p + "g": r(nv, W, std=2 * W ** -0.5), p + "o": r(W, nv)})
        t.update({p + n + ".conv": r(c, m["conv"], std=1.5 * m["conv"] ** -0.5) for n, c in (("q", nk), ("k", nk), ("v", nv))})
        t.update({p + "a": r(H, W, std=2 * W ** -0.5), p + "b": r(H, W, std=2 * W ** -0.5), p + "A_log": r(H, std=0.8) - 0.5,
                  p + "dt_bias": r(H, std=1.0) - 2.0, p + "norm": 1 + r(m["vdim"], std=0.3)})

    t = {"embed": r(cfg["vocab"], W, std=1.0), "head": r(cfg["vocab"], W), "final.norm": 1 + r(W, std=0.3)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for q in (1, 2) if layer["mlp"] else (1,):
            t[p + f"norm{q}"] = 1 + r(W, std=0.3)
            t[p + f"hc{q}.in"] = 1.0 / S + r(S, std=0.5 * uneven / S)
            t[p + f"hc{q}.out"] = gain * (1 + r(S, std=0.4 * uneven))
            t[p + f"hc{q}.mix"] = 0.8 * torch.eye(S) + r(S, S, std=0.4 * uneven / S)
        if layer["type"] == "parallel":
            attention(p + "mix.left.", m["left"], "left")
            delta_rule(p + "mix.right.", m["right"])
            t.update({p + "mix.left.out": 1 + r(W, std=0.3), p + "mix.right.out": 1 + r(W, std=0.3)})
        else:
            attention(p + "mix.", m, layer["type"])
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            t.update({p + "mlp.gate": r(ff, W, std=2 * W ** -0.5), p + "mlp.up": r(ff, W), p + "mlp.down": r(W, ff)})
    return {n: v.to(dtype) for n, v in t.items()}


def greedy(cfg, tensors, tokens, n):
    """Greedy continuation by the oracle, and the smallest gap between its best and second-best logit."""
    toks, gap = list(tokens), float("inf")
    for _ in range(n):
        z = oracle.forward(cfg, tensors, toks)[-1]
        best = torch.topk(z, 2).values
        gap = min(gap, float(best[0] - best[1]) / float(z.std()))
        toks.append(int(z.argmax()))
    return toks[len(tokens):], gap
