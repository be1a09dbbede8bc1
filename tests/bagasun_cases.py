"""Small random Bagasun models for the tests, as (config, weights) in the checkpoint format; the helpers around a model are those
of ``vasolix_cases``."""
import torch

import bagasun_oracle as oracle
from vasolix_cases import engine, prompt, rel, run_portions, write  # noqa: F401


def attn(heads=4, kv_heads=2, dim=16, vdim=24, window=13, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.4 * dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return m


def diff(heads=4, kv_heads=2, dim=16, vdim=24, window=11, rot_dims=12, mix=0.4, scale=None, base=300.0, **scaling):
    """``scaling``: factor, original, low, high."""
    rot = {"base": base, "dims": rot_dims, **({"scaling": scaling} if scaling else {})}
    return {**attn(heads, kv_heads, dim, vdim, window, scale), "diff": mix, "rot": rot}


def mamba(heads=4, groups=2, state=12, vdim=20, conv=4, norm_groups=2):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}


def config(layers, width=64, vocab=101, eps=1e-5, scale=1.0):
    """``layers``: list of (type, mixer, ff or None), or the number of an earlier layer whose weights are used again."""
    out = []
    for l in layers:
        if isinstance(l, int):
            src = out[l]
            out.append({**src, "weights_of": src.get("weights_of", l)})
        else:
            t, m, f = l
            out.append({"type": t, "mixer": m, "mlp": None if f is None else {"kind": "dense", "ff": f}})
    return {"architecture": "Bagasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": out}


BAND = dict(factor=3.0, original=40, low=0.7, high=3.0)
# every branch, and sizes that are no multiples of anything in particular: windows of different lengths (one of a single token, one layer
# without), partial rotations, head groups of different sizes, one KV head for all, norm groups that cut heads, convolutions of
# several lengths, no feed-forward, shared layers apart from and beside their source
MIXED = config([("attention", attn(6, 3, 20, 28, 9), 50), ("mamba2", mamba(6, 2, 12, 20, 3, 3), 42), ("attention_2", diff(4, 2, 18, 26, 7, 10, 0.3, **BAND), None),
                1, ("attention", attn(2, 1, 8, 12, 1, 0.5), 24), 0, 0, ("mamba2", mamba(3, 1, 18, 12, 1, 4), None), ("attention_2", diff(3, 1, 12, 8, 0, 12, 0.7), 30), 2, 8],
               width=60, vocab=101, eps=2e-3, scale=1.7)
PLAIN = config([("mamba2", mamba(conv=4), 40), ("attention_2", diff(factor=2.0, original=30, low=1.0, high=2.5), 56), ("attention", attn(), 32), 0, 1], width=64, vocab=96,
               eps=1e-3, scale=2.0)


def weights(cfg, seed=0, dtype=torch.bfloat16, sharp=2.0, gain=1.0):
    """Random weights.  Queries and keys give scores of which single ones stand out, distance terms and offsets are of the scores' size, the
    second map counts, decays reach from almost 1 to strong, norms differ from 1 (``gain``: how much a sublayer adds)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5)

    def one(mean):
        return (mean * (1 + r(1, std=0.3))).reshape(())

    t = {"embed": r(cfg["vocab"], W, std=1.0), "head": r(cfg["vocab"], W), "final.norm": one(1.2)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}.mix.", layer["mixer"]
        H = m["heads"]
        if layer["type"] == "mamba2":
            inner, shared = H * m["vdim"], m["groups"] * m["state"]
            t.update({p + "in": r(2 * inner + 2 * shared + H, W, std=1.5 * W ** -0.5), p + "conv": r(inner + 2 * shared, m["conv"], std=1.5 * m["conv"] ** -0.5),
                      p + "conv.b": r(inner + 2 * shared, std=0.4), p + "dt_bias": r(H, std=1.0) - 1.0, p + "A_log": r(H, std=0.8) - 0.5, p + "D": r(H, std=1.0),
                      p + "norm": 1 + r(inner, std=0.3), p + "o": r(W, inner)})
        else:
            G, maps = m["kv_heads"], 2 if layer["type"] == "attention_2" else 1
            rows = {"q": H * maps * m["dim"], "k": G * maps * m["dim"], "v": G * m["vdim"]}
            t.update({p + n: r(k, W, std=(sharp if maps == 2 and n != "v" else 1.0) * W ** -0.5) for n, k in rows.items()})
            t[p + "o"] = r(W, H * m["vdim"])
            if maps == 1:
                t.update({p + n + ".b": r(k, std=0.5) for n, k in rows.items()})
                t.update({p + n + ".norm": (sharp if n == "q" else 1.0) * (1 + r(rows[n], std=0.3)) for n in "qk"})
                t.update({p + "r1": 0.3 + r(H, std=1.0).abs(), p + "r2": 0.2 + r(H, std=1.0).abs(), p + "pb": r(H, std=0.7) - 0.5})
            else:
                t.update({p + n: r(m["dim"], std=0.8 * m["dim"] ** -0.25) for n in ("lq1", "lk1", "lq2", "lk2")})
                t[p + "g"] = r(H, W, std=1.5 * W ** -0.5)
        for q in (1, 2) if layer["mlp"] else (1,):
            t[f"l{i}.norm{q}"], t[f"l{i}.norm{q}b"] = one(1.0), one(gain)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            t.update({f"l{i}.mlp.gate": r(ff, W, std=2 * W ** -0.5), f"l{i}.mlp.up": r(ff, W), f"l{i}.mlp.down": r(W, ff)})
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
