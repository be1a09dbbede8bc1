"""Small random Lisenex models for the tests, as (config, weights) in the checkpoint format; the helpers around a model are those
of ``vasolix_cases``."""
import torch

import lisenex_oracle as oracle
from vasolix_cases import engine, prompt, rel, run_portions, write  # noqa: F401


def latent(heads=4, dim=16, rot=8, vdim=24, rank=40, kv_from=None, base=500.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
         "scale": scale if scale is not None else (dim + rot) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, shared=40, identity=1, groups=(2, 1)):
    r = {"experts": experts, "top": top, "identity": identity}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def config(layers, width=64, vocab=101, eps=1e-5, scale=1.0):
    """``layers``: list of (mixer, mlp or None)."""
    return {"architecture": "Lisenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


# every branch, and sizes that are no multiples of anything in particular: rows shared with the layer before, with a layer further
# back and by several layers; head counts that differ between sharers; no feed-forward; no groups, no identity, no shared expert
MIXED = config([(latent(), moe()), (latent(6, 12, 8, 20, 40, kv_from=0), dense(50)), (latent(3, 20, 12, 10, 36, base=90.0, scale=0.3), None),
                (latent(2, 18, 8, 30, 40, kv_from=0), moe(4, 3, 20, 16, 2, None)), (latent(5, 9, 12, 33, 36, kv_from=2, base=90.0), moe(7, 3, 12, 0, 1, (4, 2))),
                (latent(1, 64, 32, 8, 64), moe(3, 3, 12, 12, 0, None))], width=60, vocab=101, scale=0.6)
PLAIN = config([(latent(), dense()), (latent(kv_from=0), moe()), (latent(2, 32, 16, 16, 24), moe(7, 2, 16, 0, 1, (4, 1)))], width=64, vocab=96,
               eps=1e-3, scale=2.0)


def weights(cfg, seed=0, sharp=3.0, dtype=torch.bfloat16, clear_routing=False):
    """Random weights.  ``sharp`` scales the unrotated and rotated scores so that single keys win the softmax; norm weights differ
    from 1, choice corrections are of the scores' size and mostly negative, so that both the correction and minus infinity for the
    groups that are left out change choices.

    ``clear_routing``: the first columns of the stream hold equally spaced levels, another order for every token, that no layer
    changes and that only the routers read.  They hold most of the stream's energy, so that its root mean square hardly varies and
    the router scores of every token are (in another order) the same well-separated set.  No choice is then close enough for bf16
    rounding to flip it, which would say nothing about the implementation."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5)

    t = {"embed": r(cfg["vocab"], W, std=1.0), "final.norm": 1 + r(W, std=0.3)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, rot, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        t[p + "norm1"] = 1 + r(W, std=0.3)
        t.update({p + "mix.q": r(H * (d + rot), W, std=sharp ** 0.5 * W ** -0.5), p + "mix.uk": r(H * d, R, std=sharp ** 0.5 * R ** -0.5),
                  p + "mix.uv": r(H * dv, R), p + "mix.g": r(H * dv, W, std=2 * W ** -0.5), p + "mix.o": r(W, H * dv)})
        if "kv_from" not in m:
            dkv = r(R + rot, W)
            dkv[R:] *= sharp ** 0.5
            t.update({p + "mix.dkv": dkv, p + "mix.dkv.norm": 1 + r(R, std=0.3)})
        f = layer["mlp"]
        if f is None:
            continue
        t[p + "norm2"] = 1 + r(W, std=0.3)
        if f["kind"] == "dense":
            t.update({p + "mlp.up": r(f["ff"], W), p + "mlp.up.b": r(f["ff"], std=0.5), p + "mlp.down": r(W, f["ff"]), p + "mlp.down.b": r(W, std=0.5)})
            continue
        E = f["router"]["experts"] + f["router"]["identity"]
        t[p + "mlp.router"] = r(E, W, std=2 * W ** -0.5)
        t[p + "mlp.correction"] = r(E, std=0.2) - 0.3
        names = [f"e{e}" for e in range(f["router"]["experts"])] + (["shared"] if f["shared"] else [])
        for n in names:
            ff = f["shared"]["ff"] if n == "shared" else f["expert"]["ff"]
            t.update({p + f"mlp.{n}.gate": r(ff, W, std=2 * W ** -0.5), p + f"mlp.{n}.up": r(ff, W, std=2 * W ** -0.5), p + f"mlp.{n}.down": r(W, ff)})
    if clear_routing:
        E = max([f["router"]["experts"] + f["router"]["identity"] for f in (l["mlp"] for l in cfg["layers"]) if f and f["kind"] == "moe"] + [0])
        lev = torch.arange(E) - (E - 1) / 2
        amp = (10 * 1.5 * W / float((lev * lev).sum())) ** 0.5
        root = (11 * 1.5) ** 0.5                       # of the stream's mean square
        t["embed"][:, :E] = amp * torch.stack([lev[torch.randperm(E, generator=g)] for _ in range(cfg["vocab"])])
        t["embed"] /= cfg["embedding"]["scale"]
        for n, v in t.items():
            if n.endswith(("mix.o", ".down", "down.b")):
                v *= 0.3
                v[:E] = 0.0
            if n.endswith(("norm1", "norm2", "final.norm")):
                v *= root
                v[:E] = 0.05 if n.endswith("norm2") else 0.0
            if n.endswith("router"):
                v.mul_(0.01)[:, :E] = torch.eye(v.shape[0], E) * (1.2 * root / amp / 0.05)
            if n.endswith("correction"):
                v.copy_(-0.3 + 0.1 * (torch.arange(v.numel()) % 2))
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
