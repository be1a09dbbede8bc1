"""Small random Vasolix models for the tests, as (config, weights) in the checkpoint format, and helpers around them."""
import json
import os

import torch

import vasolix_oracle as oracle


def attention(heads=4, kv_heads=2, dim=16, block=24, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else 1.3 * dim ** -0.5}
    if block:
        m["mask"] = {"size": block}
    return "attention", m


def gla(heads=2, dim=16, vdim=32, tau=4.0):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def moe(experts=5, top=2, ff=24, shared=40):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff},
            "shared": {"ff": shared} if shared else None}


def config(layers, width=64, vocab=101, eps=1e-5):
    """``layers``: list of (mixer, mlp or None) with mixer from :func:`attention` / :func:`gla`."""
    return {"architecture": "Vasolix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": m[0], "mixer": m[1], "mlp": f} for m, f in layers]}


# every branch, and sizes that are no multiples of anything in particular
MIXED = config([(attention(), moe()), (gla(), moe(top=1, shared=0)), (attention(6, 3, 24, 17, 0.3), None),
                (gla(3, 24, 20, 7.0), moe(4, 3, 20, 16)), (attention(4, 4, 8, 0), moe(3, 3, 12, 12))], width=60, vocab=101)
PLAIN = config([(gla(), moe()), (attention(), moe()), (gla(4, 8, 16, 1.0), moe())], width=64, vocab=96, eps=1e-3)


def weights(cfg, seed=0, rank=6, sharp=3.0, dtype=torch.bfloat16, clear_routing=False):
    """Random weights.  ``sharp`` scales the key and query norms so that single keys win the softmax, sinks are of the
    scores' size, the decays reach from almost 1 to strong, and norm weights differ from 1.

    ``clear_routing``: the first columns of the stream hold well-separated levels, another order for every token, that no
    layer changes (their norm weights are zero) and that dominate the router logits.  No choice of experts is then close
    enough for bf16 rounding to flip it, which would say nothing about the implementation."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def r(*shape, std=None):
        return torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5)

    t = {"embed": r(cfg["vocab"], W, std=1.0), "head": r(cfg["vocab"], W), "final.norm": 1 + r(W, std=0.3)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"] = 1 + r(W, std=0.3)
        if layer["type"] == "attention":
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            t.update({p + "mix.q": r(nq, W), p + "mix.k": r(nk, W), p + "mix.g": r(nq, W, std=2 * W ** -0.5), p + "mix.o": r(W, nq),
                      p + "mix.q.norm": sharp ** 0.5 * (1 + r(nq, std=0.3)), p + "mix.k.norm": sharp ** 0.5 * (1 + r(nk, std=0.3)),
                      p + "mix.sink": 1.5 + r(m["heads"], std=1.0)})
        else:
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            t.update({p + "mix.q": r(nk, W), p + "mix.k": r(nk, W), p + "mix.v": r(nv, W), p + "mix.g": r(nv, W), p + "mix.o": r(W, nv),
                      p + "mix.norm": 1 + r(m["vdim"], std=0.3), p + "mix.a1": r(rank, W), p + "mix.a2": r(nk, rank, std=1.5 * rank ** -0.5),
                      p + "mix.a2.b": r(nk, std=2.0)})
        f = layer["mlp"]
        if f is None:
            continue
        t[p + "norm2"] = 1 + r(W, std=0.3)
        t[p + "mlp.router"] = r(f["router"]["experts"], W, std=2 * W ** -0.5)
        for e in range(f["router"]["experts"]):
            t[p + f"mlp.e{e}.up"], t[p + f"mlp.e{e}.down"] = r(f["expert"]["ff"], W), r(W, f["expert"]["ff"])
        if f["shared"]:
            t[p + "mlp.shared.up"], t[p + "mlp.shared.down"] = r(f["shared"]["ff"], W), r(W, f["shared"]["ff"])
            t[p + "mlp.shared.sg"] = r(1, W)
    if clear_routing:
        E = max(f["router"]["experts"] for f in (l["mlp"] for l in cfg["layers"]) if f)
        levels = torch.linspace(-2.0, 2.0, E)
        t["embed"][:, :E] = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(cfg["vocab"])])
        for n, v in t.items():
            if n.endswith(("norm1", "norm2")):
                v[:E] = 0.0
            if n.endswith("router"):
                v.mul_(0.02)[:, :E] = torch.eye(v.shape[0], E)
    return {n: v.to(dtype) for n, v in t.items()}


def write(directory, cfg, tensors):
    from triton_distributed_b200.models import save_file

    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(tensors, os.path.join(directory, "model.safetensors"))
    return directory


def engine(directory, dtype, max_length=256, **kw):
    from triton_distributed_b200.models import Engine, ModelConfig

    eng = Engine(ModelConfig(model_name="checkpoint", max_length=max_length, dtype=dtype, checkpoint_dir=str(directory)), **kw)
    eng.backend = "triton_dist_gemm_ar"
    return eng


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def rel(got, want):
    """Largest root-mean-square difference of a row of logits (means taken off), in units of the logits' spread."""
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.std()).max())


def run_portions(eng, rid, tokens, sizes):
    """All logits of one request fed in portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        part = tokens[at:at + sizes[min(i, len(sizes) - 1)]]
        out.append(eng.step([(rid, part, list(range(len(part))))]))
        at, i = at + len(part), i + 1
    eng.end([rid])
    return torch.cat(out)


def greedy(cfg, tensors, tokens, n):
    """Greedy continuation by the oracle, and the smallest gap between its best and second-best logit."""
    toks, gap = list(tokens), float("inf")
    for _ in range(n):
        z = oracle.forward(cfg, tensors, toks)[-1]
        best = torch.topk(z, 2).values
        gap = min(gap, float(best[0] - best[1]) / float(z.std()))
        toks.append(int(z.argmax()))
    return toks[len(tokens):], gap
