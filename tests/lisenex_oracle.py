"""Plain, slow restatement of the Lisenex decoder for the tests: one function per mechanism, one query at a time, no cache,
no batch, no code shared with the package.

A model is a ``config`` dictionary (``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers``) and a dictionary of
weights under the names of the checkpoint format.  Everything is computed in the dtype ``DT`` (float64 by default).
"""
import math

import torch

DT = torch.float64


def rms(x, eps, w=None):
    """Root-mean-square norm over the last dimension, the epsilon inside the root."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------ latent attention
def rotate(x, pos, base):
    """Rotation of the last dimension at one position: neighbours (2i, 2i + 1) turn by pos * base^(-2i / dims)."""
    dims = x.shape[-1]
    out = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(i, j):
    return j <= i


def latent(h, W, p, mixer, eps):
    """What a layer keeps of its tokens: the normed latent [T, kv_rank] and the rotated key part [T, rot_dim]."""
    R = mixer["kv_rank"]
    z = h @ W[p + "dkv"].T
    c = rms(z[:, :R], eps, W[p + "dkv.norm"])
    kr = torch.stack([rotate(z[t, R:], t, mixer["rot"]["base"]) for t in range(h.shape[0])])
    return c, kr


def head_scores(qn, qr, kn, kr, scale):
    """Scores of one query of one head over the keys: the unrotated and the rotated parts' products, added and scaled."""
    return (kn @ qn + kr @ qr) * scale


def latent_attention(h, W, p, mixer, eps, kept=None):
    """h [T, width] of one sequence from position 0 -> ([T, width], what the layer keeps).  ``kept``: what another layer
    keeps, which this layer then uses in place of its own."""
    T, H = h.shape[0], mixer["heads"]
    d, r, dv = mixer["dim"], mixer["rot_dim"], mixer["vdim"]
    c, kr = latent(h, W, p, mixer, eps) if kept is None else kept
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    k = (c @ W[p + "uk"].T).reshape(T, H, d)
    v = (c @ W[p + "uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        js = [j for j in range(T) if visible(i, j)]
        qr = rotate(q[i, :, d:], i, mixer["rot"]["base"])
        for a in range(H):
            s = head_scores(q[i, a, :d], qr[a], k[js, a], kr[js], mixer["scale"])
            e = torch.exp(s - s.max())
            out[i, a] = (e / e.sum()) @ v[js, a]
    return (out.reshape(T, H * dv) * gate) @ W[p + "o"].T, (c, kr)


# ------------------------------------------------------------------ feed-forward
def dense(h, W, p):
    up = h @ W[p + "up"].T + W[p + "up.b"]
    return torch.clamp(up, min=0.0) ** 2 @ W[p + "down"].T + W[p + "down.b"]


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, correction, top, groups=None):
    """Ids and weights of one token's experts, best first, from its router logits (identity experts are the last ids)."""
    e = torch.exp(z - z.max())
    s = e / e.sum()
    choice = s + correction
    if groups:
        size = z.shape[0] // groups["count"]
        best = [float(choice[g * size:(g + 1) * size].max()) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -best[g])[:groups["keep"]]
        choice = torch.stack([choice[i] if i // size in kept else torch.tensor(-math.inf, dtype=z.dtype) for i in range(z.shape[0])])
    ids = torch.argsort(choice, descending=True, stable=True)[:top]
    return ids.tolist(), s[ids]


def moe(h, W, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, w = route(W[p + "router"] @ h[t], W[p + "correction"], mlp["router"]["top"], mlp["router"].get("groups"))
        for e, we in zip(ids, w):
            out[t] += we * (expert(h[t], W, f"{p}e{e}.") if e < mlp["router"]["experts"] else h[t])
        if mlp.get("shared"):
            out[t] += expert(h[t], W, p + "shared.")
    return out


def feed_forward(h, W, p, mlp):
    return dense(h, W, p) if mlp["kind"] == "dense" else moe(h, W, p, mlp)


# ------------------------------------------------------------------ the model
def forward(config, weights, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) collects the residual stream after every layer."""
    W = {n: (t.to(DT) if t.dtype.is_floating_point else t) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        src = m.get("kv_from")
        y, kept[i] = latent_attention(rms(x, eps, W[p + "norm1"]), W, p + "mix.", m, eps, None if src is None else kept[src])
        if layer.get("mlp"):
            y = y + feed_forward(rms(x, eps, W[p + "norm2"]), W, p + "mlp.", layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x)
    return rms(x, eps, W["final.norm"]) @ W["embed"].T
