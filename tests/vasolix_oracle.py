"""Plain, slow restatement of the Vasolix decoder for the tests: one function per mechanism, one token or one sequence
at a time, no cache, no batch, no code shared with the package.

A model is a ``config`` dictionary (``vocab``, ``width``, ``norm.eps``, ``layers``) and a dictionary of weights under the
names of the checkpoint format.  Everything is computed in the dtype of ``DT`` (float64 by default).
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


# ------------------------------------------------------------------ attention
def visible(i, j, size):
    """Causal, and only inside the block of ``size`` positions that i lies in (blocks counted from position 0)."""
    return j <= i and (not size or i // size == j // size)


def sink_softmax(scores, sink):
    """Softmax of a list of scores whose denominator has one extra term exp(sink)."""
    m = max(float(scores.max()), float(sink))
    e = torch.exp(scores - m)
    return e / (e.sum() + math.exp(float(sink) - m))


def attention_scores(q, k, i, head, group, scale, size):
    """Visible positions of query i and their scaled scores for one head."""
    js = [j for j in range(k.shape[0]) if visible(i, j, size)]
    return js, torch.stack([(q[i, head] * k[j, head // group]).sum() for j in js]) * scale


def attention(h, W, p, mixer, eps):
    """h [T, width] of one sequence from position 0 -> [T, width]."""
    T = h.shape[0]
    H, G, d = mixer["heads"], mixer["kv_heads"], mixer["dim"]
    size = (mixer.get("mask") or {}).get("size", 0)
    kraw = h @ W[p + "k"].T
    q = rms(h @ W[p + "q"].T, eps, W[p + "q.norm"]).reshape(T, H, d)
    k = rms(kraw, eps, W[p + "k.norm"]).reshape(T, G, d)
    v = kraw.reshape(T, G, d)                       # the values are the keys before their norm
    gate = sigmoid(h @ W[p + "g"].T)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for i in range(T):
        for a in range(H):
            js, s = attention_scores(q, k, i, a, H // G, mixer["scale"], size)
            w = sink_softmax(s, W[p + "sink"][a])
            out[i, a] = (w[:, None] * v[js, a // (H // G)]).sum(0)
    return (out.reshape(T, H * d) * gate) @ W[p + "o"].T


# ------------------------------------------------------------------ gated linear attention
def gla_decay(h, W, p, tau):
    """Per-channel decay of every token, in (0, 1)."""
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return sigmoid(z) ** (1.0 / tau)


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, dk], v [T, H, dv] -> o [T, H, dv] and the state [H, dk, dv] after the last token."""
    T, H, dk = k.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla(h, W, p, mixer, eps):
    T = h.shape[0]
    H, dk, dv = mixer["heads"], mixer["dim"], mixer["vdim"]
    q = (h @ W[p + "q"].T * dk ** -0.5).reshape(T, H, dk)
    k = (h @ W[p + "k"].T).reshape(T, H, dk)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    alpha = gla_decay(h, W, p, mixer["tau"]).reshape(T, H, dk)
    o, _ = gla_recurrence(q, k, v, alpha)
    o = rms(o, eps, W[p + "norm"]).reshape(T, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------ mixture of experts
def expert(h, W, p):
    return torch.clamp(h @ W[p + "up"].T, min=0.0) ** 2 @ W[p + "down"].T


def route(h, W, p, top):
    """Expert ids and weights of one token, best first."""
    s = sigmoid(W[p + "router"] @ h)
    best = torch.argsort(s, descending=True, stable=True)[:top]
    return best.tolist(), s[best]


def moe(h, W, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, w = route(h[t], W, p, mlp["router"]["top"])
        for e, we in zip(ids, w):
            out[t] += expert(we * h[t], W, f"{p}e{e}.")
        if mlp.get("shared"):
            out[t] += sigmoid(W[p + "shared.sg"] @ h[t]) * expert(h[t], W, p + "shared.")
    return out


# ------------------------------------------------------------------ the model
MIXERS = {"attention": attention, "gla": gla}


def forward(config, weights, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) collects the residual stream after every layer."""
    W = {n: (t.to(DT) if t.dtype.is_floating_point else t) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + rms(MIXERS[layer["type"]](x, W, p + "mix.", layer["mixer"], eps), eps, W[p + "norm1"])
        if layer.get("mlp"):
            x = x + rms(moe(x, W, p + "mlp.", layer["mlp"]), eps, W[p + "norm2"])
        if streams is not None:
            streams.append(x)
    return rms(x, eps, W["final.norm"]) @ W["head"].T
