"""Plain, slow restatement of the Tazitar decoder for the tests: one function per mechanism, token by token, no cache, no batch,
no code shared with the package.

A model is a ``config`` dictionary (``vocab``, ``width``, ``norm.eps``, ``streams``, ``loop``, ``layers``) and a dictionary of
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


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ rotation
def frequencies(rot):
    """Angle per position of every pair, and the factor on cos and sin."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0

    def turns(t):                       # index of the pair that makes t turns within the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot, interleaved):
    """First ``dims`` elements of the last dimension, at one position: pairs (2i, 2i + 1) or (i, i + dims / 2)."""
    f, mult = frequencies(rot)
    half = rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        c, s = math.cos(pos * f[i]) * mult, math.sin(pos * f[i]) * mult
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ------------------------------------------------------------------ attention
KINDS = {   # norm with weights before the rotation, weightless norm after it, pairs, sink
    "attention": dict(norm=True, unit=False, interleaved=False, sink=None),
    "left": dict(norm=False, unit=True, interleaved=False, sink="zero"),
    "attention_2": dict(norm=False, unit=True, interleaved=True, sink="learned")}


def visible(i, j):
    return j <= i


def head_scores(q, k, mixer):
    """Scores of one query of one head over the keys [n, dim]."""
    s = (k @ q) * mixer["scale"]
    cap = mixer.get("softcap")
    return cap * torch.tanh(s / cap) if cap else s


def softmax(s, sink=None):
    """Weights of the keys; ``sink`` is one more score, without a value."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else torch.exp(sink - m)))


def queries_keys(h, W, p, mixer, eps, kind):
    """Normed and rotated queries [T, heads, dim] and keys [T, kv_heads, dim]."""
    k_ = KINDS[kind]
    out = []
    for name, n in (("q", mixer["heads"]), ("k", mixer["kv_heads"])):
        x = (h @ W[p + name].T).reshape(h.shape[0], n, mixer["dim"])
        if k_["norm"]:
            x = rms(x, eps, W[p + name + ".norm"])
        x = torch.stack([rotate(x[t], t, mixer["rot"], k_["interleaved"]) for t in range(h.shape[0])])
        out.append(rms(x, eps) if k_["unit"] else x)
    return out


def attention(h, W, p, mixer, eps, kind):
    """h [T, width] of one sequence from position 0 -> [T, width]."""
    T, H, G, dv = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["vdim"]
    q, k = queries_keys(h, W, p, mixer, eps, kind)
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        sink = {None: None, "zero": torch.zeros((), dtype=h.dtype), "learned": W.get(p + "sink", [None] * H)[a]}[KINDS[kind]["sink"]]
        for i in range(T):
            n = sum(1 for j in (i, i + 1) if visible(i, j)) + i
            out[i, a] = softmax(head_scores(q[i, a], k[:n, g], mixer), sink) @ v[:n, g]
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------ gated delta rule
def short_conv(x, w):
    """Causal convolution per channel: x [T, C], w [C, taps], the last column belongs to the current token."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            if t - j >= 0:
                out[t] += w[:, taps - 1 - j] * x[t - j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_step(S, q, k, v, g, beta):
    """One token of all heads: S [H, dk, dv] -> (new S, read-out [H, dv])."""
    S = g[:, None, None] * S
    u = beta[:, None] * (v - torch.einsum("hkv,hk->hv", S, k))
    S = S + k[:, :, None] * u[:, None, :]
    return S, torch.einsum("hkv,hk->hv", S, q)


def delta_inputs(h, W, p, mixer):
    """Per token: q, k [T, heads, dim] (every head has its own copy), v [T, heads, vdim], decay and step size [T, heads]."""
    T, H, G = h.shape[0], mixer["heads"], mixer["kv_heads"]
    q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    q, k = (unit(x.reshape(T, G, -1)).repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    return q * mixer["dim"] ** -0.5, k, v.reshape(T, H, -1), g, beta


def delta_rule(h, W, p, mixer, eps):
    T, H = h.shape[0], mixer["heads"]
    q, k, v, g, beta = delta_inputs(h, W, p, mixer)
    S = torch.zeros(H, mixer["dim"], mixer["vdim"], dtype=h.dtype)
    out = torch.zeros(T, H, mixer["vdim"], dtype=h.dtype)
    for t in range(T):
        S, out[t] = delta_step(S, q[t], k[t], v[t], g[t], beta[t])
    gate = silu(h @ W[p + "g"].T)
    return (rms(out, eps, W[p + "norm"]).reshape(T, -1) * gate) @ W[p + "o"].T


# ------------------------------------------------------------------ layers
def mixer_out(h, W, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] != "parallel":
        return attention(h, W, p, m, eps, layer["type"])
    left = attention(h, W, p + "left.", m["left"], eps, "left")
    right = delta_rule(h, W, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps, W[p + "left.out"]) + rms(right, eps, W[p + "right.out"]))


def feed_forward(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def hyper(x, W, p, sublayer):
    """Streams x [s, T, width] around one sublayer: its input is a mixture of them, its output goes to all of them."""
    y = sublayer(torch.einsum("s,stw->tw", W[p + "in"], x))
    return torch.einsum("ab,atw->btw", W[p + "mix"], x) + W[p + "out"][:, None, None] * y


def passes(config):
    """Layer numbers in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(config, weights, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) collects the sum of the streams after every layer run."""
    W = {n: (t.to(DT) if t.dtype.is_floating_point else t) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)].unsqueeze(0).repeat(config["streams"], 1, 1)
    for i in passes(config):
        p, layer = f"l{i}.", config["layers"][i]
        x = hyper(x, W, p + "hc1.", lambda u: mixer_out(rms(u, eps, W[p + "norm1"]), W, p + "mix.", layer, eps))
        if layer.get("mlp"):
            x = hyper(x, W, p + "hc2.", lambda u: feed_forward(rms(u, eps, W[p + "norm2"]), W, p + "mlp."))
        if streams is not None:
            streams.append(x.sum(0))
    return rms(x.sum(0), eps, W["final.norm"]) @ W["head"].T
