"""Plain, slow restatement of the Bagasun decoder for the tests: one function per mechanism, token by token, no cache, no batch,
no code shared with the package.

A model is a ``config`` dictionary (``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers``) and a dictionary of weights
under the names of the checkpoint format.  Everything is computed in the dtype ``DT`` (float64 by default).
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


def window_of(mixer):
    return (mixer.get("mask") or {}).get("size") or 0


def visible(i, j, window):
    """Whether position i sees position j (window 0: every earlier one)."""
    return 0 <= i - j and (window == 0 or i - j < window)


# ------------------------------------------------------------------ attention with independent sigmoid weights
def distance_bias(dist, r1, r2):
    """What a key at distance ``dist`` loses."""
    return r1 * torch.log(1.0 + r2 * dist)


def sigmoid_weights(q, k, dist, scale, r1, r2, pb):
    """Weights of the keys [n, dim] at distances ``dist`` [n] for one query of one head; they do not sum to one."""
    return sigmoid((k @ q) * scale - distance_bias(dist, r1, r2) + pb)


def projection(h, W, name):
    y = h @ W[name].T
    return y + W[name + ".b"] if name + ".b" in W else y


def sigmoid_attention(h, W, p, mixer, eps):
    """h [T, width] of one sequence from position 0 -> [T, width]."""
    T, H, G, d, dv, win = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"], window_of(mixer)
    q = rms(projection(h, W, p + "q"), eps, W[p + "q.norm"]).reshape(T, H, d)
    k = rms(projection(h, W, p + "k"), eps, W[p + "k.norm"]).reshape(T, G, d)
    v = projection(h, W, p + "v").reshape(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        seen = [j for j in range(T) if visible(i, j, win)]
        dist = torch.tensor([i - j for j in seen], dtype=h.dtype)
        for a in range(H):
            g = a // (H // G)
            out[i, a] = sigmoid_weights(q[i, a], k[seen, g], dist, mixer["scale"], W[p + "r1"][a], W[p + "r2"][a], W[p + "pb"][a]) @ v[seen, g]
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------ differential attention
def frequencies(rot):
    """Angle per position of every pair."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            turn = 2.0 * math.pi / f
            if turn > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif turn >= sc["original"] / sc["high"]:
                s = (sc["original"] / turn - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, pos, rot):
    """First ``dims`` elements of the last dimension, at one position: element i turns with i + dims / 2."""
    half = rot["dims"] // 2
    out = x.clone()
    for i, f in enumerate(frequencies(rot)):
        c, s = math.cos(pos * f), math.sin(pos * f)
        out[..., i] = x[..., i] * c - x[..., i + half] * s
        out[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return out


def softmax(s):
    e = torch.exp(s - s.max())
    return e / e.sum()


def mix_of_maps(W, p, diff):
    """How much of the second map is taken off, one number for the layer."""
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, W, p, mixer, eps):
    T, H, G, d, dv, win = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"], window_of(mixer)
    q, k = ((h @ W[p + n].T).reshape(T, m, 2, d) for n, m in (("q", H), ("k", G)))
    q, k = (torch.stack([rotate(x[t], t, mixer["rot"]) for t in range(T)]) for x in (q, k))
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    gate = sigmoid(h @ W[p + "g"].T)
    lam = mix_of_maps(W, p, mixer["diff"])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        seen = [j for j in range(T) if visible(i, j, win)]
        for a in range(H):
            g = a // (H // G)
            maps = [softmax((k[seen, g, m] @ q[i, a, m]) * mixer["scale"]) @ v[seen, g] for m in (0, 1)]
            out[i, a] = combine_maps(*maps, lam, mixer["diff"], eps) * gate[i, a]
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------ state space layer
def short_conv(x, w, b):
    """Causal convolution per channel: x [T, C], w [C, taps], the last column belongs to the current token."""
    T, taps = x.shape[0], w.shape[1]
    out = b.expand(T, -1).clone()
    for t in range(T):
        for j in range(taps):
            if t - j >= 0:
                out[t] += w[:, taps - 1 - j] * x[t - j]
    return out


def ssd_step(S, x, B, C, dt, a, D):
    """One token of all heads: S [H, N, dv], x [H, dv], B and C [H, N], step sizes and decay rates [H] -> (new S, y [H, dv])."""
    S = torch.exp(-a * dt)[:, None, None] * S + dt[:, None, None] * B[:, :, None] * x[:, None, :]
    return S, torch.einsum("hnv,hn->hv", S, C) + D[:, None] * x


def gated_group_norm(y, z, groups, w, eps):
    """y [T, inner]: the gate first, then a norm of every part of its own."""
    T = y.shape[0]
    return rms((y * silu(z)).reshape(T, groups, -1), eps).reshape(T, -1) * w


def mamba2(h, W, p, mixer, eps):
    T, H, G, N, dv = h.shape[0], mixer["heads"], mixer["groups"], mixer["state"], mixer["vdim"]
    inner = H * dv
    z, x, B, C, dt = (h @ W[p + "in"].T).split([inner, inner, G * N, G * N, H], dim=1)
    xbc = silu(short_conv(torch.cat([x, B, C], dim=1), W[p + "conv"], W[p + "conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], dim=1)
    dt = softplus(dt + W[p + "dt_bias"])
    x = x.reshape(T, H, dv)
    B, C = (t.reshape(T, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    S, y = torch.zeros(H, N, dv, dtype=h.dtype), torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S, y[t] = ssd_step(S, x[t], B[t], C[t], dt[t], torch.exp(W[p + "A_log"]), W[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, mixer["norm_groups"], W[p + "norm"], eps) @ W[p + "o"].T


# ------------------------------------------------------------------ layers
MIXERS = {"attention": sigmoid_attention, "attention_2": differential_attention, "mamba2": mamba2}


def feed_forward(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def weights_layer(config, i):
    """Layer whose tensors layer i uses."""
    return config["layers"][i].get("weights_of", i)


def sandwich(x, W, p, n, eps, sublayer):
    """A sublayer between two norms of one number each."""
    return x + rms(sublayer(rms(x, eps, W[f"{p}norm{n}"])), eps, W[f"{p}norm{n}b"])


def forward(config, weights, tokens, streams=None):
    """Logits [T, vocab] of one sequence; ``streams`` (a list) collects the residual stream after every layer."""
    W = {n: t.to(DT) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{weights_layer(config, i)}."
        x = sandwich(x, W, p, 1, eps, lambda h: MIXERS[layer["type"]](h, W, p + "mix.", layer["mixer"], eps))
        if layer.get("mlp"):
            x = sandwich(x, W, p, 2, eps, lambda h: feed_forward(h, W, p + "mlp."))
        if streams is not None:
            streams.append(x)
    return rms(x, eps, W["final.norm"]) @ W["head"].T
