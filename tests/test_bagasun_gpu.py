"""Bagasun on one GPU: every kernel alone and the whole model (bf16 and fp32) against the plain oracle on the CPU."""
import json
import os
import subprocess
import sys

import pytest
import torch

import bagasun_cases as cases
import bagasun_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {torch.bfloat16: 0.1, torch.float32: 3e-5}
DTYPES = [torch.bfloat16, torch.float32]


@pytest.fixture(scope="module")
def rt():
    import triton_distributed_b200 as tdb

    tdb.initialize_distributed(seed=0)
    return tdb.get_runtime()


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, dtype, scale=1.0):
    want = want.double()
    err = (got.double().cpu() - want).abs().max().item() / (want.abs().max().item() + 1e-9)
    assert err < scale * (1.2e-2 if dtype == torch.bfloat16 else 2e-5), err


def dev(t):
    return None if t is None else t.to(DEV)


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def i64(v):
    return torch.tensor(v, dtype=torch.int64, device=DEV)


def bounds(lens):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return cu


# ------------------------------------------------------------------ sublayers between two norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,real", [(8, 5), (72, 67), (256, 256), (4096, 4090), (4104, 4104), (9000, 9000)])
@pytest.mark.parametrize("one", [True, False])
def test_sandwich_step(rt, dtype, W, real, one):
    from triton_distributed_b200 import ops

    T, V, eps, scale = 5, 11, 1e-3, 2.5
    mask = (torch.arange(W) < real).float()
    x0, y, table = rnd(T, W) * mask, (rnd(T, W, seed=1) * mask).to(dtype), (rnd(V, W, seed=2) * mask).to(dtype)
    post, pre = (1 + 0.3 * rnd(1 if one else W, seed=i) for i in (3, 4))
    start = (torch.tensor([10, 0, 3, 3, 7]), table, scale)

    def want(x, with_y):
        x = x[:, :real].double()
        if with_y:
            x = x + oracle.rms(y[:, :real].double(), eps, post[:real].double())
        return x, oracle.rms(x, eps, pre[:real].double())

    last = (dev(y), dev(post))
    x = dev(x0)
    h = ops.sandwich_step(x, last, dev(pre), real, eps, dtype)
    xw, hw = want(x0, True)
    close(x[:, :real], xw, torch.float32)
    close(h[:, :real], hw, dtype)
    assert real == W or (float(x[:, real:].abs().max()) == 0 and float(h[:, real:].abs().max()) == 0)
    # some rows only: the stream stays as it is
    x, rows = dev(x0), torch.tensor([4, 0, 4])
    h = ops.sandwich_step(x, last, dev(pre), real, eps, dtype, dev(rows))
    assert torch.equal(x.cpu(), x0)
    close(h[:, :real], hw[rows], dtype)
    # nothing to norm; nothing to add; the start of a model
    assert ops.sandwich_step(x, last, None, real, eps, dtype) is None
    close(x[:, :real], xw, torch.float32)
    x = dev(x0)
    close(ops.sandwich_step(x, None, dev(pre), real, eps, dtype)[:, :real], want(x0, False)[1], dtype)
    assert torch.equal(x.cpu(), x0)
    x = torch.full((T, W), float("nan"), device=DEV)
    h = ops.sandwich_step(x, None, dev(pre), real, eps, dtype, start=(dev(start[0]), dev(table), scale))
    first = table.float()[start[0]] * scale
    assert torch.equal(x.cpu(), first)
    close(h[:, :real], want(first, False)[1], dtype)


# ------------------------------------------------------------------ queries, keys, values
PREPS = [(3, 1, 1, 64, 48, 64, 40, 48), (4, 4, 2, 64, 64, 128, 128, 16), (8, 4, 2, 128, 100, 64, 64, 34), (2, 2, 2, 264, 260, 136, 130, 200), (6, 2, 2, 8, 7, 16, 9, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Gk,G,dk,dim,dv,vdim,turn", PREPS)
@pytest.mark.parametrize("norm,biased,rotated", [(True, True, False), (False, False, True), (True, True, True), (False, True, False)])
def test_qkv_prep(rt, dtype, Hq, Gk, G, dk, dim, dv, vdim, turn, norm, biased, rotated):
    from triton_distributed_b200 import ops

    T, eps, far = 5, 1e-3, 6000
    raw = [rnd(T, n, d, seed=i).to(dtype) for i, (n, d) in enumerate(((Hq, dim), (Gk, dim), (G, vdim)))]
    b = [rnd(n, d, seed=5 + i, std=0.5) for i, (n, d) in enumerate(((Hq, dim), (Gk, dim), (G, vdim)))]
    pad = lambda x, d: torch.nn.functional.pad(x, (0, d - x.shape[-1]))   # noqa: E731
    sizes = (dk, dk, dv)
    z = torch.cat([pad(x, d).reshape(T, -1) for x, d in zip(raw, sizes)] + [torch.ones(T, 8, dtype=dtype)], dim=1).to(DEV)
    bias = torch.cat([pad(x, d).reshape(-1) for x, d in zip(b, sizes)]) if biased else None
    qw, kw = (1 + 0.3 * rnd(n, dim, seed=8 + i) for i, n in enumerate((Hq, Gk)))
    norms = (dev(pad(qw, dk).reshape(-1)), dev(pad(kw, dk).reshape(-1)), Hq * dim, Gk * dim) if norm else None
    pos = torch.tensor([far - 1, 0, 77, 1, 3000])
    rot = {"base": 300.0, "dims": turn, "scaling": dict(factor=3.0, original=512, low=1.0, high=8.0)}
    table = ops.rope_table(300.0, turn, turn, far, DEV, ops.BandScaling.from_json(rot["scaling"])) if rotated else None
    rows, rows2 = torch.tensor([6, 0, 3, 5, 1]), torch.tensor([2, -1, 0, 1, -1])
    ka, va, kb, vb = (torch.zeros(n, *s, dtype=dtype, device=DEV) for n, s in ((7, (Gk, dk)), (7, (G, dv)), (3, (Gk, dk)), (3, (G, dv))))
    got = ops.qkv_prep(z, Hq, Gk, G, dk, dv, dev(bias), norms, eps, table, turn if rotated else 0, dev(pos), (ka, va, dev(rows)), (kb, vb, dev(rows2)))

    def want(i, w):
        x = raw[i].double() + (b[i].double() if biased else 0)
        if norm and w is not None:
            x = oracle.rms(x.reshape(T, -1), eps).reshape(x.shape) * w.double()
        if rotated and w is not None:
            x = torch.stack([oracle.rotate(x[t], int(pos[t]), rot) for t in range(T)])
        return x

    q, k, v = want(0, qw), want(1, kw), want(2, None)
    close(got[..., :dim], q, dtype)
    close(ka[dev(rows)][..., :dim], k, dtype)
    close(va[dev(rows)][..., :vdim], v, dtype)
    for t, r2 in enumerate(rows2.tolist()):
        if r2 >= 0:
            close(kb[r2][..., :dim], k[t], dtype, 2.0)
            close(vb[r2][..., :vdim], v[t], dtype, 2.0)
    for x, d in ((got, dim), (ka, dim), (va, vdim), (kb, dim), (vb, vdim)):
        assert x.shape[-1] == d or float(x[..., d:].abs().max()) == 0
    assert float(ka[[2, 4]].abs().max()) == 0 and float(va[[2, 4]].abs().max()) == 0


# ------------------------------------------------------------------ attention over a window
class Heads:
    """Weights of a layer of one kind for random heads, and the oracle's output of one query over given keys."""

    def __init__(self, kind, H, dv, seed, n, sharp=1.0):
        self.kind, self.H, self.dv = kind, H, dv
        self.maps = 2 if kind == "differential" else 1
        self.r1, self.r2, self.pb = (rnd(H, seed=seed + i, std=s).abs() + lo for i, (s, lo) in enumerate(((0.5, 0.2), (1.0, 0.1), (1.0, -1.0))))
        self.lam, self.mix, self.eps, self.n, self.sharp = 0.7, 0.3, 1e-3, n, sharp

    def weights(self):
        from triton_distributed_b200 import ops

        if self.kind == "sigmoid":
            return ops.SigmoidWeights(ops.distance_table(self.r1, self.r2, self.pb, self.n).to(DEV))
        return ops.DifferentialWeights(self.lam, 1 - self.mix, self.eps, self.dv)

    def scale(self, dk):
        return self.sharp * 1.3 * dk ** -0.5

    def want(self, q, k, v, gate, scale):
        """q [H, maps, dk] of the newest position over k [n, G, maps, dk], v [n, G, dv] (oldest first)."""
        n, G = k.shape[:2]
        dist = torch.arange(n - 1, -1, -1, dtype=torch.float64)
        out = []
        for a in range(self.H):
            g = a // (self.H // G)
            if self.kind == "sigmoid":
                o = oracle.sigmoid_weights(q[a, 0], k[:, g, 0], dist, scale, self.r1[a].double(), self.r2[a].double(), self.pb[a].double()) @ v[:, g]
            else:
                o = oracle.combine_maps(*(oracle.softmax((k[:, g, m] @ q[a, m]) * scale) @ v[:, g] for m in (0, 1)), self.lam, self.mix, self.eps)
            out.append(o if gate is None else o * oracle.sigmoid(gate[a]))
        return torch.stack(out)


def loud(k, q, places, share):
    """Makes the keys k [n, G, maps, dk] at ``places`` answer the query q [H, maps, dk] above the others."""
    for i, j in enumerate(places):
        if 0 <= j < k.shape[0]:
            for g in range(k.shape[1]):
                k[j, g] = 0.3 * k[j, g] + (1.0 + 0.4 * (i % 2)) * q[g * share + i % share]
    return k


KINDS = ["sigmoid", "differential"]
SHAPES = [(4, 2, 64, 64), (6, 1, 64, 128), (18, 1, 128, 64), (2, 2, 128, 128)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,dk,dv", SHAPES + [(3, 1, 40, 24), (2, 1, 200, 300), (2, 2, 520, 40)])
@pytest.mark.parametrize("R", [1, 7, 64, 150, 300])
def test_window_decode(rt, kind, H, G, dk, dv, R):
    """Rings before, at and long after they are full; keys at the window's edges, beside block borders and one that has been overwritten."""
    from triton_distributed_b200 import ops

    dt = torch.bfloat16
    lens = [1, 2, R - 1, R, R + 1, 2 * R + 3, 5 * R + R // 2, 63, 64, 65, 129]
    lens = [n for n in lens if n >= 1]
    B, share = len(lens), H // G
    h = Heads(kind, H, dv, 3, R)
    m, scale = h.maps, h.scale(dk)
    slots = torch.randperm(B + 2, generator=torch.Generator().manual_seed(1))[:B].to(torch.int32)
    q, gate = rnd(B, H, m, dk, seed=1).to(dt), rnd(B, H + 3, seed=2).to(dt)
    k, v = torch.full((B + 2, R, G, m, dk), 9.0).to(dt), torch.full((B + 2, R, G, dv), 9.0).to(dt)
    want = []
    for b, n in enumerate(lens):
        lo = max(0, n - R)
        kk = loud(rnd(n - lo, G, m, dk, seed=10 + b), q[b].float(), sorted({0, 1, 62, 63, 64, 65, n - lo - 1}), share).to(dt)
        vv = rnd(n - lo, G, dv, seed=40 + b).to(dt)
        at = torch.arange(lo, n) % R
        k[slots[b], at], v[slots[b], at] = kk, vv
        want.append(h.want(q[b].double(), kk.double(), vv.double(), gate[b].double(), scale))
    want = torch.stack(want)
    qd, kd, vd = dev(q.reshape(B, H * m, dk)), dev(k.reshape(B + 2, R, G * m, dk)), dev(v)
    pos, wide = i64([n - 1 for n in lens]), dev(gate)
    if dk in ops.WINDOW_DIMS and dv in ops.WINDOW_DIMS:
        for splits in (-1, 1, 2, 5):
            for _ in range(2):                                  # the counters are left clean
                close(ops.window_attention_decode(qd, kd, vd, h.weights(), scale, wide, dev(slots), pos, splits), want, dt)
    seen = (i64((slots.long() * R).tolist()), i32([min(n, R) for n in lens]), i32([(n - 1) % R for n in lens]))
    close(ops.window_attention_simple(qd, kd, vd, h.weights(), scale, wide, *seen), want, dt)
    f = lambda t: t.float()   # noqa: E731
    close(ops.window_attention_simple(f(qd), f(kd), f(vd), h.weights(), scale, f(wide), *seen), want, torch.float32)


# (lengths, start positions) of the portions of a step
STEPS = [([150], [0]), ([300, 1], [0, 0]), ([1, 130, 64, 257], [0, 0, 0, 0]), ([2, 140, 7, 1], [63, 500, 210, 0])]
# every window with every step for the largest heads, some of them for the other sizes
PROMPTS = [(SHAPES[-1], w, s) for w in (0, 1, 2, 63, 65, 129, 200, 700) for s in STEPS] + \
    [(shape, w, s) for shape in SHAPES[:-1] for w in (0, 1, 65, 129, 700) for s in STEPS if len(s[0]) != 2]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("shape,window,step", PROMPTS)
def test_window_prompts(rt, kind, shape, window, step):
    """Prompts and portions of prompts; keys just inside and outside the window of some queries, at block and tile edges stand out."""
    from triton_distributed_b200 import ops

    (H, G, dk, dv), (lens, starts) = shape, step
    dt, T = torch.bfloat16, sum(lens)
    h = Heads(kind, H, dv, 3, window or 1000)
    m, scale, share = h.maps, h.scale(dk), H // G
    cu = bounds(lens)
    q, gate = rnd(T, H, m, dk, seed=1).to(dt), rnd(T, H + 1, seed=2).to(dt)
    ks, vs, shift, want, at = [], [], [], [], 0
    row0, n_keys = [], []
    pick = torch.Generator().manual_seed(7)
    for b, (n, s) in enumerate(zip(lens, starts)):
        first = max(0, s - window + 1) if window else 0
        kk, vv = rnd(s + n - first, G, m, dk, seed=10 + b), rnd(s + n - first, G, dv, seed=40 + b).to(dt)
        # a few queries, each with a loud key of its own at the edge of what it sees
        for i in sorted({0, n - 1, n // 2, 127, 128} & set(range(n))):
            j = s + i - (window or s + i + 1) + int(torch.randint(0, 2, (1,), generator=pick))
            kk = loud(kk, q[cu[b] + i].float(), [j - first, min(64, s) - first], share)
        kk = kk.to(dt)
        for i in range(n):
            lo = max(0, s + i - window + 1) - first if window else 0
            hi = s + i + 1 - first
            row0.append(at + lo)
            n_keys.append(hi - lo)
            want.append(h.want(q[cu[b] + i].double(), kk[lo:hi].double(), vv[lo:hi].double(), gate[cu[b] + i].double(), scale) if i % 3 == 0 or i > n - 4 or 120 < i < 136
                        else torch.full((H, dv), float("nan"), dtype=torch.float64))
        ks.append(kk)
        vs.append(vv)
        shift.append(at - first)
        at += s + n - first
    want = torch.stack(want)
    rows = torch.isfinite(want[:, 0, 0])
    qd, kd, vd = dev(q.reshape(T, H * m, dk)), dev(torch.cat(ks).reshape(-1, G * m, dk)), dev(torch.cat(vs))
    got = ops.window_attention_prompt(qd, kd, vd, h.weights(), scale, dev(gate), i32(cu), i32(starts), i32(shift), max(lens), window)
    ops.check_attention_errors()
    assert torch.isfinite(got).all()
    close(got[dev(rows)], want[rows], dt)
    seen = (i64(row0), i32(n_keys), i32([n - 1 for n in n_keys]))
    f = lambda t: t.float()   # noqa: E731
    simple = ops.window_attention_simple(f(qd), f(kd), f(vd), h.weights(), scale, f(dev(gate)), *seen)
    close(simple[dev(rows)], want[rows], torch.float32)
    close(got, simple.double().cpu(), dt)                        # all rows
    if kind == "differential":                                   # nothing besides positions, lengths and the window decides
        no_gate = ops.window_attention_prompt(qd, kd, vd, h.weights(), scale, None, i32(cu), i32(starts), i32(shift), max(lens), window)
        close(no_gate * torch.sigmoid(dev(gate).float()[:, :H, None]), simple.double().cpu(), dt)


@pytest.mark.parametrize("kind", KINDS)
def test_window_attention_of_large_scores(rt, kind):
    """Scores of tens: weights that are 0 or 1, maxima that rise block after block."""
    from triton_distributed_b200 import ops

    dt, T, H, G, dk, dv, window = torch.bfloat16, 333, 2, 1, 64, 64, 150
    h = Heads(kind, H, dv, 3, window, sharp=6.0)
    m, scale = h.maps, h.scale(dk)
    q, v = rnd(T, H, m, dk, seed=1).to(dt), rnd(T, G, dv, seed=2).to(dt)
    k = (rnd(T, G, m, dk, seed=3) * torch.linspace(0.1, 3.0, T).reshape(-1, 1, 1, 1)).to(dt)
    got = ops.window_attention_prompt(dev(q.reshape(T, -1, dk)), dev(k.reshape(T, -1, dk)), dev(v), h.weights(), scale, None, i32([0, T]), i32([0]), i32([0]), T, window)
    n = [min(t + 1, window) for t in range(T)]
    want = torch.stack([h.want(q[t].double(), k[t + 1 - n[t]:t + 1].double(), v[t + 1 - n[t]:t + 1].double(), None, scale) for t in range(T)])
    close(got, want, dt, 1.5)
    ops.check_attention_errors()


# ------------------------------------------------------------------ state space layer
class Space:
    """One random state space layer: padded inputs for the kernels, and the oracle's outputs and states.  ``quiet``: tokens that hardly
    write and hardly decay."""

    def __init__(self, H, G, N, dv, taps, lens, seed=0, dtype=torch.bfloat16, quiet=None):
        from triton_distributed_b200 import ops
        from triton_distributed_b200.parallel.tp_delta import pad_key_dim
        from triton_distributed_b200.parallel.tp_gla import pad16
        from triton_distributed_b200.parallel.tp_layer import pad_heads

        self.H, self.G, self.N, self.dv, self.taps, self.lens, self.dtype = H, G, N, dv, taps, lens, dtype
        self.Np, self.Dv = pad_key_dim(N), pad16(dv)
        T = sum(lens)
        parts = ((H, dv, self.Dv), (G, N, self.Np), (G, N, self.Np))
        raw = [rnd(T, n * d, seed=seed + i).to(dtype) for i, (n, d, _) in enumerate(parts)]
        conv_w = [rnd(n * d, taps, seed=seed + 4 + i, std=1.5 * taps ** -0.5) for i, (n, d, _) in enumerate(parts)]
        conv_b = [rnd(n * d, seed=seed + 8 + i, std=0.4) for i, (n, d, _) in enumerate(parts)]
        dt_in = rnd(T, H, seed=seed + 12, std=1.5).to(dtype)
        a_log, dt_bias, skip = 0.7 * rnd(H, seed=seed + 13), rnd(H, seed=seed + 14) - 1.0, rnd(H, seed=seed + 15)
        if quiet:
            a_log = torch.full((H,), -3.0)
            dt_in[quiet[0]:quiet[1]] = -9.0
        self.channels = H * self.Dv + 2 * G * self.Np
        z = [pad_heads(x.T, *p).T for x, p in zip(raw, parts)] + [torch.ones(T, 8, dtype=dtype), dt_in]
        self.z = torch.cat(z + [torch.zeros(T, -(-H // 8) * 8 - H, dtype=dtype)], dim=1)
        self.dt_col = self.channels + 8
        self.w = ops.SsdWeights(*(dev(t) for t in (torch.cat([pad_heads(x, *p) for x, p in zip(conv_w, parts)]),
                                                   torch.cat([pad_heads(x, *p) for x, p in zip(conv_b, parts)]), a_log, dt_bias, skip)))
        cu, outs, self.states = bounds(lens), [], []
        d = lambda t: t.double()   # noqa: E731
        for lo, hi in zip(cu, cu[1:]):
            x, B, C = (oracle.silu(oracle.short_conv(d(r[lo:hi]), d(w), d(b))) for r, w, b in zip(raw, conv_w, conv_b))
            x, (B, C) = x.reshape(-1, H, dv), (t.reshape(-1, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
            dt = oracle.softplus(d(dt_in[lo:hi]) + d(dt_bias))
            S, y = torch.zeros(H, N, dv, dtype=torch.float64), []
            for t in range(hi - lo):
                S, o = oracle.ssd_step(S, x[t], B[t], C[t], dt[t], torch.exp(d(a_log)), d(skip))
                y.append(o)
            self.states.append(S)
            outs.append(torch.stack(y))
        self.want, self.cu = torch.cat(outs), cu
        # slots in another order, and rows that hold garbage: nothing of it may be read
        n = len(lens)
        self.slots = torch.randperm(n + 2, generator=torch.Generator().manual_seed(seed))[:n].to(torch.int32)
        self.state = torch.full((n + 2, H, self.Np, self.Dv), float("nan"), device=DEV)
        self.ring = torch.full((n + 2, taps, self.channels), float("nan"), dtype=dtype, device=DEV)
        self.out = torch.full((T, H, dv), float("nan"))

    def run(self, parts, impl="auto"):
        """``parts``: list of (sequence, first token, end); one call."""
        from triton_distributed_b200 import ops

        rows = torch.cat([torch.arange(self.cu[s] + lo, self.cu[s] + hi) for s, lo, hi in parts])
        seqs, cu = [s for s, _, _ in parts], bounds([hi - lo for _, lo, hi in parts])
        wide = torch.cat([torch.zeros(len(rows), 16, dtype=self.dtype), self.z[rows]], dim=1).to(DEV)[:, 16:]
        decode = impl == "decode" or (impl == "auto" and cu[-1] == len(parts))
        got = ops.state_space(wide, self.dt_col, self.w, self.state, self.ring, dev(self.slots[seqs]), i64([lo for _, lo, _ in parts]), None if decode else i32(cu),
                              self.G, ops.gla_chunk_tables(cu, DEV), impl).reshape(len(rows), self.H, self.Dv)
        assert self.Dv == self.dv or float(got[..., self.dv:].abs().max()) == 0
        self.out[rows] = got[..., :self.dv].float().cpu()

    def check(self, scale=1.0):
        close(self.out, self.want, self.dtype, scale)
        for s, S in enumerate(self.states):
            close(self.state[self.slots[s].item()][:, :self.N, :self.dv], S, self.dtype, scale)


SPACES = [(4, 2, 128, 64, 4), (6, 3, 40, 72, 3), (2, 2, 64, 64, 1), (2, 1, 256, 250, 2), (3, 3, 10, 20, 7), (16, 1, 100, 16, 4), (1, 1, 24, 128, 12), (24, 2, 16, 32, 4)]


@pytest.mark.parametrize("shape", SPACES)
@pytest.mark.parametrize("impl,dtype", [("chunk", torch.bfloat16), ("recurrent", torch.bfloat16), ("recurrent", torch.float32)])
def test_state_space_prompts(rt, shape, impl, dtype):
    r = Space(*shape, lens=[130, 1, 64, 65, 200], dtype=dtype)
    r.run([(s, 0, n) for s, n in enumerate(r.lens)], impl)
    r.check()


def test_state_space_of_many_chunks(rt):
    """Enough chunks for several heads of a group to share a CTA."""
    r = Space(8, 2, 32, 16, 4, lens=[9600, 100])
    r.run([(s, 0, n) for s, n in enumerate(r.lens)], "chunk")
    r.check()


@pytest.mark.parametrize("shape", SPACES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_state_space_portions_and_decoding(rt, shape, dtype):
    """Portions down to one and two tokens, decode steps, and prompts of other sequences beside them continue where the last call left
    state and convolutions."""
    r = Space(*shape, lens=[90, 20, 75], dtype=dtype)
    r.run([(0, 0, 5), (1, 0, 1), (2, 0, 64)])
    for t in range(5, 12):
        r.run([(0, t, t + 1)])
    r.run([(1, 1, 3), (0, 12, 13), (2, 64, 66)])
    r.run([(1, 3, 4), (0, 13, 14)])
    r.run([(0, 14, 80), (2, 66, 75)])
    for t in range(4, 14):
        r.run([(1, t, t + 1), (0, t + 76, t + 77)], "decode")
    r.run([(1, 14, 20)])
    r.check()


def test_state_space_decode_is_repeatable(rt):
    """A step that runs again at the same position (as graph capture does) leaves the convolutions' inputs as they were."""
    r = Space(4, 2, 32, 48, 4, lens=[12])
    r.run([(0, 0, 9)])
    state, ring = r.state.clone(), None
    for _ in range(3):
        r.state.copy_(state)
        r.run([(0, 9, 10)])
        slot = r.slots[0].item()
        assert ring is None or torch.equal(ring, r.ring[slot])
        ring = r.ring[slot].clone()
    r.run([(0, 10, 11)])
    r.run([(0, 11, 12)])
    r.check()


def test_state_space_keeps_what_it_wrote_long_ago(rt):
    """Hardly any decay: what the first tokens wrote is read more than ten chunks later, in all forms."""
    for dtype, impl in ((torch.bfloat16, "chunk"), (torch.bfloat16, "recurrent"), (torch.float32, "recurrent")):
        r = Space(2, 1, 32, 32, 2, [700], 3, dtype, quiet=(3, 690))
        r.run([(0, 0, 700)], impl)
        r.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv,pad,parts", [(8, 64, 64, 1), (8, 64, 64, 8), (6, 20, 32, 3), (6, 20, 32, 4), (3, 16, 16, 12), (4, 24, 24, 3), (128, 64, 64, 2), (128, 64, 64, 1),
                                            (160, 64, 64, 1), (1, 8, 8, 1)])
def test_gated_group_norm(rt, dtype, H, dv, pad, parts):
    from triton_distributed_b200 import ops

    T, eps = 5, 1e-3
    y, g, w = rnd(T, H, dv).to(dtype), rnd(T, H, dv, seed=1, std=2.0).to(dtype), 1 + 0.3 * rnd(H, dv, seed=2)
    p = lambda t: torch.nn.functional.pad(t, (0, pad - dv)).reshape(*t.shape[:-2], H * pad)   # noqa: E731
    gate = torch.cat([p(g), torch.ones(T, 24, dtype=dtype)], dim=1)
    out = ops.gated_group_norm(dev(p(y)), dev(gate), dev(p(w)), H, dv, parts, eps).reshape(T, H, pad)
    assert pad == dv or float(out[..., dv:].abs().max()) == 0
    want = oracle.gated_group_norm(y.double().reshape(T, -1), g.double().reshape(T, -1), parts, w.double().reshape(-1), eps)
    close(out[..., :dv].reshape(T, -1), want, dtype)


# ------------------------------------------------------------------ whole models
# sizes of the tensor-core kernels, windows longer than a tile, a shared layer of every kind
WIDE = cases.config([("attention", cases.attn(8, 2, 128, 128, 70), 136), ("mamba2", cases.mamba(4, 2, 128, 96, 4, 2), 72),
                     ("attention_2", cases.diff(4, 4, 40, 64, 150, 40, 0.5, factor=4.0, original=96, low=1.0, high=4.0), 264), 0, 1, 2,
                     ("attention_2", cases.diff(2, 1, 160, 200, 33, 160, 0.2), None), ("attention", cases.attn(4, 1, 100, 136, 129), None)], width=200, vocab=203, eps=1e-4, scale=0.8)
MODELS = {"mixed": cases.MIXED, "plain": cases.PLAIN, "wide": WIDE}
_MADE = {}


@pytest.fixture(params=[(n, t) for n in sorted(MODELS) for t in DTYPES], ids=lambda p: f"{p[0]}-{'bf16' if p[1] == torch.bfloat16 else 'fp32'}")
def model(request, rt, tmp_path_factory):
    """(dtype, directory, config, weights, tokens, the oracle's logits)."""
    name, dtype = request.param
    if request.param not in _MADE:
        cfg = MODELS[name]
        w = cases.weights(cfg, seed=3, sharp=1.5, gain=0.5)
        toks = cases.prompt(cfg, 301 if name == "wide" else 157)
        _MADE[request.param] = (dtype, str(cases.write(tmp_path_factory.mktemp(name), cfg, w)), cfg, w, toks, oracle.forward(cfg, w, toks))
    return _MADE[request.param]


def test_prompts_portions_and_decoding(model):
    dtype, d, _, _, toks, want = model
    n = len(toks)
    eng = cases.engine(d, dtype, max_length=400)
    for sizes in ([n], [n - 60, 1], [2], [97, 64, 3, 30], [150, 1, 1, 100]):
        assert cases.rel(cases.run_portions(eng, "r", toks, sizes), want) < TOL[dtype], sizes
    eng.check_errors()


def test_rings_shorter_than_the_window(model):
    """A cache that holds no more tokens than the request has."""
    dtype, d, _, _, toks, want = model
    eng = cases.engine(d, dtype, max_length=60)
    for sizes in ([60], [40, 1], [1]):
        assert cases.rel(cases.run_portions(eng, "r", toks[:60], sizes), want[:60]) < TOL[dtype], sizes


def test_unequal_batch_and_reused_slots(model):
    dtype, d, cfg, w, toks, want = model
    eng = cases.engine(d, dtype, max_length=400)
    other = {i: cases.prompt(cfg, m, i) for i, m in ((1, 1), (2, 66), (3, 29))}
    ref = {i: oracle.forward(cfg, w, p) for i, p in other.items()}
    n = len(toks)
    got = {i: [] for i in (0, 1, 2, 3)}
    seqs, refs = {0: toks, **other}, {0: want, **ref}

    def step(parts):
        z = eng.step([(i, seqs[i][lo:hi], list(range(hi - lo))) for i, lo, hi in parts])
        for i, lo, hi in parts:
            got[i].append(z[:hi - lo])
            z = z[hi - lo:]

    step([(1, 0, 1), (2, 0, 50), (0, 0, n - 40)])
    eng.end([1])
    for k in range(16):
        step([(2, 50 + k, 51 + k), (0, n - 40 + k, n - 39 + k)])
    eng.end([2])
    step([(0, n - 24, n - 23), (3, 0, 20)])              # a new request in a used slot, beside a decoding one
    for k in range(9):
        step([(3, 20 + k, 21 + k), (0, n - 23 + k, n - 22 + k)])
    step([(0, n - 14, n)])
    for i in got:
        assert cases.rel(torch.cat(got[i]), refs[i]) < TOL[dtype], i


def test_residual_stream_after_every_layer(model):
    dtype, d, cfg, w, toks, _ = model
    eng = cases.engine(d, dtype, max_length=400)
    streams, ref = [], []
    toks = toks[:50]
    want = oracle.forward(cfg, w, toks, ref)
    cache = eng.model.new_cache(1, 64)
    got = eng.model.forward_step(torch.tensor(toks, device=DEV), cache.plan([0], [len(toks)]), None, False, streams)
    assert len(streams) == len(ref)
    for a, b in zip(streams, ref):
        close(a, b, dtype, 3.0)
    assert cases.rel(got, want) < TOL[dtype]


def test_wide_decode_batches(rt, tmp_path):
    """More sequences than the fused decode projections take."""
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=5, sharp=1.5)
    d = cases.write(tmp_path, cfg, w)
    lens = [5 + 3 * (i % 7) for i in range(21)]
    prompts = [cases.prompt(cfg, n + 3, i) for i, n in enumerate(lens)]
    for dtype in DTYPES:
        eng = cases.engine(d, dtype, max_length=64)
        eng.step([(i, p[:n], []) for i, (p, n) in enumerate(zip(prompts, lens))])
        rows = [eng.step([(i, [p[n + k]], [0]) for i, (p, n) in enumerate(zip(prompts, lens))]) for k in range(3)]
        for i in range(0, 21, 4):
            want = oracle.forward(cfg, w, prompts[i])[lens[i]:]
            assert cases.rel(torch.stack([r[i] for r in rows]), want) < TOL[dtype], i


def test_greedy_generation_with_cuda_graph(rt, tmp_path):
    """Generation through serve() (graph-replayed decode steps) equals the oracle's."""
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=3, sharp=1.5)
    d = cases.write(tmp_path, cfg, w)
    prompts = [cases.prompt(cfg, 22, s) for s in range(3)]
    want = [cases.greedy(cfg, w, p, 8)[0] for p in prompts]
    for graph in (True, False):
        eng = cases.engine(d, torch.float32, max_length=64)
        eng.no_graph = not graph
        assert eng.serve(torch.tensor(prompts), 8).tolist() == want
    lens = [22, 5, 1]
    short = [cases.greedy(cfg, w, p[:n], 5)[0] for p, n in zip(prompts, lens)]
    assert eng.serve(torch.tensor(prompts), 5, seq_lens=lens).tolist() == short
    # bf16 generates what its own steps say, position by position
    eng = cases.engine(d, torch.bfloat16, max_length=64)
    eng.keep_logits = True
    for _ in range(2):                                    # the second call reuses cache and states
        out = eng.serve(torch.tensor(prompts), 8)
        full = torch.cat([torch.tensor(prompts), out.cpu()], dim=1).tolist()
        for b, toks in enumerate(full):
            ref = oracle.forward(cfg, w, toks[:-1])[21:]
            assert cases.rel(torch.stack([z[b] for z in eng.step_logits]), ref) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(rt, tmp_path, dtype):
    cfg = cases.config([("mamba2", cases.mamba(2, 1, 16, 8, 3, 1), 24), ("attention", cases.attn(3, 1, 16, 16, 20), None), ("attention_2", cases.diff(2, 2, 8, 16, 33, 8, **cases.BAND), 16), 1, 0],
                       32, 64, scale=1.5)
    w = cases.weights(cfg, seed=4, sharp=1.5)
    toks = cases.prompt(cfg, 300)
    eng = cases.engine(cases.write(tmp_path, cfg, w), dtype, max_length=300)
    assert cases.rel(cases.run_portions(eng, 0, toks, [1]), oracle.forward(cfg, w, toks)) < TOL[dtype]


def test_trace_runner_program(rt, tmp_path):
    cfg = cases.MIXED
    w = cases.weights(cfg, seed=1)
    d = cases.write(tmp_path, cfg, w)
    toks = cases.prompt(cfg, 50)
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:49], "want": [0, 48]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[49:], "want": [0]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out), "--max-tokens", "60"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300,
                       env={**os.environ, "PATH": os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"]})
    assert r.returncode == 0, r.stderr[-2000:]
    got = torch.cat([torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, 101) for n in (0, 1)])
    assert cases.rel(got, oracle.forward(cfg, w, toks)[[0, 48, 49]]) < TOL[torch.float32]
