"""Tazitar on one GPU: every kernel alone and the whole model (bf16 and fp32) against the plain oracle on the CPU."""
import json
import os
import subprocess
import sys

import pytest
import torch

import tazitar_cases as cases
import tazitar_oracle as oracle

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


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def bounds(lens):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return cu


# ------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,W,real", [(1, 72, 67), (2, 256, 256), (3, 64, 60), (4, 4096, 4090), (7, 136, 136), (16, 80, 75)])
def test_hyper_step(rt, dtype, S, W, real):
    from triton_distributed_b200 import ops

    T, V, eps = 5, 11, 1e-3
    mask = (torch.arange(W) < real).float()
    x0, table = rnd(T, S, W) * mask, (rnd(V, W, seed=1) * mask).to(dtype)
    y, y2 = ((rnd(T, W, seed=i) * mask).to(dtype) for i in (2, 3))
    wa, wb, wn = ((1 + 0.3 * rnd(W, seed=i)) * mask for i in (4, 5, 6))
    P = {"in": rnd(S, seed=7), "out": rnd(S, seed=8), "mix": rnd(S, S, seed=9)}
    dev = lambda t: None if t is None else t.to(DEV)   # noqa: E731
    hc = ops.HyperWeights(dev(P["in"]), dev(P["out"]), dev(P["mix"]))
    nxt = (dev(rnd(S, seed=10)), dev(wn))
    Pd = {n: t.double() for n, t in P.items()}

    def after(x, out):
        return oracle.hyper(x.double().transpose(0, 1), Pd, "", lambda u: out).transpose(0, 1)

    def normed(x):
        return oracle.rms(torch.einsum("s,tsw->tw", rnd(S, seed=10).double(), x.double())[:, :real], eps, wn[:real].double())

    a, b = y.double()[:, :real], y2.double()[:, :real]
    both = torch.zeros(T, W, dtype=torch.float64)
    both[:, :real] = 0.5 * (oracle.rms(a, eps, wa[:real].double()) + oracle.rms(b, eps, wb[:real].double()))
    for sub, out in ((ops.SublayerOutput(dev(y)), y.double()), (ops.SublayerOutput(dev(y), dev(y2), dev(wa), dev(wb)), both)):
        x = dev(x0)
        h = ops.hyper_step(x, (hc, sub), nxt, real, eps, dtype)
        close(x, after(x0, out), torch.float32)
        close(h[:, :real], normed(after(x0, out)), dtype)
        # some rows only: the streams stay as they are
        x, rows = dev(x0), torch.tensor([4, 0, 4])
        h = ops.hyper_step(x, (hc, sub), nxt, real, eps, dtype, dev(rows))
        assert torch.equal(x.cpu(), x0)
        close(h[:, :real], normed(after(x0, out))[rows], dtype)
        # nothing to norm
        assert ops.hyper_step(x, (hc, sub), None, real, eps, dtype) is None
        close(x, after(x0, out), torch.float32)
    # no sublayer behind it
    x = dev(x0)
    close(ops.hyper_step(x, None, nxt, real, eps, dtype)[:, :real], normed(x0), dtype)
    assert torch.equal(x.cpu(), x0)
    # the start of a model
    ids = torch.tensor([10, 0, 3, 3, 7])
    x = torch.full((T, S, W), float("nan"), device=DEV)
    h = ops.hyper_step(x, None, nxt, real, eps, dtype, start=(dev(ids), dev(table)))
    start = table.double()[ids].unsqueeze(1).expand(T, S, W)
    assert torch.equal(x.cpu().double(), start)
    close(h[:, :real], normed(start), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_activations(rt, dtype):
    from triton_distributed_b200 import ops

    x = rnd(7, 176, std=3.0).to(dtype)
    g, u = x.double()[:, :88], x.double()[:, 88:]
    close(ops.gated_act(x.to(DEV), "gelu"), oracle.gelu_tanh(g) * u, dtype)
    close(ops.gated_act(x.to(DEV), "silu"), oracle.silu(g) * u, dtype)
    if dtype == torch.bfloat16:
        w = rnd(136, 88, seed=1, std=88 ** -0.5).to(dtype)
        for n in (1, 3, 7):
            for act, f in (("gelu", oracle.gelu_tanh), ("silu", oracle.silu)):
                close(ops.gemv_fused(x[:n].to(DEV), w.to(DEV), silu_mul=True, act=act), (f(g) * u)[:n] @ w.double().T, dtype)


# ------------------------------------------------------------------ queries and keys
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,G,D,dim,turn", [(1, 3, 1, 64, 48, 48), (5, 2, 2, 64, 64, 16), (17, 4, 2, 128, 100, 34), (3, 2, 1, 256, 200, 200), (2, 1, 1, 512, 300, 2)])
@pytest.mark.parametrize("interleaved,norm,unit,yarn", [(False, True, False, False), (True, False, True, True), (False, False, True, False), (True, True, True, True)])
def test_head_prep(rt, dtype, T, H, G, D, dim, turn, interleaved, norm, unit, yarn):
    from triton_distributed_b200 import ops

    eps, far = 1e-3, 6000
    q, k, v = rnd(T, H, dim).to(dtype), rnd(T, G, dim, seed=1).to(dtype), rnd(T, G, dim, seed=2).to(dtype)
    qw, kw = 1 + 0.3 * rnd(dim, seed=3), 1 + 0.3 * rnd(dim, seed=4)
    pos = torch.randint(0, far, (T,), generator=torch.Generator().manual_seed(5))
    pos[0] = far - 1
    r = cases.rot(turn, 300.0, **(dict(factor=3.0, original=512, fast=16.0, slow=1.0) if yarn else {}))
    padded = [torch.nn.functional.pad(x, (0, D - dim)).reshape(T, -1) for x in (q, k, v)]
    z = torch.cat(padded + [torch.ones(T, 8, dtype=dtype)], dim=1).to(DEV)
    rows = torch.randperm(T + 3, generator=torch.Generator().manual_seed(6))[:T]
    kc, vc = (torch.zeros(T + 3, G, D, dtype=dtype, device=DEV) for _ in range(2))
    pad = lambda w: torch.nn.functional.pad(w, (0, D - dim)).to(DEV) if norm else None   # noqa: E731
    table = ops.rope_table(300.0, turn, turn, far, DEV, ops.YarnScaling.from_json(r.get("scaling")))
    got = ops.head_prep(z, H, G, D, dim, pad(qw), pad(kw), unit, eps, table, turn, interleaved, pos.to(DEV), kc, vc, rows.to(DEV))

    def want(x, w):
        x = x.double()
        if norm:
            x = oracle.rms(x, eps, w.double())
        x = torch.stack([oracle.rotate(x[t], int(pos[t]), r, interleaved) for t in range(T)])
        return oracle.rms(x, eps) if unit else x

    close(got[..., :dim], want(q, qw), dtype)
    close(kc[rows.to(DEV)][..., :dim], want(k, kw), dtype)
    assert torch.equal(vc[rows.to(DEV)][..., :dim].cpu(), v)
    assert float(got[..., dim:].abs().max() if D > dim else 0) == 0 and float(kc[..., dim:].abs().max() if D > dim else 0) == 0
    rest = [i for i in range(T + 3) if i not in rows.tolist()]
    assert float(kc[rest].abs().max()) == 0 and float(vc[rest].abs().max()) == 0
    # a negative row is not stored
    kc.zero_()
    neg = rows.clone()
    neg[-1] = -1
    ops.head_prep(z, H, G, D, dim, pad(qw), pad(kw), unit, eps, table, turn, interleaved, pos.to(DEV), kc, vc, neg.to(DEV))
    assert float(kc[rows[-1]].abs().max()) == 0


# ------------------------------------------------------------------ attention: soft cap and sink
def _want_attention(q, k, v, mixer, sink):
    """q [H, D] of one query over k [n, G, D], v [n, G, D]."""
    H, G = q.shape[0], k.shape[1]
    return torch.stack([oracle.softmax(oracle.head_scores(q[a], k[:, a // (H // G)], mixer), None if sink is None else sink[a].double())
                        @ v[:, a // (H // G)] for a in range(H)])


def _loud_keys(n, G, D, q, loud, seed, dtype):
    """Keys [n, G, D]; those in ``loud`` are made to answer the queries above all others."""
    k = rnd(n, G, D, seed=seed)
    share = q.shape[0] // G
    for i, j in enumerate(loud):
        for g in range(G):
            k[j, g] = 0.3 * k[j, g] + (1.2 + 0.4 * (i % 2)) * q[g * share + i % share]
    return k.to(dtype)


# small scores (the series), scores around the cap and far beyond it
CAPS = [(0.0, 1.0), (50.0, 1.0), (3.0, 1.0), (0.7, 6.0)]


@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (6, 1, 128), (18, 1, 64), (2, 2, 256), (3, 1, 512)])
@pytest.mark.parametrize("cap,sharp", CAPS)
@pytest.mark.parametrize("sink", [None, "mixed"])
def test_decode_attention(rt, H, G, D, cap, sharp, sink):
    """Far keys, keys beside the borders of blocks and splits, and the first key that is not visible stand out."""
    from triton_distributed_b200 import ops

    dt, M = torch.bfloat16, 520
    lens = [1, 2, 63, 64, 65, 128, 129, 300, 512, 520]
    B = len(lens)
    mixer = {"scale": sharp * 1.6 * D ** -0.5, "softcap": cap or None}
    q = rnd(B, H, D, seed=2).to(dt)
    sk = None if sink is None else 2.0 + 2.0 * rnd(H, seed=3)
    slots = torch.randperm(B + 2, generator=torch.Generator().manual_seed(1))[:B]
    k, v = rnd(B + 2, M, G, D, seed=4).to(dt), rnd(B + 2, M, G, D, seed=5).to(dt)
    for b, n in enumerate(lens):
        k[slots[b]] = _loud_keys(M, G, D, q[b].float(), sorted({j for j in (0, 63, 64, 127, 128, n - 1, n) if j < M}), 10 + b, dt)
    want = torch.stack([_want_attention(q[b].double(), k[slots[b], :n].double(), v[slots[b], :n].double(), mixer, sk) for b, n in enumerate(lens)])
    s = None if sk is None else sk.to(DEV)
    if D in ops.TENSOR_CORE_DIMS:
        for splits in (-1, 1, 5, 40):
            got = ops.gqa_fwd_batch_decode(q.to(DEV), k.to(DEV), v.to(DEV), None, None, i32(lens), slots.to(torch.int32).unsqueeze(1).to(DEV), mixer["scale"], cap,
                                           kv_split=splits, sink=s)
            close(got, want, dt)
    simple = ops.attention_simple(q.to(DEV), k.to(DEV), v.to(DEV), (slots * M).to(DEV), i32(lens), s, mixer["scale"], cap)
    close(simple, want, dt)
    exact = ops.attention_simple(q.float().to(DEV), k.float().to(DEV), v.float().to(DEV), (slots * M).to(DEV), i32(lens), s, mixer["scale"], cap)
    close(exact, want, torch.float32)


@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (2, 1, 128), (2, 1, 256)])
@pytest.mark.parametrize("cap,sharp", CAPS)
@pytest.mark.parametrize("lens,starts", [([150], [0]), ([1, 130, 64], [0, 0, 0]), ([2, 140, 7], [63, 100, 210])])
def test_prompt_attention(rt, H, G, D, cap, sharp, lens, starts):
    """Prompts and portions of prompts over the cache, keys at block edges stand out."""
    from triton_distributed_b200 import ops

    dt, M, T, N = torch.bfloat16, 320, sum(lens), len(lens)
    mixer = {"scale": sharp * 1.6 * D ** -0.5, "softcap": cap or None}
    cu = bounds(lens)
    q, v = rnd(T, H, D).to(dt), rnd(N + 1, M, G, D, seed=1).to(dt)
    k = torch.zeros(N + 1, M, G, D, dtype=dt)
    pages = list(range(N, 0, -1))
    for b, (n, s) in enumerate(zip(lens, starts)):
        k[pages[b]] = _loud_keys(M, G, D, q[cu[b] + n // 2].float(), sorted({0, 63, 64, 127, 128, s, n + s - 1} & set(range(n + s))), 10 + b, dt)
    sink = 1.0 + 2.0 * rnd(H, seed=3)
    ends = [n + s for n, s in zip(lens, starts)]
    forms = ["mma", "sm100"] if D == 128 else ["mma"]
    for sk in (None, sink):
        want = torch.cat([torch.stack([_want_attention(q[cu[b] + i].double(), k[pages[b], :s + i + 1].double(), v[pages[b], :s + i + 1].double(), mixer, sk)
                                       for i in range(n)]) for b, (n, s) in enumerate(zip(lens, starts))])
        for impl in forms:
            got = ops.flash_attn_varlen(q.to(DEV), k.to(DEV), v.to(DEV), i32(pages).unsqueeze(1), i32(cu), i32(ends), max(lens), i32(starts), True, mixer["scale"],
                                        cap, max_kv_len=max(ends), impl=impl, sink=None if sk is None else sk.to(DEV))
            close(got, want, dt)
    ops.check_attention_errors()


def test_lse_is_that_of_the_keys(rt):
    from triton_distributed_b200 import ops

    q, k, v = (rnd(1, 20, 2, 128, seed=i).to(torch.bfloat16).to(DEV) for i in range(3))
    _, lse = ops.flash_attn_varlen(q[0], k, v, i32([[0]]), i32([0, 20]), i32([20]), 20, softcap=2.0, return_lse=True)
    _, ref = ops.attention_reference(q[0], k, v, i32([[0]]), i32([0, 20]), i32([20]), None, True, None, 2.0, True)
    assert (lse - ref).abs().max() < 1e-2
    with pytest.raises(ValueError, match="sink"):
        ops.gqa_fwd_batch_decode(q[0, :1], k, v, None, None, i32([20]), i32([[0]]), return_lse=True, sink=torch.zeros(2, device=DEV))


# ------------------------------------------------------------------ gated delta rule
class Rule:
    """One random delta rule: padded inputs for the kernels, and the oracle's outputs and states.  ``quiet``: tokens that write nothing."""

    def __init__(self, H, G, dk, dv, taps, lens, seed=0, dtype=torch.bfloat16, quiet=None):
        from triton_distributed_b200.parallel.tp_delta import pad_key_dim
        from triton_distributed_b200.parallel.tp_gla import pad16
        from triton_distributed_b200.parallel.tp_layer import pad_heads, pad_rows

        self.H, self.G, self.dk, self.dv, self.taps, self.lens, self.dtype = H, G, dk, dv, taps, lens, dtype
        self.Dk, self.Dv = pad_key_dim(dk), pad16(dv)
        T = sum(lens)
        pz = lambda x, n, d, to: pad_heads(x.T, n, d, to).T   # noqa: E731
        raw = {"q": rnd(T, G * dk, seed=seed), "k": rnd(T, G * dk, seed=seed + 1), "v": rnd(T, H * dv, seed=seed + 2), "g": rnd(T, H * dv, seed=seed + 3)}
        raw = {n: t.to(dtype) for n, t in raw.items()}
        dims = {"q": (G, dk, self.Dk), "k": (G, dk, self.Dk), "v": (H, dv, self.Dv), "g": (H, dv, self.Dv)}
        self.z = torch.cat([pz(raw[n], *dims[n]) for n in "qkvg"], dim=1)
        conv = {n: rnd(dims[n][0] * dims[n][1], taps, seed=seed + 4, std=1.5 * taps ** -0.5) for n in "qkv"}
        self.conv_w = torch.cat([pad_heads(conv[n], *dims[n]) for n in "qkv"])
        self.ab = rnd(T, 2 * H, seed=seed + 5, std=2.0)
        self.a_log, self.dt, norm = 0.7 * rnd(H, seed=seed + 6), rnd(H, seed=seed + 7) - 2.0, 1 + 0.3 * rnd(dv, seed=seed + 8)
        self.norm = pad_rows(norm, self.Dv)
        if quiet:                                            # nothing is written there, and hardly anything decays
            self.a_log = torch.full((H,), -9.0)
            self.ab[quiet[0]:quiet[1], H:] = -12.0
        # the oracle on every sequence; its projections are the identity
        cu, outs, self.states = bounds(lens), [], []
        for lo, hi in zip(cu, cu[1:]):
            x = {n: t[lo:hi].double() for n, t in raw.items()}
            q, k, v = (oracle.silu(oracle.short_conv(x[n], conv[n].double())) for n in "qkv")
            q, k = (oracle.unit(t.reshape(hi - lo, G, dk)).repeat_interleave(H // G, dim=1) for t in (q, k))
            a, b = self.ab[lo:hi, :H].double(), self.ab[lo:hi, H:].double()
            g, beta = torch.exp(-torch.exp(self.a_log.double()) * oracle.softplus(a + self.dt.double())), oracle.sigmoid(b)
            S, o = torch.zeros(H, dk, dv, dtype=torch.float64), []
            for t in range(hi - lo):
                S, y = oracle.delta_step(S, q[t] * dk ** -0.5, k[t], v[t].reshape(H, dv), g[t], beta[t])
                o.append(y)
            self.states.append(S)
            outs.append(oracle.rms(torch.stack(o), 1e-3, norm.double()) * oracle.silu(x["g"].reshape(hi - lo, H, dv)))
        self.want = torch.cat(outs)
        self.cu = cu
        # slots in another order, and rows that hold garbage: nothing of it may be read
        n = len(lens)
        self.slots = torch.randperm(n + 2, generator=torch.Generator().manual_seed(seed))[:n].to(torch.int32)
        self.state = torch.full((n + 2, H, self.Dk, self.Dv), float("nan"), device=DEV)
        self.ring = torch.full((n + 2, taps, self.conv_w.shape[0]), float("nan"), dtype=dtype, device=DEV)
        self.out = torch.full((T, H, self.dv), float("nan"))

    def run(self, parts, impl="auto"):
        """``parts``: list of (sequence, first token, end); one call."""
        from triton_distributed_b200 import ops

        rows = torch.cat([torch.arange(self.cu[s] + lo, self.cu[s] + hi) for s, lo, hi in parts])
        seqs = [s for s, _, _ in parts]
        cu = bounds([hi - lo for _, lo, hi in parts])
        wide = torch.cat([torch.zeros(len(rows), 16, dtype=self.dtype), self.z[rows]], dim=1).to(DEV)[:, 16:]
        d = lambda t: t.to(DEV)   # noqa: E731
        decode = impl == "decode" or (impl == "auto" and cu[-1] == len(parts))
        got = ops.gated_delta_rule(wide, d(self.ab[rows]), d(self.conv_w), d(self.a_log), d(self.dt), d(self.norm), self.state, self.ring, d(self.slots[seqs]),
                                   torch.tensor([lo for _, lo, _ in parts], device=DEV), None if decode else i32(cu), self.G, self.dv, self.dk ** -0.5, 1e-3,
                                   ops.gla_chunk_tables(cu, DEV), impl)
        got = got.reshape(len(rows), self.H, self.Dv)
        assert float(got[..., self.dv:].abs().max() if self.Dv > self.dv else 0) == 0
        self.out[rows] = got[..., :self.dv].float().cpu()

    def check(self, scale=1.0):
        close(self.out, self.want, self.dtype, scale)
        for s, S in enumerate(self.states):
            close(self.state[self.slots[s].item()][:, :self.dk, :self.dv], S, self.dtype, scale)


RULES = [(4, 2, 128, 128, 4), (6, 3, 40, 72, 3), (2, 2, 64, 64, 1), (2, 1, 256, 250, 2), (3, 3, 10, 20, 7), (4, 4, 96, 160, 4), (1, 1, 100, 16, 12)]


@pytest.mark.parametrize("shape", RULES)
@pytest.mark.parametrize("impl,dtype", [("chunk", torch.bfloat16), ("recurrent", torch.bfloat16), ("recurrent", torch.float32)])
def test_delta_rule_prompts(rt, shape, impl, dtype):
    r = Rule(*shape, lens=[130, 1, 64, 65, 200], dtype=dtype)
    r.run([(s, 0, n) for s, n in enumerate(r.lens)], impl)
    r.check()


@pytest.mark.parametrize("shape", RULES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_portions_and_decoding(rt, shape, dtype):
    """Portions down to one and two tokens, decode steps, and prompts of other sequences beside them continue where the last call left
    state and convolutions."""
    r = Rule(*shape, lens=[90, 20, 75], dtype=dtype)
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


def test_delta_rule_decode_is_repeatable(rt):
    """A step that runs again at the same position (as graph capture does) leaves the convolutions' inputs as they were."""
    r = Rule(4, 2, 32, 48, 4, lens=[12])
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


def test_delta_rule_keeps_what_it_wrote_long_ago(rt):
    """Hardly any decay: a value written in the first tokens is read back more than ten chunks later, in all forms."""
    for dtype, impl in ((torch.bfloat16, "chunk"), (torch.bfloat16, "recurrent"), (torch.float32, "recurrent")):
        r = Rule(2, 1, 32, 32, 2, [700], 3, dtype, quiet=(3, 690))
        assert float(r.states[0].abs().max()) > 0.1
        r.run([(0, 0, 700)], impl)
        r.check()


# ------------------------------------------------------------------ whole models
WIDE = cases.config([("attention", cases.attn(8, 2, 128, 128, 64, cap=8.0), 136), ("parallel", {"left": cases.attn(6, 2, 100, 72, 40, scale=0.1), "right": cases.delta(4, 2, 128, 96, 4)}, 72),
                     ("attention_2", cases.attn(4, 4, 40, 64, 40, factor=4.0, original=96, fast=8.0, slow=1.0), 264),
                     ("attention", cases.attn(2, 1, 160, 200, 160, cap=20.0), None)], width=200, vocab=203, eps=1e-4, streams=4, loop=(0, 2, 2))
MODELS = {"mixed": cases.MIXED, "plain": cases.PLAIN, "wide": WIDE}
_MADE = {}


@pytest.fixture(params=[(n, t) for n in sorted(MODELS) for t in DTYPES], ids=lambda p: f"{p[0]}-{'bf16' if p[1] == torch.bfloat16 else 'fp32'}")
def model(request, rt, tmp_path_factory):
    """(dtype, directory, config, weights, tokens, the oracle's logits); bf16 models do not amplify rounding much."""
    name, dtype = request.param
    if request.param not in _MADE:
        cfg = MODELS[name]
        w = cases.weights(cfg, seed=3, sharp=1.5, **(dict(uneven=0.5, gain=0.4) if dtype == torch.bfloat16 else {}))
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


def test_residual_streams_after_every_layer(model):
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
    cfg = cases.config([("parallel", {"left": cases.attn(2, 1, 16, 8, 8), "right": cases.delta(2, 1, 16, 8, 3)}, 24), ("attention", cases.attn(3, 1, 16, 16, 16, cap=4.0), None),
                        ("attention_2", cases.attn(2, 2, 8, 16, 8, **cases.YARN), 16)], 32, 64, streams=2, loop=(1, 3, 2))
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
