"""Lisenex on one GPU: every kernel alone and the whole model (bf16 and fp32) against the plain oracle on the CPU."""
import json
import os
import subprocess
import sys

import pytest
import torch

import lisenex_cases as cases
import lisenex_oracle as oracle

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


def pad8(n):
    return (n + 7) // 8 * 8


# ------------------------------------------------------------------ stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,real,rows", [(72, 67, 1), (256, 256, 3), (4096, 4096, 2)])
def test_parallel_add(rt, dtype, W, real, rows):
    from triton_distributed_b200 import ops

    T, E = 5, 4
    mask = (torch.arange(W) < real).float()
    mix, y, sh, hin = (rnd(n, W, seed=i) * mask for i, n in enumerate((T, T * rows, T, T)))
    x0, bias = rnd(T, W, seed=7) * mask, rnd(W, seed=8) * mask
    mix, sh, hin = (t.to(dtype) for t in (mix, sh, hin))
    w1, w2 = (1 + 0.2 * rnd(W, seed=9)) * mask, (1 + 0.2 * rnd(W, seed=10)) * mask
    ids = torch.arange(T * rows).reshape(T, rows).to(torch.int32) % (E + 2)          # ids E, E + 1: identity
    wts = torch.rand(T, rows)
    own = (ids < E).unsqueeze(-1)
    dev = lambda t: None if t is None else t.to(DEV)   # noqa: E731
    for ydt in {dtype, torch.float32}:
        yy = y.to(ydt)
        stale = yy.reshape(T, rows, W).clone()
        stale[~own.expand_as(stale)] = float("nan")                                  # rows of identity experts are never read
        pick = torch.where(own, yy.double().reshape(T, rows, W), wts.double().unsqueeze(-1) * hin.double().unsqueeze(1)).sum(1)
        full = mix.double() + pick + sh.double() + bias.double()
        ff = ops.FeedForward(dev(stale.reshape(T * rows, W)), rows, dev(ids), dev(wts), E, dev(hin), dev(sh), dev(bias))
        x = x0.to(DEV)
        close(ops.parallel_sum(x, dev(mix), ff), full, torch.float32)
        h1, h2 = ops.parallel_add(x, dev(mix), ff, dev(w1), dev(w2), real, 1e-4, dtype)
        close(x, x0.double() + full, torch.float32)
        norm = oracle.rms((x0.double() + full)[:, :real], 1e-4)
        close(h1[:, :real], norm * w1[:real].double(), dtype)
        close(h2[:, :real], norm * w2[:real].double(), dtype)
        # pieces left out: no mixer, no second norm, nothing at all, no norm
        x = x0.to(DEV)
        h1, h2 = ops.parallel_add(x, None, ops.FeedForward(dev(yy), rows), dev(w1), None, real, 1e-4, dtype)
        assert h2 is None
        close(x, x0.double() + yy.double().reshape(T, rows, W).sum(1), torch.float32)
        # another rank adds the identity experts
        ff.hin = None
        close(ops.parallel_sum(x, dev(mix), ff), full - torch.where(own, torch.zeros(1, dtype=torch.float64), wts.double().unsqueeze(-1)
                                                                     * hin.double().unsqueeze(1)).sum(1), torch.float32)
    x = x0.to(DEV)
    h1, h2 = ops.parallel_add(x, None, None, dev(w1), dev(w2), real, 1e-4, dtype)
    assert torch.equal(x.cpu(), x0)
    close(h2[:, :real], oracle.rms(x0[:, :real].double(), 1e-4, w2[:real].double()), dtype)
    assert ops.parallel_add(x, dev(mix), None, None, None, real, 1e-4, dtype) == (None, None)
    close(x, x0.double() + mix.double(), torch.float32)
    table = rnd(11, W, seed=4).to(dtype)
    ex, exb = ops.embed_stream(torch.tensor([10, 0, 3]).to(DEV), table.to(DEV), 0.3, copy=False)
    assert exb is None
    close(ex, table[[10, 0, 3]].double() * 0.3, torch.float32)


# ------------------------------------------------------------------ what surrounds the attention
def _table(base, r, n):
    from triton_distributed_b200 import ops
    return ops.rope_table(base, r, pad8(r), n, DEV)


def _padded_z(q, row, H, d, r, R):
    """q [T, H, d + r] and row [T, R + r] in the padded column layout (padding filled with zeros), and three more columns."""
    T = q.shape[0]
    zp = torch.zeros(T, H, pad8(d) + pad8(r))
    zp[:, :, :d], zp[:, :, pad8(d):pad8(d) + r] = q[:, :, :d], q[:, :, d:]
    rp = torch.zeros(T, pad8(R) + pad8(r))
    rp[:, :R], rp[:, pad8(R):pad8(R) + r] = row[:, :R], row[:, R:]
    return torch.cat([zp.reshape(T, -1), rp, torch.zeros(T, 8)], dim=1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,d,r,R", [(1, 3, 16, 8, 40), (5, 2, 20, 12, 36), (17, 4, 128, 64, 512), (40, 1, 9, 6, 72)])
def test_latent_rotate_and_absorb(rt, dtype, T, H, d, r, R):
    from triton_distributed_b200 import ops

    base, eps, far = 700.0, 1e-4, 5000
    q, row = rnd(T, H, d + r).to(dtype), rnd(T, R + r, seed=1, std=2.0).to(dtype)
    uk = rnd(H, d, R, seed=2, std=d ** -0.5).to(dtype)
    nw = 1 + 0.3 * rnd(R, seed=3)
    pos = torch.randint(0, far, (T,), generator=torch.Generator().manual_seed(4))
    pos[0] = far - 1
    z = _padded_z(q.float(), row.float(), H, d, r, R).to(dtype).to(DEV)
    ukt = torch.zeros(H, pad8(R), pad8(d), dtype=dtype)
    ukt[:, :R, :d] = uk.transpose(1, 2)
    nwp = torch.nn.functional.pad(nw, (0, pad8(R) - R)).to(DEV)
    c = oracle.rms(row[:, :R].double(), eps, nw.double())
    kr = torch.stack([oracle.rotate(row[t, R:].double(), int(pos[t]), base) for t in range(T)])
    qr = torch.stack([oracle.rotate(q[t, :, d:].double(), int(pos[t]), base) for t in range(T)])
    Wp = pad8(R) + pad8(r)
    rows, rows2 = torch.randperm(T + 3, generator=torch.Generator().manual_seed(5))[:T], torch.arange(T) + 1
    rows2[-1] = -1
    for form in ("absorb", "rotate"):
        home, ctx = torch.zeros(T + 3, Wp, dtype=dtype, device=DEV), torch.zeros(T + 1, Wp, dtype=dtype, device=DEV)
        zz = z.clone()
        if form == "absorb":
            qe = ops.latent_absorb(zz, ukt.to(DEV), pad8(r), nwp, R, eps, _table(base, r, far), pos.to(DEV), (home, rows.to(DEV)))
            assert torch.equal(zz, z)
            close(qe[..., :R], torch.einsum("hdr,thd->thr", uk.double(), q[..., :d].double()), dtype)
            got = qe[..., pad8(R):pad8(R) + r]
            shared = ops.latent_absorb(zz, ukt.to(DEV), pad8(r), None, R, eps, _table(base, r, far), pos.to(DEV))
            assert torch.equal(shared, qe)
        else:
            ops.latent_rotate(zz, H, pad8(d), pad8(r), nwp, pad8(R), R, eps, _table(base, r, far), pos.to(DEV), (home, rows.to(DEV)),
                              (ctx, rows2.to(DEV)))
            heads = zz[:, :H * (pad8(d) + pad8(r))].reshape(T, H, -1)
            assert torch.equal(heads[..., :d].cpu(), q[..., :d])
            got = heads[..., pad8(d):pad8(d) + r]
            assert torch.equal(ctx[1:T], home[rows.to(DEV)][:T - 1]) and float(ctx[0].abs().max()) == 0 and float(ctx[T:].abs().max()) == 0
        close(got, qr, dtype)
        close(home[rows.to(DEV)][:, :R], c, dtype)
        close(home[rows.to(DEV)][:, pad8(R):pad8(R) + r], kr, dtype)
        rest = [i for i in range(T + 3) if i not in rows.tolist()]
        assert float(home[rest].abs().max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,R,dv,splits", [(1, 3, 40, 24, 1), (5, 2, 512, 128, 7), (33, 4, 72, 72, 64)])
def test_latent_out_merges_partials(rt, dtype, T, H, R, dv, splits):
    from triton_distributed_b200 import ops

    o, uv, gate = rnd(T, H, splits, R), rnd(H, dv, R, seed=1, std=R ** -0.5).to(dtype), rnd(T, H * dv, seed=2).to(dtype)
    ml = torch.stack([rnd(T, H, splits, seed=3, std=6.0), torch.rand(T, H, splits) + 0.1], dim=-1)
    empty = torch.rand(T, H, splits, generator=torch.Generator().manual_seed(6)) < 0.4
    empty[..., 0] = False
    ml[empty] = torch.tensor([float("-inf"), 0.0])
    stale = o.clone()
    stale[empty] = float("nan")
    w = torch.where(empty, torch.zeros(1, dtype=torch.float64), torch.exp2(ml[..., 0].double()))
    merged = (w.unsqueeze(-1) * o.double()).sum(2) / (w * ml[..., 1].double()).sum(-1, keepdim=True)
    wide = torch.cat([torch.zeros(T, 16, dtype=dtype), gate], dim=1).to(DEV)[:, 16:]

    def want(m):
        return torch.einsum("hvr,thr->thv", uv.double(), m).flatten(1) * oracle.sigmoid(gate.double())

    close(ops.latent_out(stale.to(DEV), ml.to(DEV), uv.to(DEV), wide), want(merged), dtype)
    close(ops.latent_out(o[:, :, 0].contiguous().to(DEV), None, uv.to(DEV), wide), want(o[:, :, 0].double()), dtype)


# ------------------------------------------------------------------ attention
def _sharp_rows(n, R, r, q, seed, dtype, loud):
    """Cached rows [n, R + r]; those in ``loud`` are made to answer the queries ``q`` [H, R + r] above all others."""
    c = rnd(n, R + r, seed=seed)
    for i, j in enumerate(loud):
        c[j] = 0.3 * c[j] + (1.5 + 0.5 * (i % 2)) * q[i % q.shape[0]]
    return c.to(dtype)


def _absorbed_want(q, rows, R, scale):
    """q [H, R + r] over rows [n, R + r] -> [H, R]"""
    s = torch.stack([oracle.head_scores(q[h, :R], q[h, R:], rows[:, :R], rows[:, R:], scale) for h in range(q.shape[0])])
    return torch.softmax(s, dim=-1) @ rows[:, :R]


@pytest.mark.parametrize("H,R,r", [(4, 40, 8), (32, 512, 64), (33, 256, 32), (70, 128, 64), (1, 136, 16), (8, 448, 40)])
@pytest.mark.parametrize("splits", [0, 1, 3])
def test_latent_decode(rt, H, R, r, splits):
    """Split-KV decode over scattered slots, lengths around the tile's edges; far keys and keys beside the tile and split borders
    stand out, so that one that is missed or one that is too many shows."""
    from triton_distributed_b200 import ops

    dt, M = torch.bfloat16, 700
    lens = [1, 2, 127, 128, 129, 255, 256, 257, 384, 513, 700]
    B = len(lens)
    scale = 2.0 * (R + r) ** -0.5
    slots = torch.randperm(B + 2, generator=torch.Generator().manual_seed(1))[:B].to(torch.int32)
    q = rnd(B, H, R + r, seed=2).to(dt)
    cache = rnd(B + 2, M, R + r, seed=3).to(dt)
    for b, n in enumerate(lens):
        loud = sorted({j for j in (0, 127, 128, 255, 256, 383, 384, n - 1, n) if j < M})       # key n is not visible yet
        cache[slots[b]] = _sharp_rows(M, R, r, q[b].float(), 10 + b, dt, loud)
    lens_d = torch.tensor(lens, dtype=torch.int32, device=DEV)
    o, ml = ops.latent_decode(q.to(DEV), cache.to(DEV), slots.to(DEV), lens_d, R, scale, splits)
    ops.check_latent_errors()
    w = torch.where(ml[..., 1] > 0, torch.exp2(ml[..., 0] - ml[..., 0].amax(-1, keepdim=True)), torch.zeros_like(ml[..., 0]))
    o = torch.where(w.unsqueeze(-1) > 0, o, torch.zeros_like(o))
    got = (w.unsqueeze(-1) * o).sum(2) / (w * ml[..., 1]).sum(-1, keepdim=True)
    want = torch.stack([_absorbed_want(q[b].double(), cache[slots[b], :n].double(), R, scale) for b, n in enumerate(lens)])
    close(got, want, dt)
    simple = ops.latent_attention(q.to(DEV), cache.to(DEV), slots.to(DEV).long() * M, lens_d, R, scale)
    close(simple, want, torch.float32)


def test_latent_decode_with_growing_maxima(rt):
    """Scores that rise tile after tile, far beyond the range of an exponential: the reference maximum has to follow."""
    from triton_distributed_b200 import ops

    H, R, r, n = 5, 64, 8, 640
    q = rnd(1, H, R + r).to(torch.bfloat16)
    rows = rnd(n, R + r, seed=1) * 0.1
    rows += torch.linspace(0, 4, n)[:, None] * q[0].float().mean(0)
    rows = rows.to(torch.bfloat16)
    for flip in (False, True):
        c = rows.flip(0).contiguous() if flip else rows
        o, ml = ops.latent_decode(q.to(DEV), c[None].to(DEV), torch.zeros(1, dtype=torch.int32, device=DEV),
                                  torch.tensor([n], dtype=torch.int32, device=DEV), R, 3.0, 1)
        close(o[:, :, 0] / ml[:, :, 0, 1:], _absorbed_want(q[0].double(), c.double(), R, 3.0)[None], torch.bfloat16)


@pytest.mark.parametrize("H,d,r,dv", [(3, 128, 64, 128), (2, 64, 32, 64), (4, 16, 8, 24), (2, 72, 40, 104), (1, 96, 16, 40)])
@pytest.mark.parametrize("lens,starts", [([300], [0]), ([1, 130, 64, 257], [0, 0, 0, 0]), ([2, 200, 7], [63, 100, 640]), ([128, 1], [1, 256])])
def test_latent_prefill(rt, H, d, r, dv, lens, starts):
    """Prompts and portions of prompts on packed rows, each sequence's start padded to 64."""
    from triton_distributed_b200 import ops

    dt, R = torch.bfloat16, 48
    T = sum(lens)
    scale = 1.5 * (d + r) ** -0.5
    z = torch.cat([rnd(T, H * (d + r)), rnd(T, H * dv, seed=1)], dim=1).to(dt)
    q, gate = z[:, :H * (d + r)].reshape(T, H, d + r), z[:, H * (d + r):]
    ctx0, at = [], 0
    for n, s in zip(lens, starts):
        ctx0.append(at)
        at += (n + s + 63) // 64 * 64
    k, v, kr = rnd(at, H, d, seed=2), rnd(at, H, dv, seed=3).to(dt), rnd(at, r, seed=4)
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    for b, (n, s) in enumerate(zip(lens, starts)):      # keys that stand out: the first, block edges, the last ones
        for i, j in enumerate(sorted({0, 63, 64, 127, 128, n + s - 1, n + s - 2} & set(range(n + s)))):
            t = min(cu[b] + max(0, j - s) + 1, cu[b + 1] - 1)
            k[ctx0[b] + j] = 0.3 * k[ctx0[b] + j] + 1.6 * q[t, :, :d].float()
    k, kr = k.to(dt), kr.to(dt)
    ctx = torch.cat([rnd(at, R, seed=5), kr.float()], dim=1).to(dt)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)   # noqa: E731
    got = ops.latent_prefill(z.to(DEV), k.reshape(at, -1).to(DEV), ctx.to(DEV), v.reshape(at, -1).T.contiguous().to(DEV), i32(cu), i32(starts),
                             i32([n + s for n, s in zip(lens, starts)]), i32(ctx0), max(lens), H, d, r, dv, scale, z.to(DEV)[:, H * (d + r):])
    ops.check_latent_errors()
    want = torch.zeros(T, H, dv, dtype=torch.float64)
    for b, (n, s) in enumerate(zip(lens, starts)):
        for i in range(n):
            sl = slice(ctx0[b], ctx0[b] + s + i + 1)
            for h in range(H):
                x = oracle.head_scores(q[cu[b] + i, h, :d].double(), q[cu[b] + i, h, d:].double(), k[sl, h].double(), kr[sl].double(), scale)
                want[cu[b] + i, h] = torch.softmax(x, 0) @ v[sl, h].double()
    close(got, want.flatten(1) * oracle.sigmoid(gate.double()), dt)


# ------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,K,E,top,groups", [(1, 64, 6, 2, None), (17, 72, 33, 1, (3, 1)), (150, 512, 128, 8, (8, 3)), (65, 256, 512, 32, (16, 15)),
                                              (2077, 136, 130, 5, (130, 7)), (4096, 64, 16, 4, (2, 1)), (33, 64, 40, 3, (1, 1))])
def test_softmax_router(rt, dtype, T, K, E, top, groups):
    from triton_distributed_b200 import ops

    x, w = rnd(T, K).to(dtype), rnd(E, K, seed=1, std=2 * K ** -0.5).to(dtype)
    # mostly negative choice scores: groups that are left out must count as minus infinity, not as zero
    corr = rnd(E, seed=2, std=0.05) - 0.5
    g = {"count": groups[0], "keep": groups[1]} if groups else None
    for _ in range(2):                                   # the arrival counters are left clean
        ids, wts = ops.softmax_router(x.to(DEV), w.to(DEV), corr.to(DEV), top, *(groups or (0, 0)))
    z = x.double() @ w.double().T
    s = torch.softmax(z, dim=-1)
    assert (torch.gather(s, 1, ids.cpu().long()) - wts.cpu().double()).abs().max() < 1e-5
    assert all(len(set(row)) == top for row in ids.tolist())
    same = 0
    for t in range(0, T, max(1, T // 150)):
        want, _ = oracle.route(z[t], corr.double(), top, g)
        if ids[t].tolist() == want:
            same += 1
            continue
        # only a choice that is close to a tie may differ
        c = s[t] + corr.double()
        assert abs(float(c[ids[t].long().cpu()].sum() - c[want].sum())) < 1e-5 * top, (ids[t].tolist(), want)
    assert same > 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,K,F,Fs,E,top,ident", [(1, 64, 24, 40, 5, 2, 1), (9, 72, 80, 0, 4, 1, 2), (16, 256, 96, 136, 6, 3, 0), (5, 2048, 40, 768, 3, 3, 3),
                                                  (40, 64, 24, 16, 5, 2, 2)])
def test_gated_experts(rt, dtype, T, K, F, Fs, E, top, ident):
    from triton_distributed_b200 import ops

    x = rnd(T, K).to(dtype)
    W = {}
    for e in range(E):
        for i, (n, shape) in enumerate((("gate", (F, K)), ("up", (F, K)), ("down", (K, F)))):
            W[f"e{e}.{n}"] = rnd(*shape, seed=10 * e + i, std=shape[1] ** -0.5).to(dtype)
    if Fs:
        W["s.gate"], W["s.up"], W["s.down"] = (rnd(*s, seed=90 + i, std=s[1] ** -0.5).to(dtype) for i, s in enumerate(((Fs, K), (Fs, K), (K, Fs))))
    gu = torch.stack([torch.cat([W[f"e{e}.gate"], W[f"e{e}.up"]]) for e in range(E)]).to(DEV)
    down = torch.stack([W[f"e{e}.down"] for e in range(E)]).to(DEV)
    sgu, sd = (torch.cat([W["s.gate"], W["s.up"]]).to(DEV), W["s.down"].to(DEV)) if Fs else (None, None)
    ids = torch.stack([torch.randperm(E + ident, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)]).to(torch.int32)
    if ident >= top:
        ids[0] = torch.arange(E, E + top)                # a token whose experts are all identity
    wts = torch.rand(T, top)
    Wd = {n: t.double() for n, t in W.items()}
    routed, own, shared = (torch.zeros(T, K, dtype=torch.float64) for _ in range(3))
    for t in range(T):
        h = x[t].double()
        for e, we in zip(ids[t].tolist(), wts[t].double()):
            if e < E:
                routed[t] += we * oracle.expert(h, Wd, f"e{e}.")
            else:
                own[t] += we * h
        if Fs:
            shared[t] = oracle.expert(h, Wd, "s.")
    args = (x.to(DEV), gu, down, ids.to(DEV), wts.to(DEV), sgu, sd)
    got = ops.gated_experts_gemv(*args, identity=ident)
    assert got.dtype == torch.float32
    close(got, routed + own + shared, dtype)
    if ident:
        close(ops.gated_experts_gemv(*args, identity=ident, skip_identity=True), routed + shared, dtype)
    if dtype == torch.bfloat16:                          # the grouped-GEMM form of the same sum
        srt = ops.sort_topk_ids_align_block_size(ids.to(DEV), E)
        h = ops.silu_mul(ops.group_gemm_gather(x.to(DEV), gu, srt, a_row_div=top, scatter_out=True))
        y = ops.group_gemm_gather(h, down, srt, a_row_div=1, scatter_out=True, row_weight=wts.to(DEV))
        ff = ops.FeedForward(y, top, ids.to(DEV), wts.to(DEV), E, x.to(DEV))
        close(ops.parallel_sum(torch.zeros(T, K, device=DEV), torch.zeros(T, K, device=DEV, dtype=dtype), ff), routed + own, dtype, 1.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_biased_squared_relu(rt, dtype):
    from triton_distributed_b200 import ops

    x, b, w = rnd(7, 88).to(dtype), rnd(88, seed=1), torch.rand(7)
    close(ops.relu2(x.to(DEV), None, b.to(DEV)), torch.clamp(x.double() + b.double(), min=0) ** 2, dtype)
    close(ops.relu2(x.to(DEV), w.to(DEV), b.to(DEV)), torch.clamp(w.double()[:, None] * x.double() + b.double(), min=0) ** 2, dtype)


# ------------------------------------------------------------------ whole models
WIDE = cases.config([(cases.latent(8, 128, 64, 128, 200), cases.moe(6, 3, 72, 136, 2, (4, 2))), (cases.latent(33, 40, 64, 72, 200, kv_from=0), cases.dense(136)),
                     (cases.latent(2, 160, 32, 136, 520), cases.moe(6, 3, 40, 0, 3, None)), (cases.latent(4, 64, 32, 16, 520, kv_from=2), cases.moe(5, 2, 64, 64, 1, (2, 1)))],
                    width=200, vocab=203, scale=1.7)
MODELS = {"mixed": cases.MIXED, "plain": cases.PLAIN, "wide": WIDE}
_MADE = {}


@pytest.fixture(params=sorted(MODELS))
def model(request, rt, tmp_path_factory):
    """(directory, config, weights, tokens, the oracle's logits)"""
    name = request.param
    if name not in _MADE:
        cfg = MODELS[name]
        # bf16 rounding grows with the sharpness of the softmax: 1.5 keeps single keys dominant at a rounding error of 1-2 %
        w = cases.weights(cfg, seed=11, sharp=1.5, clear_routing=True)
        toks = cases.prompt(cfg, 301 if name == "wide" else 157)
        _MADE[name] = (str(cases.write(tmp_path_factory.mktemp(name), cfg, w)), cfg, w, toks, oracle.forward(cfg, w, toks))
    return _MADE[name]


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_portions_and_decoding(model, dtype):
    d, _, _, toks, want = model
    n = len(toks)
    eng = cases.engine(d, dtype, max_length=400)
    for sizes in ([n], [n - 60, 1], [2], [97, 64, 3, 30], [150, 1, 1, 100]):
        assert cases.rel(cases.run_portions(eng, "r", toks, sizes), want) < TOL[dtype], sizes
    from triton_distributed_b200 import ops
    ops.check_latent_errors()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_and_reused_slots(model, dtype):
    d, cfg, w, toks, want = model
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


def test_wide_decode_batches(rt, tmp_path):
    """More sequences than the pair-by-pair expert kernel takes: decode steps through the grouped GEMMs."""
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=5, sharp=1.5, clear_routing=True)
    d = cases.write(tmp_path, cfg, w)
    lens = [5 + 3 * (i % 7) for i in range(21)]
    prompts = [cases.prompt(cfg, n + 3, i) for i, n in enumerate(lens)]
    for dtype in DTYPES:
        eng = cases.engine(d, dtype, max_length=64)
        rows = [eng.step([(i, p[:n], []) for i, (p, n) in enumerate(zip(prompts, lens))])]
        rows = [eng.step([(i, [p[n + k]], [0]) for i, (p, n) in enumerate(zip(prompts, lens))]) for k in range(3)]
        for i in range(0, 21, 4):
            want = oracle.forward(cfg, w, prompts[i])[lens[i]:]
            assert cases.rel(torch.stack([r[i] for r in rows]), want) < TOL[dtype], i


def test_greedy_generation_with_cuda_graph(rt, tmp_path):
    """Generation through serve() (graph-replayed decode steps) equals the oracle's."""
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=3, sharp=1.5, clear_routing=True)
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
    out = eng.serve(torch.tensor(prompts), 8)
    full = torch.cat([torch.tensor(prompts), out.cpu()], dim=1).tolist()
    for b, toks in enumerate(full):
        ref = oracle.forward(cfg, w, toks[:-1])[21:]
        assert cases.rel(torch.stack([z[b] for z in eng.step_logits]), ref) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode_across_tiles(rt, tmp_path, dtype):
    cfg = cases.config([(cases.latent(2, 16, 8, 8, 24), cases.dense(24)), (cases.latent(3, 16, 8, 16, 24, kv_from=0), cases.moe(3, 1, 16, 8, 1, None))], 32, 64)
    w = cases.weights(cfg, seed=4, sharp=1.5, clear_routing=True)
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
