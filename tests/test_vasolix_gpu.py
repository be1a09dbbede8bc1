"""Vasolix on one GPU: every kernel alone and the whole model (bf16 and fp32) against the plain oracle on the CPU."""
import json
import os
import subprocess
import sys

import pytest
import torch

import vasolix_cases as cases
import vasolix_oracle as oracle

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


# ------------------------------------------------------------------ stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,real,rows", [(72, 67, 1), (256, 256, 3), (4096, 4096, 2)])
def test_stream_kernels(rt, dtype, W, real, rows):
    from triton_distributed_b200 import ops

    T = 5
    mask = (torch.arange(W) < real).float()
    y, sh, x0 = rnd(T * rows, W) * mask, rnd(T, W, seed=1) * mask, rnd(T, W, seed=2) * mask
    y, sh = y.to(dtype), sh.to(dtype)
    w, gate = (1 + 0.2 * rnd(W, seed=3)) * mask, torch.rand(T)
    for shared in (None, sh):
        x = x0.to(DEV)
        xb = x if dtype == torch.float32 else x.to(dtype)
        args = (rows, None if shared is None else shared.to(DEV), None if shared is None else gate.to(DEV))
        ops.postnorm_add(x, xb, y.to(DEV), w.to(DEV), real, 1e-4, *args)
        s = y.double().reshape(T, rows, W).sum(1) + (0 if shared is None else gate.double()[:, None] * shared.double())
        want = x0.double()
        want[:, :real] += oracle.rms(s[:, :real], 1e-4, w[:real].double())
        close(x, want, torch.float32)
        assert torch.equal(xb.float(), x.to(dtype).float())
        close(ops.combine_rows(y.to(DEV), T, *args), s, dtype)
    pick = torch.tensor([4, 0, 4])
    got = ops.stream_norm(x, w.to(DEV), real, 1e-4, dtype, pick.to(DEV))
    close(got[:, :real], oracle.rms(x.cpu().double()[pick][:, :real], 1e-4, w[:real].double()), dtype)
    table = rnd(11, W, seed=4).to(dtype)
    ids = torch.tensor([10, 0, 3])
    ex, exb = ops.embed_stream(ids.to(DEV), table.to(DEV))
    assert torch.equal(ex.cpu(), table[ids].float()) and torch.equal(exb.cpu(), table[ids])


# ------------------------------------------------------------------ attention
def _tied_inputs(T, Hq, Hkv, D, dtype, seed=0):
    """q (already normed), raw keys and factors; query Hq - 1 of every token is made to stand out against one key."""
    q, k, f = rnd(T, Hq, D, seed=seed), rnd(T, Hkv, D, seed=seed + 1), torch.rand(T, generator=torch.Generator().manual_seed(seed)) + 0.5
    q = (q * D ** -0.5).to(dtype)
    return q, k.to(dtype), f


def _tied_want(q, k, f, lo, sink, gate):
    """Token t of one sequence sees keys lo[t] .. t."""
    T, Hq, D = q.shape
    g = Hq // k.shape[1]
    out = torch.zeros(T, Hq, D, dtype=torch.float64)
    for t in range(T):
        for h in range(Hq):
            kk = k[lo[t]:t + 1, h // g].double()
            s = kk @ q[t, h].double() * f[lo[t]:t + 1].double()
            out[t, h] = oracle.sink_softmax(s, sink[h]) @ kk
    return (out.reshape(T, -1) * oracle.sigmoid(gate.double())).reshape(T, Hq, D)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N", [(48, 16), (24, 24), (2048, 512)])
def test_qk_norm_tied(rt, dtype, N):
    from triton_distributed_b200 import ops

    nq, nk = N
    T = 6
    qk = rnd(T, nq + nk + 8, std=3.0).to(dtype)
    w = 1 + 0.3 * rnd(nq, seed=1)
    kc, sc = torch.zeros(10, nk, dtype=dtype, device=DEV), torch.zeros(10, device=DEV)
    k2, s2 = torch.zeros(4, nk, dtype=dtype, device=DEV), torch.zeros(4, device=DEV)
    rows, rows2 = torch.tensor([9, 0, 5, 2, 7, 1]), torch.tensor([-1, 3, -1, 0, -1, 99])
    d = qk.to(DEV)
    for sumsq in (None, ops.qk_sumsq(d, nq, nk)):
        q = ops.qk_norm_tied(d, w.to(DEV), nk, nq, nk, 1e-5, (kc, sc, rows.to(DEV)), (k2, s2, rows2.to(DEV)), sumsq)
        close(q, oracle.rms(qk[:, :nq].double(), 1e-5, w.double()), dtype)
        raw = qk[:, nq:nq + nk]
        assert torch.equal(kc.cpu()[rows], raw) and torch.equal(k2.cpu()[[3, 0]], raw[[1, 3]])
        fac = 1 / torch.sqrt(raw.double().pow(2).mean(-1) + 1e-5)
        close(sc[rows.to(DEV)], fac, torch.float32)
        close(s2[[3, 0]], fac[[1, 3]], torch.float32)
        assert float(k2[1:3].abs().max()) == 0.0


@pytest.mark.parametrize("D,Hq,Hkv,impl", [(32, 4, 2, "mma"), (64, 6, 2, "mma"), (128, 4, 1, "mma"), (128, 4, 1, "sm100"), (256, 2, 2, "mma")])
@pytest.mark.parametrize("T,block,start", [(150, 64, 0), (141, 70, 0), (300, 150, 0), (33, 4096, 0)])
def test_tied_prefill(rt, D, Hq, Hkv, impl, T, block, start):
    """Prompt attention through the blocks a cache plan makes, scattered over a page pool; one far key of every block is
    made to dominate, so that an edge that is one token off shows."""
    from triton_distributed_b200 import ops
    from triton_distributed_b200.models import HybridCache, TiedKVSpec

    dt = torch.bfloat16
    q, k, f = _tied_inputs(T, Hq, Hkv, D, dt)
    for b in range(0, T, block):                        # the first key of a block answers all of its queries and the next block's
        k[b] = (2.0 * q.float().mean(0).reshape(Hkv, -1, D).mean(1) + 0.5 * k[b].float()).to(dt)
        f[b] = 4.0
    sink, gate = rnd(Hq, seed=5), rnd(T, Hq * D, seed=6).to(dt)
    spec = TiedKVSpec(Hkv, D, block)
    cache = HybridCache([spec], 1, 8192, dt, DEV)
    bp = cache.plan([0], [T]).blocks(spec)
    pages = torch.zeros(bp.pages, bp.page_rows, Hkv, D, dtype=dt, device=DEV)
    scale = torch.zeros(bp.pages, bp.page_rows, device=DEV)
    pages.view(-1, Hkv, D)[bp.scratch_rows] = k.to(DEV)
    scale.view(-1)[bp.scratch_rows] = f.to(DEV)
    wide = torch.zeros(T, Hq * D + 64, dtype=dt, device=DEV)
    wide[:, 64:] = gate.to(DEV)
    want = _tied_want(q, k, f, [t // block * block for t in range(T)], sink, gate)
    for got in (ops.tied_attn_varlen(q.to(DEV), pages, scale, bp.block_table, bp.cu, bp.q_pos0, bp.kv_lens, bp.max_q, bp.max_kv,
                                     sink.to(DEV), wide[:, 64:], impl=impl),
                ops.tied_attention_simple(q.to(DEV), pages, scale, bp.row0, bp.n_keys, sink.to(DEV), wide[:, 64:])):
        close(got, want, dt)
    from triton_distributed_b200.ops.attention import check_attention_errors
    check_attention_errors()


@pytest.mark.parametrize("D,Hq,Hkv", [(32, 4, 4), (64, 40, 2), (128, 8, 2), (256, 3, 1)])
@pytest.mark.parametrize("splits", [1, 3])
def test_tied_decode(rt, D, Hq, Hkv, splits):
    from triton_distributed_b200 import ops

    dt, block = torch.bfloat16, 150
    lens = [1, 64, 149, 150, 151, 215, 300, 301, 700]
    B = len(lens)
    slots = torch.randperm(B + 3, generator=torch.Generator().manual_seed(1))[:B]
    kc = rnd(B + 3, block, Hkv, D, seed=2).to(dt)
    sc = torch.rand(B + 3, block) + 0.5
    q = (rnd(B, Hq, D, seed=3) * 2 * D ** -0.5).to(dt)
    sink, gate = rnd(Hq, seed=4), rnd(B, Hq * D, seed=5).to(dt)
    got = ops.tied_attn_decode(q.to(DEV), kc.to(DEV), sc.to(DEV), slots.to(torch.int32).to(DEV).unsqueeze(1).contiguous(),
                               torch.tensor(lens, dtype=torch.int32, device=DEV), block, splits, sink.to(DEV), gate.to(DEV))
    want = torch.zeros(B, Hq, D, dtype=torch.float64)
    for b, n in enumerate(lens):
        m = (n - 1) % block + 1
        for h in range(Hq):
            kk = kc[slots[b], :m, h // (Hq // Hkv)].double()
            want[b, h] = oracle.sink_softmax(kk @ q[b, h].double() * sc[slots[b], :m].double(), sink[h]) @ kk
    close(got, (want.reshape(B, -1) * oracle.sigmoid(gate.double())).reshape(B, Hq, D), dt)


# ------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,K,E,top,gated", [(1, 64, 5, 2, True), (17, 72, 33, 1, False), (150, 512, 128, 8, True), (65, 256, 511, 32, True), (2077, 136, 130, 5, True),
                                             (2100, 200, 300, 4, False), (4096, 64, 16, 16, True)])
def test_sigmoid_router(rt, dtype, T, K, E, top, gated):
    from triton_distributed_b200 import ops

    x, w = rnd(T, K).to(dtype), rnd(E + gated, K, seed=1, std=2 * K ** -0.5).to(dtype)
    for _ in range(2):                                   # the arrival counters are left clean
        ids, wts, gate = ops.sigmoid_router(x.to(DEV), w.to(DEV), top, gated)
    s = oracle.sigmoid(x.double() @ w.double().T)
    best = torch.sort(s[:, :E], dim=1, descending=True)
    assert (wts.cpu().double() - best.values[:, :top]).abs().max() < 1e-4
    picked = torch.gather(s, 1, ids.cpu().long())
    assert (picked - wts.cpu().double()).abs().max() < 1e-4 and all(len(set(r)) == top for r in ids.tolist())
    assert gate is None if not gated else (gate.cpu().double() - s[:, E]).abs().max() < 1e-4
    lin = ops.narrow_linear(x.to(DEV), w.to(DEV))
    assert lin.dtype == torch.float32
    close(lin, x.double() @ w.double().T, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,K,F,Fs,E,top", [(1, 64, 24, 40, 5, 2), (9, 72, 80, 0, 4, 1), (16, 256, 96, 136, 6, 3)])
def test_experts_gemv(rt, dtype, T, K, F, Fs, E, top):
    from triton_distributed_b200 import ops

    x = rnd(T, K).to(dtype)
    W = {}
    for e in range(E):
        W[f"e{e}.up"], W[f"e{e}.down"] = rnd(F, K, seed=e, std=K ** -0.5).to(dtype), rnd(K, F, seed=90 + e, std=F ** -0.5).to(dtype)
    up, down = (torch.stack([W[f"e{e}.{n}"] for e in range(E)]).to(DEV) for n in ("up", "down"))
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)])
    wts, gate = torch.rand(T, top), torch.rand(T)
    sh = (rnd(Fs, K, seed=7, std=K ** -0.5).to(dtype), rnd(K, Fs, seed=8, std=Fs ** -0.5).to(dtype)) if Fs else (None, None)
    want = torch.zeros(T, K, dtype=torch.float64)
    Wd = {n: t.double() for n, t in W.items()}
    if Fs:
        Wd["s.up"], Wd["s.down"] = sh[0].double(), sh[1].double()
    for t in range(T):
        for e, we in zip(ids[t].tolist(), wts[t].double()):
            want[t] += oracle.expert(we * x[t].double(), Wd, f"e{e}.")
        if Fs:
            want[t] += gate[t].double() * oracle.expert(x[t].double(), Wd, "s.")
    dev = lambda t: None if t is None else t.to(DEV)   # noqa: E731
    got = ops.relu2_experts_gemv(x.to(DEV), up, down, ids.to(torch.int32).to(DEV), wts.to(DEV), dev(sh[0]), dev(sh[1]),
                                 gate.to(DEV) if Fs else None)
    assert got.dtype == torch.float32
    close(got, want, dtype)
    if dtype == torch.bfloat16:                          # the grouped-GEMM form of the same sum, without the shared expert
        srt = ops.sort_topk_ids_align_block_size(ids.to(torch.int32).to(DEV), E)
        h = ops.relu2(ops.group_gemm_gather(x.to(DEV), up, srt, a_row_div=top, scatter_out=True), wts.reshape(-1).to(DEV))
        y = ops.group_gemm_gather(h, down, srt, a_row_div=1, scatter_out=True)
        y = ops.combine_rows(y, T, top, None if not Fs else (ops.relu2(x.to(DEV) @ sh[0].to(DEV).T) @ sh[1].to(DEV).T), gate.to(DEV))
        close(y, want, dtype, 1.5)


# ------------------------------------------------------------------ gated linear attention
def _gla_case(lens, H, dk, dv, dtype, strong, seed=0):
    T, R = sum(lens), 5
    qkvg = rnd(T, 2 * H * (dk + dv), seed=seed).to(dtype)
    low, a2 = rnd(T, R, seed=seed + 1), rnd(R, H * dk, seed=seed + 2, std=1.5)
    # strong: decays from none to e^-60 per token, so that differences of cumulative logs leave the range of exp
    b = rnd(H * dk, seed=seed + 3, std=30.0 if strong else 2.0) + (0.0 if strong else 2.0)
    state = rnd(len(lens) + 2, H, dk, dv, seed=seed + 4)
    slots = torch.randperm(len(lens) + 2, generator=torch.Generator().manual_seed(seed))[:len(lens)].to(torch.int32)
    pos0 = torch.tensor([0 if i % 2 else 7 for i in range(len(lens))])
    return qkvg, low, a2, b, state, slots, pos0


def _gla_want(case, lens, H, dk, dv, tau, norm_w, scale, eps, dv_real):
    qkvg, low, a2, b, state, slots, pos0 = case
    f = qkvg.double()
    T = f.shape[0]
    q, k, v, g = f.split([H * dk, H * dk, H * dv, H * dv], dim=1)
    alpha = (oracle.sigmoid(low.double() @ a2.double() + b.double()) ** (1 / tau)).reshape(T, H, dk)
    out, states, at = [], state.double().clone(), 0
    for i, n in enumerate(lens):
        sl = slice(at, at + n)
        S0 = None if pos0[i] == 0 else state[slots[i]].double()
        o, S = oracle.gla_recurrence(q[sl].reshape(n, H, dk) * scale, k[sl].reshape(n, H, dk), v[sl].reshape(n, H, dv), alpha[sl], S0)
        states[slots[i]] = S
        norm = o[..., :dv_real] / torch.sqrt(o[..., :dv_real].pow(2).mean(-1, keepdim=True) + eps)
        out.append(torch.cat([norm * norm_w[:dv_real].double(), torch.zeros(n, H, dv - dv_real).double()], -1).reshape(n, H * dv)
                   * oracle.silu(g[sl]))
        at += n
    return torch.cat(out), states


@pytest.mark.parametrize("impl", ["chunk", "recurrent", "decode"])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,dk,dv,dv_real", [(2, 16, 16, 16), (3, 48, 48, 41), (2, 64, 128, 128), (1, 128, 256, 256), (1, 256, 112, 112)])
def test_gla_kernels(rt, impl, strong, H, dk, dv, dv_real):
    from triton_distributed_b200 import ops

    lens = [1, 1, 1, 1, 1] if impl == "decode" else [64, 1, 130, 15, 65, 2]
    for dtype in ([torch.bfloat16] if impl == "chunk" else DTYPES):
        case = _gla_case(lens, H, dk, dv, dtype, strong)
        if dv_real < dv:                                  # padded value columns are zero
            case[0][:, 2 * H * dk:2 * H * dk + H * dv].reshape(-1, H, dv)[..., dv_real:] = 0
            case[4][..., dv_real:] = 0
        norm_w = 1 + 0.2 * rnd(dv, seed=20)
        norm_w[dv_real:] = 0
        want, want_state = _gla_want(case, lens, H, dk, dv, 2.0, norm_w, 0.3, 1e-5, dv_real)
        qkvg, low, a2, b, state, slots, pos0 = (t.to(DEV) for t in case)
        cu_host = [0]
        for n in lens:
            cu_host.append(cu_host[-1] + n)
        cu = None if impl == "decode" else torch.tensor(cu_host, dtype=torch.int32, device=DEV)
        got = ops.gated_linear_attention(qkvg, low, a2, b, 2.0, norm_w.to(DEV), state, slots, pos0, cu, dv_real, 0.3, 1e-5,
                                         ops.gla_chunk_tables(cu_host, DEV), impl)
        assert bool(torch.isfinite(got.float()).all())
        close(got, want, dtype)
        close(state, want_state, torch.float32, 5.0)      # the state stays 32-bit whatever the activations are
        rest = [i for i in range(state.shape[0]) if i not in slots.tolist()]
        assert torch.equal(state[rest].cpu(), case[4][rest])


# ------------------------------------------------------------------ whole models
WIDE = cases.config([(cases.attention(8, 2, 128, 150), cases.moe(6, 2, 72, 136)), (cases.gla(2, 64, 128, 8.0), cases.moe(6, 3, 64, 64)),
                     (cases.attention(3, 1, 256, 40), cases.moe(3, 1, 40, 0)), (cases.attention(4, 2, 64, 64), cases.moe(6, 2, 72, 24))],
                    width=200, vocab=203)
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
        toks = cases.prompt(cfg, 331 if name == "wide" else 157)
        _MADE[name] = (str(cases.write(tmp_path_factory.mktemp(name), cfg, w)), cfg, w, toks, oracle.forward(cfg, w, toks))
    return _MADE[name]


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_portions_and_decoding(model, dtype):
    d, _, _, toks, want = model
    n = len(toks)
    eng = cases.engine(d, dtype, max_length=400)
    for sizes in ([n], [n - 60, 1], [2], [97, 64, 3, 30], [150, 1, 1, 100]):
        assert cases.rel(cases.run_portions(eng, "r", toks, sizes), want) < TOL[dtype], sizes


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


def test_greedy_generation_with_cuda_graph(rt, tmp_path):
    """Generation through serve() (graph-replayed decode steps, recurrent states included) equals the oracle's."""
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


def test_long_decode_through_many_blocks(rt, tmp_path):
    cfg = cases.config([(cases.attention(2, 1, 16, 9), None), (cases.gla(1, 16, 16, 16.0), cases.moe(3, 1, 16, 8))], 32, 64)
    w = cases.weights(cfg, seed=4)
    toks = cases.prompt(cfg, 300)
    eng = cases.engine(cases.write(tmp_path, cfg, w), torch.float32, max_length=300)
    assert cases.rel(cases.run_portions(eng, 0, toks, [1]), oracle.forward(cfg, w, toks)) < TOL[torch.float32]


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
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1"]
    got = torch.cat([torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, 101) for n in (0, 1)])
    assert cases.rel(got, oracle.forward(cfg, w, toks)[[0, 48, 49]]) < TOL[torch.float32]
