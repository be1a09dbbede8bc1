"""Tazitar on CPU ranks (fp32): configuration, weights, cache plans, engine steps, generation, tensor parallelism.  The kernels are
covered by test_tazitar_gpu.py; here the host logic runs over the ops' CPU backend."""
import io
import json
import math

import pytest
import torch

import tazitar_cases as cases
import tazitar_oracle as oracle
from dist_utils import run_cpu_ranks

TOL = 2e-5


@pytest.fixture(scope="module")
def rt():
    import triton_distributed_b200 as tdb

    tdb.initialize_distributed(seed=0, device="cpu")
    yield tdb.get_runtime()
    tdb.finalize_distributed()


@pytest.fixture(scope="module")
def mixed(rt, tmp_path_factory):
    w = cases.weights(cases.MIXED, seed=1)
    d = cases.write(tmp_path_factory.mktemp("mixed"), cases.MIXED, w)
    toks = cases.prompt(cases.MIXED, 61)
    return d, w, toks, oracle.forward(cases.MIXED, w, toks)


# ------------------------------------------------------------------ the oracle itself
@pytest.mark.parametrize("interleaved", [False, True])
def test_oracle_rotation(interleaved):
    x = torch.tensor([1.0, 0.0, 0.5, 2.0, 3.0, 4.0, 7.0, -1.0], dtype=torch.float64)
    y = oracle.rotate(x, 5, cases.rot(6, 100.0), interleaved)
    for i in range(3):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + 3)
        ang = 5 * 100.0 ** (-2 * i / 6)
        turned = complex(x[a], x[b]) * complex(math.cos(ang), math.sin(ang))
        assert abs(turned - complex(y[a], y[b])) < 1e-12
    assert torch.equal(y[6:], x[6:]) and torch.equal(oracle.rotate(x, 0, cases.rot(6, 100.0), interleaved), x)
    q, k = torch.randn(8, dtype=torch.float64), torch.randn(8, dtype=torch.float64)
    near = oracle.rotate(q, 9, cases.rot(8, 50.0), interleaved) @ oracle.rotate(k, 4, cases.rot(8, 50.0), interleaved)
    far = oracle.rotate(q, 1009, cases.rot(8, 50.0), interleaved) @ oracle.rotate(k, 1004, cases.rot(8, 50.0), interleaved)
    assert abs(float(near - far)) < 1e-9


def test_oracle_yarn():
    """Fast pairs keep their frequency, slow ones are divided by the factor, and the ramp between them is monotone."""
    base, dims = 1e4, 64
    f, mult = oracle.frequencies(cases.rot(dims, base, factor=8.0, original=2048, fast=32.0, slow=1.0))
    plain, one = oracle.frequencies(cases.rot(dims, base))
    assert one == 1.0 and abs(mult - (0.1 * math.log(8.0) + 1)) < 1e-15
    ratio = [a / b for a, b in zip(f, plain)]
    assert all(x >= y - 1e-15 for x, y in zip(ratio, ratio[1:]))
    for r, p in zip(ratio, plain):
        turns = 2048 * p / (2 * math.pi)
        if turns > 64:
            assert r == 1.0
        if turns < 0.5:
            assert abs(r - 1 / 8) < 1e-15
    assert any(0.2 < r < 0.9 for r in ratio)
    same, mult = oracle.frequencies(cases.rot(dims, base, factor=1.0, original=2048, fast=32.0, slow=1.0))
    assert mult == 1.0 and max(abs(a - b) for a, b in zip(same, plain)) < 1e-15
    # ends that coincide: a step
    step, _ = oracle.frequencies(cases.rot(8, 10.0, factor=2.0, original=6, fast=64.0, slow=32.0))
    assert len(step) == 4


def test_oracle_delta_rule():
    """With beta = 1 and no decay the state answers a key with the last value written for it; decay and step size act as stated."""
    g = torch.Generator().manual_seed(0)
    k = oracle.unit(torch.randn(1, 6, generator=g, dtype=torch.float64))
    one, S = torch.ones(1, dtype=torch.float64), torch.zeros(1, 6, 3, dtype=torch.float64)
    v1, v2 = torch.randn(1, 3, generator=g, dtype=torch.float64), torch.randn(1, 3, generator=g, dtype=torch.float64)
    S, o = oracle.delta_step(S, k, k, v1, one, one)
    assert torch.allclose(o, v1, atol=1e-5)
    S, o = oracle.delta_step(S, k, k, v2, one, one)
    assert torch.allclose(o, v2, atol=1e-5)                       # the read-out sees the write, which replaced the old value
    S, o = oracle.delta_step(S, k, k, v1, 0.5 * one, 0.25 * one)
    assert torch.allclose(o, 0.75 * 0.5 * v2 + 0.25 * v1, atol=1e-5)


def test_oracle_short_conv_and_softplus():
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=torch.float64)
    w = torch.tensor([[2.0, 3.0, 5.0]], dtype=torch.float64)       # two back, one back, current
    assert oracle.short_conv(x, w).flatten().tolist() == [5.0, 53.0, 532.0, 5320.0]
    z = torch.tensor([-50.0, -1.0, 0.0, 3.0, 60.0], dtype=torch.float64)
    assert torch.allclose(oracle.softplus(z), torch.log1p(torch.exp(z)), atol=1e-15)


# ------------------------------------------------------------------ configuration and registry
def test_configuration_is_read_and_checked(mixed, tmp_path):
    from triton_distributed_b200 import ops
    from triton_distributed_b200.models import ModelConfig, TazitarConfig

    a = ModelConfig(checkpoint_dir=str(mixed[0])).arch()
    assert isinstance(a, TazitarConfig) and a.vocab_size == 101 and a.hidden_size == 60 and a.streams == 3 and a.rms_norm_eps == 2e-3
    assert a.passes == (0, 1, 2, 3, 1, 2, 3, 4) and a.num_hidden_layers == 5 and not a.is_moe
    m = a.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.rot_dims, m.softcap, m.qk_norm, m.unit, m.interleaved, m.sink) == (6, 3, 20, 28, 14, 3.0, True, False, False, None)
    m = a.layers[2].mixer
    assert m.scaling == ops.YarnScaling(4.0, 48.0, 6.0, 0.8) and m.rot_base == 60.0 and (m.unit, m.interleaved, m.sink) == (True, True, "learned")
    m = a.layers[1].mixer
    assert (m.left.sink, m.left.unit, m.left.interleaved, m.left.softcap) == (0.0, True, False, 0.0)
    assert (m.right.heads, m.right.kv_heads, m.right.dim, m.right.vdim, m.right.conv) == (4, 2, 12, 20, 4)
    assert a.layers[2].mlp is None and a.layers[1].mlp.ff == 42

    def broken(i=0, mixer=None, mlp=None, layer=None, **change):
        c = json.loads(json.dumps(cases.MIXED))
        c["layers"][i].update(layer or {})
        c["layers"][i]["mixer"].update(mixer or {})
        if mlp:
            c["layers"][i]["mlp"].update(mlp)
        c.update(change)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return TazitarConfig.from_json(str(tmp_path))

    assert broken(loop=None).passes == (0, 1, 2, 3, 4) and broken(loop={"start": 0, "stop": 1, "times": 3}).passes == (0, 0, 0, 1, 2, 3, 4)
    for kw, what in ((dict(layer={"type": "other"}), "mixer"), (dict(mlp={"kind": "other"}), "kind"), (dict(mixer={"heads": 7}), "multiple"),
                     (dict(mixer={"rot": {"base": 10.0, "dims": 22}}), "rotation"), (dict(mixer={"rot": {"base": 10.0, "dims": 5}}), "rotation"),
                     (dict(i=1, mixer={"right": cases.delta(3, 2)}), "multiple"), (dict(i=1, mixer={"right": cases.delta(conv=0)}), "tap"),
                     (dict(streams=0), "streams"), (dict(streams=17), "streams"), (dict(loop={"start": 3, "stop": 3, "times": 2}), "loop"),
                     (dict(loop={"start": 0, "stop": 6, "times": 2}), "loop"), (dict(loop={"start": 0, "stop": 2, "times": 0}), "loop")):
        with pytest.raises(ValueError, match=what):
            broken(**kw)


def test_registry_presets_and_limits(rt):
    from triton_distributed_b200.models import TAZITAR_PRESETS, AutoLLM, ModelConfig, TazitarLLM
    from triton_distributed_b200.models.tazitar import DeltaRuleSpec, RotaryAttnSpec
    from triton_distributed_b200.parallel import TP_DeltaRule, TP_RotaryAttn

    m = AutoLLM.from_pretrained(ModelConfig(model_name="tiny-tazitar", dtype=torch.float32))
    assert isinstance(m, TazitarLLM) and m.arch.passes == (0, 1, 2, 1, 2, 3) and len(m.cache_specs()) == 6
    out = m.inference(torch.tensor([[3, 5, 9]]), torch.arange(3)[None], m.new_cache(1, 8))
    assert out.shape == (1, 1000) and torch.isfinite(out).all()
    short = ModelConfig(model_name="tiny-tazitar", num_layers_override=2).arch()
    assert short.passes == (0, 1, 1) and ModelConfig(model_name="tiny-tazitar", num_layers_override=1).arch().loop is None
    assert TAZITAR_PRESETS["tiny-tazitar"].with_num_layers(6).num_hidden_layers == 6
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        AutoLLM.from_pretrained(ModelConfig(model_name="tiny-tazitar", dtype=torch.float16))
    with pytest.raises(ValueError, match="256"):
        TP_DeltaRule(DeltaRuleSpec(2, 2, 300, 16, 4))
    with pytest.raises(ValueError, match="1024"):
        TP_RotaryAttn(RotaryAttnSpec(2, 2, 1100, 16, 1.0, 1e4, 8))
    dims = [TP_RotaryAttn(RotaryAttnSpec(2, 2, d, v, 1.0, 1e4, 8)).head_dim for d, v in ((8, 8), (44, 72), (64, 64), (200, 16), (64, 300))]
    assert dims == [64, 128, 64, 256, 512]
    assert [TP_DeltaRule(DeltaRuleSpec(2, 2, d, 16, 4)).dk for d in (9, 48, 100, 130, 200)] == [16, 48, 128, 192, 256]


# ------------------------------------------------------------------ forward
def test_prompt_matches_oracle_layer_by_layer(mixed):
    d, w, toks, want = mixed
    eng = cases.engine(d, torch.float32)
    streams, ref = [], []
    oracle.forward(cases.MIXED, w, toks, ref)
    cache = eng.model.new_cache(1, 64)
    got = eng.model.forward_step(torch.tensor(toks), cache.plan([0], [len(toks)]), None, False, streams)
    assert len(streams) == len(ref) == 8
    for a, b in zip(streams, ref):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)
    assert cases.rel(got, want) < TOL


@pytest.mark.parametrize("sizes", [[2], [1], [7], [24, 1], [17, 3, 50], [60, 1], [5, 40]])
def test_portions_of_any_size(mixed, sizes):
    d, _, toks, want = mixed
    assert cases.rel(cases.run_portions(cases.engine(d, torch.float32), "r", toks, sizes), want) < TOL


def test_batches_of_unequal_requests_and_reused_slots(mixed):
    d, w, _, _ = mixed
    eng = cases.engine(d, torch.float32)
    prompts = {i: cases.prompt(cases.MIXED, n, i) for i, n in enumerate([1, 30, 17, 52, 24])}
    want = {i: oracle.forward(cases.MIXED, w, p) for i, p in prompts.items()}
    got = {i: [] for i in prompts}

    def step(parts):
        z = eng.step([(i, prompts[i][lo:hi], list(range(hi - lo))) for i, lo, hi in parts])
        for i, lo, hi in parts:
            got[i].append(z[:hi - lo])
            z = z[hi - lo:]

    step([(0, 0, 1), (1, 0, 20), (2, 0, 16)])
    eng.end([0])
    step([(2, 16, 17), (1, 20, 22), (3, 0, 25)])          # takes the freed slot, mixes a decode with portions
    eng.end([2])
    step([(4, 0, 23), (3, 25, 26)])
    for k in range(22, 30):
        step([(1, k, k + 1), (3, k + 4, k + 5)])
    step([(3, 34, 52), (4, 23, 24)])
    assert eng.step_cache.capacity <= 6
    for i in prompts:
        assert cases.rel(torch.cat(got[i]), want[i]) < TOL, i


def test_cache_storage_and_plans():
    from triton_distributed_b200.models import DeltaSpec, GroupSpec, HybridCache, KVSpec, StateSpec

    pair = GroupSpec((KVSpec(2, 64), DeltaSpec(3, 16, 32, 160, 4)))
    c = HybridCache([KVSpec(1, 128), pair, pair], 2, 100, torch.bfloat16, "cpu")
    assert c.layers[0]["k"].shape == c.layers[0]["v"].shape == (2, 100, 1, 128) and c.layers[0]["k"].dtype == torch.bfloat16
    st = c.layers[1]
    assert set(st) == {"k", "v", "state", "conv"} and st["state"].shape == (2, 3, 16, 32) and st["state"].dtype == torch.float32
    assert st["conv"].shape == (2, 4, 160) and st["conv"].dtype == torch.bfloat16 and c.layers[2]["k"] is not st["k"]
    st["state"][1], st["conv"][1] = 3.0, 2.0
    snap = c.snapshot()
    assert snap[0] is None and float(snap[1][1].min()) == 3.0
    assert c.alloc() == 2 and c.capacity == 4                # grows: what is there stays
    assert float(c.layers[1]["state"][1].min()) == 3.0 and float(c.layers[1]["conv"][1].min()) == 2.0 and c.layers[0]["v"].shape[0] == 4
    with pytest.raises(ValueError, match="different names"):
        HybridCache([GroupSpec((StateSpec(1, 8, 8), DeltaSpec(1, 8, 8, 24, 2)))], 1, 8, torch.float32, "cpu")
    c.advance([0, 2], [5, 63])
    p = c.plan([0, 2, 1], [2, 3, 1]).kv()                    # positions 5..6, 63..65 and 0
    assert p.home_rows.tolist() == [5, 6, 263, 264, 265, 100] and p.n_keys.tolist() == [6, 7, 64, 65, 66, 1]
    assert p.row0.tolist() == [0, 0, 200, 200, 200, 100] and p.kv_lens.tolist() == [7, 66, 1] and p.q_pos0.tolist() == [5, 63, 0]
    assert p.block_table.tolist() == [[0], [2], [1]] and p.max_q == 3 and p.max_kv == 66
    q = c.plan([2, 0], [1, 1]).kv()
    assert q.home_rows.tolist() == [263, 5] and q.kv_lens.tolist() == [64, 6] and q.row0.tolist() == [200, 0]


def test_rope_table_with_scaling():
    from triton_distributed_b200 import ops

    r = cases.rot(12, 60.0, **cases.YARN)
    y = ops.YarnScaling.from_json(r["scaling"])
    t = ops.rope_table(60.0, 12, 16, 5000, "cpu", y)
    f, mult = oracle.frequencies(r)
    for p in (0, 1, 47, 4999):
        for i in range(6):
            assert abs(float(t[p, 2 * i]) - mult * math.cos(p * f[i])) < 1e-6 and abs(float(t[p, 2 * i + 1]) - mult * math.sin(p * f[i])) < 1e-6
    assert float(t[:, 12:].abs().max()) == 0
    assert ops.rope_table(60.0, 12, 16, 10, "cpu") is not t and ops.rope_table(60.0, 12, 16, 10, "cpu", y) is t
    assert ops.YarnScaling.from_json(None) is None


# ------------------------------------------------------------------ generation
def test_greedy_generation_through_serve(rt, tmp_path):
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=3)
    eng = cases.engine(cases.write(tmp_path, cfg, w), torch.float32, max_length=64)
    prompts = [cases.prompt(cfg, 22, s) for s in range(3)]
    want = [cases.greedy(cfg, w, p, 6) for p in prompts]
    assert min(g for _, g in want) > 1e-3
    assert eng.serve(torch.tensor(prompts), 6).tolist() == [t for t, _ in want]
    # unequal prompts, right-padded: the same continuations as alone
    lens = [22, 5, 13]
    short = [cases.greedy(cfg, w, p[:n], 6)[0] for p, n in zip(prompts, lens)]
    assert eng.serve(torch.tensor(prompts), 6, seq_lens=lens).tolist() == short
    # sampling goes through the engine as for the other models
    hot = cases.engine(tmp_path, torch.float32, max_length=64, temperature=0.8, top_p=0.9, seed=5)
    assert hot.serve(torch.tensor(prompts), 4).shape == (3, 4)


def test_trace_replay(mixed, tmp_path):
    from triton_distributed_b200.models import trace

    d, _, toks, want = mixed
    eng = trace.make_engine(str(d), torch.float32, 64)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:40], "want": [3, 39]}, {"id": "b", "tokens": toks[:9], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [toks[9]], "want": []}, {"id": "a", "tokens": [toks[40]], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [toks[41]], "want": [0]}], "end": ["a"]}]
    out = io.StringIO()
    trace.replay(eng, [json.dumps(s) + "\n" for s in steps], str(tmp_path), out)
    assert out.getvalue().split("\n") == ["done 0", "done 1", "done 2", ""]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, 101)   # noqa: E731
    assert cases.rel(read(0), want[[3, 39]]) < TOL and cases.rel(read(2), want[[41]]) < TOL
    assert not (tmp_path / "1.f32").exists() and not eng._step_slots


# ------------------------------------------------------------------ tensor parallelism
TP = cases.config([("parallel", {"left": cases.attn(4, 2, 12, 16, 8), "right": cases.delta(4, 2, 8, 12, 3)}, 40), ("attention", cases.attn(4, 4, 16, 8, cap=5.0), 24),
                   ("attention_2", cases.attn(6, 2, 10, 12, 6, factor=2.0, original=16, fast=4.0, slow=1.0), None)], 48, 77, streams=2, loop=(0, 2, 2))


def _tp_rank(rank, world, d, toks):
    import tazitar_cases as cases_
    import tazitar_oracle as oracle_

    w = cases_.weights(TP, seed=9)
    for backend in ("torch", "triton_dist_AR", "triton_dist_gemm_ar", "triton_dist"):
        eng = cases_.engine(d, torch.float32, max_length=64)
        eng.backend = backend
        got = cases_.run_portions(eng, 0, toks, [20, 1])
        assert cases_.rel(got, oracle_.forward(TP, w, toks)) < TOL, backend
        eng.no_graph = True
        assert eng.serve(torch.tensor([toks[:10], toks[10:20]]), 3).shape == (2, 3)


def test_two_ranks_match_the_oracle(tmp_path):
    cases.write(tmp_path, TP, cases.weights(TP, seed=9))
    run_cpu_ranks(_tp_rank, 2, (str(tmp_path), cases.prompt(TP, 27)))


def test_heads_that_cannot_be_split():
    from triton_distributed_b200.models.tazitar import DeltaRuleSpec, RotaryAttnSpec
    from triton_distributed_b200.parallel import TP_DeltaRule, TP_RotaryAttn

    with pytest.raises(ValueError, match="KV heads"):
        TP_RotaryAttn(RotaryAttnSpec(4, 1, 8, 8, 1.0, 1e4, 8), 0, 2)
    with pytest.raises(ValueError, match="key heads"):
        TP_DeltaRule(DeltaRuleSpec(6, 3, 8, 8, 4), 0, 2)


# ------------------------------------------------------------------ the tests' own sharpness
def _mistakes():
    o = {n: getattr(oracle, n) for n in ("rotate", "frequencies", "softmax", "head_scores", "queries_keys", "short_conv", "unit", "delta_step",
                                         "delta_inputs", "hyper", "passes", "mixer_out", "rms", "softplus")}

    def capless(q, k, mixer):
        return (k @ q) * mixer["scale"]

    def cap_before_scale(q, k, mixer):
        cap = mixer.get("softcap")
        return cap * torch.tanh((k @ q) / cap) * mixer["scale"] if cap else (k @ q) * mixer["scale"]

    def norms_before_rotation(h, W, p, mixer, eps, kind):
        if not oracle.KINDS[kind]["unit"]:
            return o["queries_keys"](h, W, p, mixer, eps, kind)
        out = []
        for name, n in (("q", mixer["heads"]), ("k", mixer["kv_heads"])):
            x = oracle.rms((h @ W[p + name].T).reshape(h.shape[0], n, mixer["dim"]), eps)
            out.append(torch.stack([oracle.rotate(x[t], t, mixer["rot"], oracle.KINDS[kind]["interleaved"]) for t in range(h.shape[0])]))
        return out

    def late_conv(x, w):                       # the current token's tap is missing, everything one token late
        return torch.cat([torch.zeros_like(x[:1]), o["short_conv"](x, w)[:-1]])

    def old_readout(S, q, k, v, g, beta):
        new, _ = o["delta_step"](S, q, k, v, g, beta)
        return new, torch.einsum("hkv,hk->hv", g[:, None, None] * S, q)

    def undecayed_answer(S, q, k, v, g, beta):
        u = beta[:, None] * (v - torch.einsum("hkv,hk->hv", S, k))
        S = g[:, None, None] * S + k[:, :, None] * u[:, None, :]
        return S, torch.einsum("hkv,hk->hv", S, q)

    def inputs(change):
        def f(h, W, p, mixer):
            return change(*o["delta_inputs"](h, W, p, mixer), h, W, p, mixer)
        return f

    def hyper(change):
        def f(x, W, p, sub):
            return o["hyper"](x, {**W, **change(W, p)}, p, sub)
        return f

    def unhalved(h, W, p, layer, eps):
        return (2.0 if layer["type"] == "parallel" else 1.0) * o["mixer_out"](h, W, p, layer, eps)

    def layer_by_layer(config):                # every looped layer twice in a row
        a, b, n = config["loop"]["start"], config["loop"]["stop"], config["loop"]["times"]
        return list(range(a)) + [i for i in range(a, b) for _ in range(n)] + list(range(b, len(config["layers"])))

    return [("rotate", lambda x, pos, rot, inter: o["rotate"](x, pos, rot, not inter)),
            ("rotate", lambda x, pos, rot, inter: o["rotate"](x, pos + 1, {**rot, "base": rot["base"] * 2}, inter)),
            ("frequencies", lambda rot: o["frequencies"]({"base": rot["base"], "dims": rot["dims"]})),
            ("softmax", lambda s, sink=None: o["softmax"](s)),
            ("softmax", lambda s, sink=None: o["softmax"](s, None if sink is None else sink + 1.5)),
            ("head_scores", capless), ("head_scores", cap_before_scale), ("queries_keys", norms_before_rotation),
            ("visible", lambda i, j: j < i or i == j == 0),
            ("short_conv", late_conv), ("short_conv", lambda x, w: o["short_conv"](x, w.flip(1))),
            ("unit", lambda x: x), ("delta_step", old_readout), ("delta_step", undecayed_answer),
            ("delta_inputs", inputs(lambda q, k, v, g, b, *a: (q, k, v, torch.ones_like(g), b))),
            ("delta_inputs", inputs(lambda q, k, v, g, b, *a: (q, k, v, g, torch.ones_like(b)))),
            ("delta_inputs", inputs(lambda q, k, v, g, b, h, W, p, m: (q.roll(1, 1), k.roll(1, 1), v, g, b))),
            ("delta_inputs", inputs(lambda q, k, v, g, b, h, W, p, m: (q, k, v, torch.exp(-oracle.softplus(h @ W[p + "a"].T + W[p + "dt_bias"])), b))),
            ("hyper", hyper(lambda W, p: {p + "mix": W[p + "mix"].T})), ("hyper", hyper(lambda W, p: {p + "in": W[p + "in"].flip(0)})),
            ("hyper", hyper(lambda W, p: {p + "out": torch.ones_like(W[p + "out"])})),
            ("mixer_out", unhalved), ("passes", layer_by_layer), ("rms", lambda x, eps, w=None: o["rms"](x, 0.0, w))]


@pytest.mark.parametrize("i", range(24))
def test_a_mistake_in_one_mechanism_shows(i, mixed, monkeypatch):
    """A fault of one mechanism moves logits far beyond the tolerances used here (and those of fp32 on the GPU)."""
    _, w, toks, want = mixed
    name, wrong = _mistakes()[i]
    monkeypatch.setattr(oracle, name, wrong)
    got = oracle.forward(cases.MIXED, w, toks)
    print(name, cases.rel(got, want))
    assert cases.rel(got, want) > (0.02 if name == "rms" else 0.15), name
