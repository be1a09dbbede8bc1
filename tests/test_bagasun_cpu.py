"""Bagasun on CPU ranks (fp32): configuration, weights, cache plans, engine steps, generation, tensor parallelism.  The kernels are
covered by test_bagasun_gpu.py; here the host logic runs over the ops' CPU backend."""
import io
import json
import math

import pytest
import torch

import bagasun_cases as cases
import bagasun_oracle as oracle
from dist_utils import run_cpu_ranks

TOL = 3e-5


@pytest.fixture(scope="module")
def rt():
    import triton_distributed_b200 as tdb

    tdb.initialize_distributed(seed=0, device="cpu")
    yield tdb.get_runtime()
    tdb.finalize_distributed()


@pytest.fixture(scope="module")
def mixed(rt, tmp_path_factory):
    w = cases.weights(cases.MIXED, seed=1, gain=0.6)
    d = cases.write(tmp_path_factory.mktemp("mixed"), cases.MIXED, w)
    toks = cases.prompt(cases.MIXED, 61)
    return d, w, toks, oracle.forward(cases.MIXED, w, toks)


# ------------------------------------------------------------------ the oracle itself
def test_oracle_rotation():
    rot = {"base": 100.0, "dims": 6}
    x = torch.tensor([1.0, 0.0, 0.5, 2.0, 3.0, 4.0, 7.0, -1.0], dtype=torch.float64)
    y = oracle.rotate(x, 5, rot)
    for i in range(3):
        ang = 5 * 100.0 ** (-2 * i / 6)
        turned = complex(x[i], x[i + 3]) * complex(math.cos(ang), math.sin(ang))
        assert abs(turned - complex(y[i], y[i + 3])) < 1e-12
    assert torch.equal(y[6:], x[6:]) and torch.equal(oracle.rotate(x, 0, rot), x)


def test_oracle_scaled_frequencies():
    """Short wavelengths keep their frequency, long ones are divided by the factor, and the values between them are monotone."""
    rot = {"base": 1e4, "dims": 64}
    plain = oracle.frequencies(rot)
    ratio = [a / b for a, b in zip(oracle.frequencies({**rot, "scaling": dict(factor=8.0, original=2048, low=1.0, high=4.0)}), plain)]
    assert all(x >= y - 1e-15 for x, y in zip(ratio, ratio[1:])) and any(0.2 < r < 0.9 for r in ratio)
    for r, f in zip(ratio, plain):
        turns = 2048 * f / (2 * math.pi)
        if turns > 4:
            assert r == 1.0
        if turns < 1:
            assert abs(r - 1 / 8) < 1e-15


def test_oracle_weights_and_windows():
    one = torch.ones((), dtype=torch.float64)
    q, k = torch.tensor([2.0, 0.0], dtype=torch.float64), torch.tensor([[1.0, 5.0], [0.0, 1.0]], dtype=torch.float64)
    w = oracle.sigmoid_weights(q, k, torch.tensor([3.0, 0.0]), 0.5, 2 * one, one, 0.25 * one)
    assert torch.allclose(w, 1 / (1 + torch.exp(-torch.tensor([1.0 - 2 * math.log(4.0) + 0.25, 0.25], dtype=torch.float64))))
    assert [j for j in range(9) if oracle.visible(5, j, 3)] == [3, 4, 5] and [j for j in range(9) if oracle.visible(2, j, 0)] == [0, 1, 2]
    a, b = torch.tensor([3.0, 1.0], dtype=torch.float64), torch.tensor([1.0, 1.0], dtype=torch.float64)
    assert torch.allclose(oracle.combine_maps(a, b, 1.0, 0.25, 0.0), torch.tensor([math.sqrt(2.0), 0.0], dtype=torch.float64) * 0.75)


def test_oracle_state_space_step():
    """Without decay the state sums dt B x^T; the read-out sees the write; the skip adds the input."""
    t = lambda *v: torch.tensor(v, dtype=torch.float64)   # noqa: E731
    S, y = oracle.ssd_step(torch.zeros(1, 2, 1, dtype=torch.float64), t([3.0]), t([1.0, 2.0]), t([10.0, 100.0]), t(0.5), t(0.0), t(7.0))
    assert S.flatten().tolist() == [1.5, 3.0] and y.item() == 15.0 + 300.0 + 21.0
    S, y = oracle.ssd_step(S, t([0.0]), t([1.0, 2.0]), t([1.0, 0.0]), t(2.0), t(math.log(2.0)), t(0.0))
    assert torch.allclose(S.flatten(), t(1.5 / 4, 3.0 / 4)) and abs(y.item() - 1.5 / 4) < 1e-12
    x, w = t([1.0], [10.0], [100.0], [1000.0]), t([2.0, 3.0, 5.0])                 # two back, one back, current
    assert oracle.short_conv(x, w, t(1.0)).flatten().tolist() == [6.0, 54.0, 533.0, 5321.0]
    z = t(-50.0, -1.0, 0.0, 3.0, 60.0)
    assert torch.allclose(oracle.softplus(z), torch.log1p(torch.exp(z)), atol=1e-15)


# ------------------------------------------------------------------ configuration and registry
def test_configuration_is_read_and_checked(mixed, tmp_path):
    from triton_distributed_b200 import ops
    from triton_distributed_b200.models import BagasunConfig, ModelConfig

    a = ModelConfig(checkpoint_dir=str(mixed[0])).arch()
    assert isinstance(a, BagasunConfig) and (a.vocab_size, a.hidden_size, a.embed_scale, a.rms_norm_eps) == (101, 60, 1.7, 2e-3)
    assert a.num_hidden_layers == 11 and not a.is_moe and [a.source(i) for i in range(11)] == [0, 1, 2, 1, 4, 0, 0, 7, 8, 2, 8]
    m = a.layers[5].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.window) == (6, 3, 20, 28, 9)
    m = a.layers[2].mixer
    assert (m.diff, m.rot_base, m.rot_dims, m.window) == (0.3, 300.0, 10, 7) and m.scaling == ops.BandScaling(3.0, 40.0, 0.7, 3.0) and a.layers[2].mlp is None
    assert a.layers[8].mixer.window == 0 and a.layers[8].mixer.scaling is None
    m = a.layers[3].mixer
    assert (m.heads, m.groups, m.state, m.vdim, m.conv, m.norm_groups) == (6, 2, 12, 20, 3, 3) and a.layers[3].mlp.ff == 42

    def broken(i=0, mixer=None, mlp=None, layer=None, **change):
        c = json.loads(json.dumps(cases.PLAIN))
        c["layers"][i].update(layer or {})
        c["layers"][i]["mixer"].update(mixer or {})
        if mlp:
            c["layers"][i]["mlp"].update(mlp)
        c.update(change)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return BagasunConfig.from_json(str(tmp_path))

    assert broken(2, mixer={"mask": None}).layers[2].mixer.window == 0
    for kw, what in ((dict(layer={"type": "other"}), "mixer"), (dict(i=2, mlp={"kind": "other"}), "kind"), (dict(i=2, mixer={"heads": 5}), "multiple"),
                     (dict(i=2, mixer={"mask": {"size": 0}}), "window"), (dict(i=1, mixer={"rot": {"base": 10.0, "dims": 18}}), "rotation"),
                     (dict(i=1, mixer={"rot": {"base": 10.0, "dims": 5}}), "rotation"), (dict(mixer={"groups": 3}), "multiple"), (dict(mixer={"conv": 0}), "tap"),
                     (dict(mixer={"norm_groups": 7}), "norm_groups"), (dict(i=3, mixer={"heads": 2}), "sizes differ"), (dict(i=2, layer={"weights_of": 0}), "sizes differ"),
                     (dict(i=0, layer={"weights_of": 3}), "does not lead"), (dict(i=3, layer={"weights_of": 9}), "does not lead")):
        with pytest.raises(ValueError, match=what):
            broken(**kw)


def test_registry_presets_and_limits(rt):
    from triton_distributed_b200.models import BAGASUN_PRESETS, AutoLLM, BagasunLLM, ModelConfig
    from triton_distributed_b200.models.bagasun import SigmoidAttnSpec, StateSpaceSpec
    from triton_distributed_b200.parallel import TP_SigmoidAttn, TP_StateSpace

    m = AutoLLM.from_pretrained(ModelConfig(model_name="tiny-bagasun", dtype=torch.float32))
    assert isinstance(m, BagasunLLM) and len(m.cache_specs()) == 8
    assert [m.layers[i].mixer is m.layers[i % 4].mixer for i in range(8)] == [True] * 8 and m.layers[4].mixer is not m.layers[5].mixer
    out = m.inference(torch.tensor([[3, 5, 9]]), torch.arange(3)[None], m.new_cache(1, 8))
    assert out.shape == (1, 1000) and torch.isfinite(out).all()
    short = ModelConfig(model_name="tiny-bagasun", num_layers_override=5).arch()
    assert short.num_hidden_layers == 5 and short.source(4) == 0
    assert BAGASUN_PRESETS["tiny-bagasun"].with_num_layers(11).num_hidden_layers == 11
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        AutoLLM.from_pretrained(ModelConfig(model_name="tiny-bagasun", dtype=torch.float16))
    with pytest.raises(ValueError, match="256"):
        TP_StateSpace(StateSpaceSpec(2, 2, 300, 16, 4, 1))
    with pytest.raises(ValueError, match="1024"):
        TP_SigmoidAttn(SigmoidAttnSpec(2, 2, 1100, 16, 1.0))
    dims = [(lambda t: (t.dk, t.dv))(TP_SigmoidAttn(SigmoidAttnSpec(2, 2, d, v, 1.0))) for d, v in ((8, 8), (44, 72), (64, 64), (100, 16), (130, 20), (30, 300))]
    assert dims == [(64, 64), (64, 128), (64, 64), (128, 64), (136, 24), (32, 304)]


def test_weights_with_one_number_survive_the_checkpoint_format(tmp_path):
    from triton_distributed_b200.models import SafetensorsFile, save_file

    save_file({"a": torch.tensor(2.5, dtype=torch.bfloat16), "b": torch.tensor(-1.0)}, str(tmp_path / "x.safetensors"))
    f = SafetensorsFile(str(tmp_path / "x.safetensors"))
    assert f.get("a").shape == () and float(f.get("a")) == 2.5 and float(f.get("b")) == -1.0


# ------------------------------------------------------------------ forward
def test_prompt_matches_oracle_layer_by_layer(mixed):
    d, w, toks, want = mixed
    eng = cases.engine(d, torch.float32)
    streams, ref = [], []
    oracle.forward(cases.MIXED, w, toks, ref)
    cache = eng.model.new_cache(1, 64)
    got = eng.model.forward_step(torch.tensor(toks), cache.plan([0], [len(toks)]), None, False, streams)
    assert len(streams) == len(ref) == 11
    for a, b in zip(streams, ref):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)
    assert cases.rel(got, want) < TOL


@pytest.mark.parametrize("sizes", [[2], [1], [7], [24, 1], [17, 3, 50], [60, 1], [5, 40]])
@pytest.mark.parametrize("max_length", [256, 61])
def test_portions_of_any_size(mixed, sizes, max_length):
    d, _, toks, want = mixed
    assert cases.rel(cases.run_portions(cases.engine(d, torch.float32, max_length=max_length), "r", toks, sizes), want) < TOL


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
    from triton_distributed_b200.models import DeltaSpec, HybridCache, WindowKVSpec

    near, far = WindowKVSpec(2, 128, 64, 5), WindowKVSpec(1, 64, 64)
    c = HybridCache([near, far, DeltaSpec(3, 16, 32, 160, 4)], 3, 100, torch.bfloat16, "cpu")
    assert c.layers[0]["k"].shape == (3, 5, 2, 128) and c.layers[0]["v"].shape == (3, 5, 2, 64) and c.layers[1]["k"].shape == (3, 100, 1, 64)
    assert WindowKVSpec(1, 8, 8, 200).rows(100) == 100
    c.advance([0, 2], [7, 3])
    p = c.plan([0, 2, 1], [2, 7, 1])                         # positions 7..8, 3..9 and 0
    w = p.window(near)
    assert p.window(WindowKVSpec(2, 64, 64, 5)) is w and p.window(far) is not w
    # slot 0 still sees positions 3..6 of its ring, slot 2 all of 0..2
    assert w.carry_src.tolist() == [3, 4, 0, 1] + [10, 11, 12] and w.carry_dst.tolist() == [0, 1, 2, 3] + [6, 7, 8]
    assert w.packed_rows.tolist() == [4, 5] + list(range(9, 16)) + [16] and w.total == 17 and w.max_q == 7
    assert w.home_rows.tolist() == [2, 3] + [-1, -1, 10, 11, 12, 13, 14] + [5]
    assert w.q_pos0.tolist() == [7, 3, 0] and w.shift.tolist() == [-3, 6, 16]
    row0, n, own = w.visible()
    assert row0.tolist() == [0, 1] + [6, 6, 7, 8, 9, 10, 11] + [16] and n.tolist() == [5, 5, 4, 5, 5, 5, 5, 5, 5, 1] and own.tolist() == [k - 1 for k in n.tolist()]
    f = p.window(far)
    assert f.total == 9 + 10 + 1 and f.home_rows.tolist() == [7, 8] + [203 + i for i in range(7)] + [100] and f.shift.tolist() == [0, 9, 19]
    q = c.plan([2, 0], [1, 1]).window(near)                  # positions 3 and 7
    assert q.home_rows.tolist() == [13, 2] and [t.tolist() for t in q.visible()] == [[10, 0], [4, 5], [3, 2]]


def test_rope_table_with_band_scaling():
    from triton_distributed_b200 import ops

    for sc in (cases.BAND, dict(factor=4.0, original=64, low=2.0, high=2.0)):
        rot = {"base": 60.0, "dims": 12, "scaling": sc}
        y = ops.BandScaling.from_json(sc)
        t = ops.rope_table(60.0, 12, 16, 5000, "cpu", y)
        f = oracle.frequencies(rot) if sc["low"] < sc["high"] else [b if b * 64 / (2 * math.pi) > 2 else b / 4 for b in oracle.frequencies({"base": 60.0, "dims": 12})]
        for p in (0, 1, 47, 4999):
            for i in range(6):
                assert abs(float(t[p, 2 * i]) - math.cos(p * f[i])) < 1e-6 and abs(float(t[p, 2 * i + 1]) - math.sin(p * f[i])) < 1e-6
    assert ops.BandScaling.from_json(None) is None


def test_decode_splits():
    from triton_distributed_b200 import ops

    for batch in (1, 3, 8, 64, 500):
        for units in (1, 4, 8):
            for rows in (1, 64, 65, 1024, 100000):
                assert 1 <= ops.pick_window_splits(batch, units, rows) <= min(32, (rows + 63) // 64)
    assert ops.pick_window_splits(1, 8, 4096) > 8 and ops.pick_window_splits(500, 8, 64) == 1


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
TP = cases.config([("mamba2", cases.mamba(4, 2, 8, 12, 3, 4), 40), ("attention", cases.attn(4, 2, 12, 16, 9), 24), ("attention_2", cases.diff(6, 2, 10, 12, 6, 6, **cases.BAND), None),
                   0, 1], 48, 77, scale=2.0)


def _tp_rank(rank, world, d, toks):
    import bagasun_cases as cases_
    import bagasun_oracle as oracle_

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


def test_sizes_that_cannot_be_split():
    from triton_distributed_b200.models.bagasun import SigmoidAttnSpec, StateSpaceSpec
    from triton_distributed_b200.parallel import TP_SigmoidAttn, TP_StateSpace

    with pytest.raises(ValueError, match="KV heads"):
        TP_SigmoidAttn(SigmoidAttnSpec(4, 1, 8, 8, 1.0), 0, 2)
    with pytest.raises(ValueError, match="groups"):
        TP_StateSpace(StateSpaceSpec(4, 1, 8, 8, 4, 2), 0, 2)
    with pytest.raises(ValueError, match="groups"):
        TP_StateSpace(StateSpaceSpec(4, 2, 8, 8, 4, 1), 0, 2)


# ------------------------------------------------------------------ the tests' own sharpness
def _mistakes():
    o = {n: getattr(oracle, n) for n in ("rotate", "frequencies", "softmax", "sigmoid_weights", "distance_bias", "projection", "mix_of_maps", "combine_maps", "short_conv",
                                         "ssd_step", "gated_group_norm", "sandwich", "rms", "visible", "window_of", "softplus", "weights_layer")}

    def interleaved(x, pos, rot):
        half, out = rot["dims"] // 2, x.clone()
        for i, f in enumerate(o["frequencies"](rot)):
            c, s = math.cos(pos * f), math.sin(pos * f)
            out[..., 2 * i], out[..., 2 * i + 1] = x[..., 2 * i] * c - x[..., 2 * i + 1] * s, x[..., 2 * i + 1] * c + x[..., 2 * i] * s
        return out

    def normalised(*a):
        w = o["sigmoid_weights"](*a)
        return w / w.sum()

    def norm_before_gate(y, z, groups, w, eps):
        return oracle.rms(y.reshape(y.shape[0], groups, -1), eps).reshape(y.shape) * w * oracle.silu(z)

    def old_readout(S, x, B, C, dt, a, D):
        new, _ = o["ssd_step"](S, x, B, C, dt, a, D)
        return new, torch.einsum("hnv,hn->hv", S, C) + D[:, None] * x

    def unstepped(S, x, B, C, dt, a, D):
        S = torch.exp(-a * dt)[:, None, None] * S + B[:, :, None] * x[:, None, :]
        return S, torch.einsum("hnv,hn->hv", S, C) + D[:, None] * x

    def only_before(x, W, p, n, eps, sub):
        return x + sub(o["rms"](x, eps, W[f"{p}norm{n}"])) * W[f"{p}norm{n}b"]

    def only_after(x, W, p, n, eps, sub):
        return x + o["rms"](sub(x * W[f"{p}norm{n}"]), eps, W[f"{p}norm{n}b"])

    return [("rotate", interleaved), ("rotate", lambda x, pos, rot: x), ("frequencies", lambda rot: o["frequencies"]({"base": rot["base"], "dims": rot["dims"]})),
            ("visible", lambda i, j, w: o["visible"](i, j, w + 1 if w else 0)), ("visible", lambda i, j, w: o["visible"](i, j, max(1, w - 1) if w else 0)),
            ("visible", lambda i, j, w: o["visible"](i, j, w) or j == 0 <= i), ("window_of", lambda m: 0),
            ("sigmoid_weights", normalised), ("sigmoid_weights", lambda q, k, d, s, r1, r2, pb: o["sigmoid_weights"](q, k, d, s, r1, r2, 0 * pb)),
            ("sigmoid_weights", lambda q, k, d, s, r1, r2, pb: o["softmax"]((k @ q) * s - o["distance_bias"](d, r1, r2) + pb)),
            ("distance_bias", lambda d, r1, r2: 0 * d), ("distance_bias", lambda d, r1, r2: o["distance_bias"](d + 1, r1, r2)),
            ("distance_bias", lambda d, r1, r2: o["distance_bias"](d, r2, r1)), ("projection", lambda h, W, n: h @ W[n].T),
            ("mix_of_maps", lambda W, p, diff: torch.zeros((), dtype=oracle.DT)), ("mix_of_maps", lambda W, p, diff: o["mix_of_maps"](W, p, 0.0)),
            ("combine_maps", lambda a, b, lam, diff, eps: o["combine_maps"](a, b, lam, 0.0, eps)), ("combine_maps", lambda a, b, lam, diff, eps: (a - lam * b) * (1 - diff)),
            ("short_conv", lambda x, w, b: o["short_conv"](x, w.flip(1), b)), ("short_conv", lambda x, w, b: o["short_conv"](x, w, 0 * b)),
            ("ssd_step", old_readout), ("ssd_step", unstepped), ("ssd_step", lambda S, x, B, C, dt, a, D: o["ssd_step"](S, x, B, C, dt, a, 0 * D)),
            ("ssd_step", lambda S, x, B, C, dt, a, D: o["ssd_step"](S, x, B.roll(1, 0), C.roll(1, 0), dt, a, D)),
            ("ssd_step", lambda S, x, B, C, dt, a, D: o["ssd_step"](S, x, B, C, dt, 0 * a, D)),
            ("gated_group_norm", norm_before_gate), ("gated_group_norm", lambda y, z, g, w, eps: o["gated_group_norm"](y, z, 1, w, eps)),
            ("sandwich", only_before), ("sandwich", only_after), ("rms", lambda x, eps, w=None: o["rms"](x, 0.0, w))]


@pytest.mark.parametrize("i", range(30))
def test_a_mistake_in_one_mechanism_shows(i, mixed, monkeypatch):
    """A fault of one mechanism moves logits far beyond the tolerances used here (and those of fp32 on the GPU)."""
    _, w, toks, want = mixed
    name, wrong = _mistakes()[i]
    monkeypatch.setattr(oracle, name, wrong)
    got = oracle.forward(cases.MIXED, w, toks)
    print(name, cases.rel(got, want))
    assert cases.rel(got, want) > (0.02 if name == "rms" else 0.08), name


def test_the_list_of_mistakes_is_covered():
    assert len(_mistakes()) == 30
