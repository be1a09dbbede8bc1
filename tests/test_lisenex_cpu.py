"""Lisenex on CPU ranks (fp32): configuration, weights, cache plans, engine steps, generation, tensor parallelism.  The kernels
are covered by test_lisenex_gpu.py; here the host logic runs over the ops' CPU backend."""
import io
import json
import math

import pytest
import torch

import lisenex_cases as cases
import lisenex_oracle as oracle
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
def test_oracle_rotation():
    x = torch.tensor([1.0, 0.0, 0.0, 2.0, 3.0, 4.0], dtype=torch.float64)
    y = oracle.rotate(x, 5, 100.0)
    for i in range(3):
        a = 5 * 100.0 ** (-2 * i / 6)
        turned = complex(x[2 * i], x[2 * i + 1]) * complex(math.cos(a), math.sin(a))
        assert abs(turned - complex(y[2 * i], y[2 * i + 1])) < 1e-12
    assert torch.equal(oracle.rotate(x, 0, 100.0), x)
    # scores of rotated vectors depend on the distance alone
    q, k = torch.randn(6, dtype=torch.float64), torch.randn(6, dtype=torch.float64)
    near = oracle.rotate(q, 9, 50.0) @ oracle.rotate(k, 4, 50.0)
    far = oracle.rotate(q, 1009, 50.0) @ oracle.rotate(k, 1004, 50.0)
    assert abs(float(near - far)) < 1e-9


def test_oracle_choice():
    z = torch.log(torch.tensor([0.4, 0.1, 0.05, 0.2, 0.15, 0.1], dtype=torch.float64))
    none = torch.zeros(6, dtype=torch.float64)
    ids, w = oracle.route(z, none, 2)
    assert ids == [0, 3] and torch.allclose(w, torch.tensor([0.4, 0.2], dtype=torch.float64))
    # the correction moves the choice, not the weights
    ids, w = oracle.route(z, torch.tensor([-0.5, 0, 0, 0, 0.1, 0], dtype=torch.float64), 2)
    assert ids == [4, 3] and torch.allclose(w, torch.tensor([0.15, 0.2], dtype=torch.float64))
    # all choice scores negative: experts of groups left out still lose
    ids, w = oracle.route(z, torch.tensor([-1.0] * 6, dtype=torch.float64), 2, {"count": 3, "keep": 1})
    assert ids == [0, 1] and torch.allclose(w, torch.tensor([0.4, 0.1], dtype=torch.float64))


# ------------------------------------------------------------------ configuration and registry
def test_configuration_is_read_and_checked(mixed, tmp_path):
    from triton_distributed_b200.models import LisenexConfig, ModelConfig

    a = ModelConfig(checkpoint_dir=str(mixed[0])).arch()
    assert isinstance(a, LisenexConfig) and a.vocab_size == 101 and a.hidden_size == 60 and a.num_hidden_layers == 6
    assert a.embedding_scale == 0.6 and a.layers[2].mlp is None and a.layers[1].mlp.ff == 50 and a.layers[1].mixer.kv_from == 0
    m = a.layers[3].mlp
    assert (m.experts, m.identity, m.top, m.ff, m.shared_ff, m.groups, m.keep) == (4, 2, 3, 20, 16, 0, 0)
    assert a.layers[4].mixer.rot_base == 90.0 and a.layers[4].mlp.shared_ff == 0 and a.layers[4].mlp.keep == 2

    def broken(i=0, mixer=None, mlp=None, **change):
        c = json.loads(json.dumps(cases.MIXED))
        c["layers"][i].update(change)
        c["layers"][i]["mixer"].update(mixer or {})
        if mlp:
            c["layers"][i]["mlp"].update(mlp)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return LisenexConfig.from_json(str(tmp_path))

    with pytest.raises(ValueError, match="mixer"):
        broken(type="other")
    with pytest.raises(ValueError, match="kind"):
        broken(mlp={"kind": "other"})
    with pytest.raises(ValueError, match="rotated part"):
        broken(mixer={"rot": {"base": 10.0, "dims": 4}})
    for j in (0, 1, 2, 9):                                  # itself, a later one, one without rows, none
        with pytest.raises(ValueError, match="kv_from"):
            broken(0 if j < 2 else 5, mixer={"kv_from": 1 if j == 2 else j})
    for other in ({"kv_rank": 48}, {"rot": {"base": 7.0, "dims": 8}}):
        with pytest.raises(ValueError, match="rank and rotation"):
            broken(1, mixer=other)
    with pytest.raises(ValueError, match="groups"):
        broken(mlp={"router": {"experts": 5, "top": 2, "identity": 0, "groups": {"count": 2, "keep": 1}}})
    with pytest.raises(ValueError, match="cannot be chosen"):
        broken(mlp={"router": {"experts": 5, "top": 3, "identity": 1, "groups": {"count": 3, "keep": 1}}})


def test_registry_and_presets(rt):
    from triton_distributed_b200.models import LISENEX_PRESETS, AutoLLM, LisenexLLM, ModelConfig

    m = AutoLLM.from_pretrained(ModelConfig(model_name="tiny-lisenex", dtype=torch.float32, num_layers_override=6))
    assert isinstance(m, LisenexLLM) and [l.mixer.source for l in m.layers] == [0, 0, 2, 2, 4, 4]
    assert m.layers[4].mixer.shared and m.layers[3].mlp is None and m.layers[5].spec.mlp == m.layers[1].spec.mlp
    assert all(c.is_moe for c in LISENEX_PRESETS.values())
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        AutoLLM.from_pretrained(ModelConfig(model_name="tiny-lisenex", dtype=torch.float16))
    big = cases.latent(1, 8, 8, 8, 1100)
    from triton_distributed_b200.models.lisenex import LatentAttnSpec
    from triton_distributed_b200.parallel import TP_LatentAttn
    with pytest.raises(ValueError, match="1024"):
        TP_LatentAttn(LatentAttnSpec.from_json(big), 0)


# ------------------------------------------------------------------ forward
def test_prompt_matches_oracle_layer_by_layer(mixed):
    d, w, toks, want = mixed
    eng = cases.engine(d, torch.float32)
    streams, ref = [], []
    oracle.forward(cases.MIXED, w, toks, ref)
    cache = eng.model.new_cache(1, 64)
    got = eng.model.forward_step(torch.tensor(toks), cache.plan([0], [len(toks)]), None, False, streams)
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
    from triton_distributed_b200.models import HybridCache, LatentSpec, SharedSpec

    c = HybridCache([LatentSpec(40, 8), SharedSpec(0), LatentSpec(16, 8), SharedSpec(0)], 2, 100, torch.float32, "cpu")
    assert c.layers[1] is c.layers[0] and c.layers[3] is c.layers[0] and c.layers[2]["latent"].shape == (2, 100, 24)
    c.layers[0]["latent"][1] = 3.0
    assert c.alloc() == 2 and c.capacity == 4                # grows: what is there stays, sharers see the new storage
    assert c.layers[3] is c.layers[0] and c.layers[0]["latent"].shape == (4, 100, 48) and float(c.layers[3]["latent"][1].min()) == 3.0
    for specs in ([SharedSpec(0)], [LatentSpec(8, 8), SharedSpec(0), SharedSpec(1)], [LatentSpec(8, 8), SharedSpec(2)]):
        with pytest.raises(ValueError, match="share"):
            HybridCache(specs, 1, 8, torch.float32, "cpu")
    c.advance([0, 2], [5, 63])
    p = c.plan([0, 2, 1], [2, 3, 1]).latent()                # positions 5..6, 63..65 and 0
    assert p.home_rows.tolist() == [5, 6, 263, 264, 265, 100] and p.n_keys.tolist() == [6, 7, 64, 65, 66, 1]
    assert p.row0.tolist() == [0, 0, 200, 200, 200, 100] and p.kv_lens.tolist() == [7, 66, 1] and p.q_pos0.tolist() == [5, 63, 0]
    assert p.ctx0.tolist() == [0, 64, 192] and p.ctx_len == 256 and p.ctx_rows.tolist() == [5, 6, 127, 128, 129, 192]
    assert p.carry_src.tolist() == list(range(5)) + list(range(200, 263)) and p.carry_dst.tolist() == list(range(5)) + list(range(64, 127))
    q = c.plan([2, 0], [1, 1]).latent()
    assert q.home_rows.tolist() == [263, 5] and q.kv_lens.tolist() == [64, 6] and q.ctx_rows is None


def test_rope_table_grows_and_keeps_far_positions_exact():
    from triton_distributed_b200 import ops

    a = ops.rope_table(1e4, 6, 8, 10, "cpu")
    b = ops.rope_table(1e4, 6, 8, 60000, "cpu")
    assert torch.equal(a, b[:10]) and float(b[:, 6:].abs().max()) == 0
    p = 59999
    for i in range(3):
        ang = p * 1e4 ** (-2 * i / 6)
        assert abs(float(b[p, 2 * i]) - math.cos(ang)) < 1e-7 and abs(float(b[p, 2 * i + 1]) - math.sin(ang)) < 1e-7


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
TP = cases.config([(cases.latent(4, 16, 8, 24, 40), cases.moe(4, 2, 16, 32, 2, (3, 1))), (cases.latent(2, 16, 8, 12, 40, kv_from=0), cases.dense(24)),
                   (cases.latent(2, 8, 6, 8, 20), None)], 48, 77)


def _tp_rank(rank, world, d, toks):
    import lisenex_cases as cases_
    import lisenex_oracle as oracle_

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


# ------------------------------------------------------------------ the tests' own sharpness
def _mistakes():
    rotate, route, latent, attn, moe = oracle.rotate, oracle.route, oracle.latent, oracle.latent_attention, oracle.moe

    def halves(x, pos, base):                  # the first half turned with the second
        n = x.shape[-1]
        order = [i // 2 + (i % 2) * (n // 2) for i in range(n)]
        y = rotate(x[..., order], pos, base)
        out = x.clone()
        out[..., order] = y
        return out

    def normed_key_part(h, W, p, mixer, eps):
        c, kr = latent(h, W, p, mixer, eps)
        return c, oracle.rms(kr, eps)

    def raw_latent(h, W, p, mixer, eps):
        c, kr = latent(h, W, p, mixer, eps)
        return (h @ W[p + "dkv"].T)[:, :mixer["kv_rank"]], kr

    def own_rows(h, W, p, mixer, eps, kept=None):       # a sharing layer that misses the last key
        if kept is None:
            return attn(h, W, p, mixer, eps)
        return attn(h, W, p, mixer, eps, (torch.roll(kept[0], 1, 0), torch.roll(kept[1], 1, 0)))

    def corrected_weights(z, correction, top, groups=None):
        ids, w = route(z, correction, top, groups)
        return ids, w + correction[ids]

    def renormalised(z, correction, top, groups=None):
        ids, w = route(z, correction, top, groups)
        return ids, w / w.sum()

    def zero_outside(z, correction, top, groups=None):  # groups left out count as 0
        ids, w = route(z, correction, top, groups)
        if not groups:
            return ids, w
        s = torch.softmax(z, 0)
        size = z.shape[0] // groups["count"]
        c = s + correction
        best = torch.stack([c[g * size:(g + 1) * size].max() for g in range(groups["count"])])
        kept = torch.topk(best, groups["keep"]).indices.tolist()
        c = torch.stack([c[i] if i // size in kept else torch.zeros((), dtype=c.dtype) for i in range(z.shape[0])])
        ids = torch.argsort(c, descending=True, stable=True)[:top]
        return ids.tolist(), s[ids]

    def no_groups(z, correction, top, groups=None):
        return route(z, correction, top, None)

    def no_identity(h, W, p, mlp):
        return moe(h, W, p, mlp) - sum_identity(h, W, p, mlp)

    def sum_identity(h, W, p, mlp):
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            ids, w = route(W[p + "router"] @ h[t], W[p + "correction"], mlp["router"]["top"], mlp["router"].get("groups"))
            for e, we in zip(ids, w):
                if e >= mlp["router"]["experts"]:
                    out[t] += we * h[t]
        return out

    def blind(i, j):                           # the query's own key is missing
        return j < i or i == j == 0

    return [("rotate", halves), ("latent", normed_key_part), ("latent", raw_latent), ("latent_attention", own_rows), ("route", corrected_weights),
            ("route", renormalised), ("route", zero_outside), ("route", no_groups), ("moe", no_identity), ("visible", blind)]


@pytest.mark.parametrize("i", range(10))
def test_a_mistake_in_one_mechanism_shows(i, mixed, monkeypatch):
    """A fault of one mechanism moves logits far beyond the tolerances used here and on the GPU."""
    _, w, toks, want = mixed
    name, wrong = _mistakes()[i]
    monkeypatch.setattr(oracle, name, wrong)
    got = oracle.forward(cases.MIXED, w, toks)
    assert cases.rel(got, want) > 0.25, name
