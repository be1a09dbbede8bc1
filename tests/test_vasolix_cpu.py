"""Vasolix on CPU ranks (fp32): configuration, weights, cache plans, engine steps, generation, tensor parallelism.  The
kernels are covered by test_vasolix_gpu.py; here the host logic runs over the ops' CPU backend."""
import io
import json

import pytest
import torch

import vasolix_cases as cases
import vasolix_oracle as oracle
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
def test_oracle_sink_and_blocks():
    s = torch.tensor([0.3, -1.0, 2.0], dtype=torch.float64)
    p = oracle.sink_softmax(s, torch.tensor(0.7))
    full = torch.softmax(torch.cat([s, torch.tensor([0.7], dtype=torch.float64)]), 0)
    torch.testing.assert_close(p, full[:3])
    assert [j for j in range(12) if oracle.visible(9, j, 4)] == [8, 9]
    assert [j for j in range(12) if oracle.visible(8, j, 4)] == [8]
    assert [j for j in range(12) if oracle.visible(7, j, 4)] == [4, 5, 6, 7]


# ------------------------------------------------------------------ configuration and registry
def test_configuration_is_read_and_checked(mixed, tmp_path):
    from triton_distributed_b200.models import ModelConfig, VasolixConfig

    a = ModelConfig(checkpoint_dir=str(mixed[0])).arch()
    assert isinstance(a, VasolixConfig) and a.vocab_size == 101 and a.hidden_size == 60 and a.num_hidden_layers == 5
    assert a.layers[2].mlp is None and a.layers[1].mlp.shared_ff == 0 and a.layers[4].mixer.block == 0
    assert a.layers[2].mixer.block == 17 and a.layers[3].mixer.tau == 7.0

    def broken(**change):
        c = json.loads(json.dumps(cases.MIXED))
        c["layers"][0].update(change)
        (tmp_path / "config.json").write_text(json.dumps(c))
        return VasolixConfig.from_json(str(tmp_path))

    with pytest.raises(ValueError, match="mixer"):
        broken(type="other")
    with pytest.raises(ValueError, match="kind"):
        broken(mlp={"kind": "other"})
    with pytest.raises(ValueError, match="vdim"):
        broken(mixer={"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 16, "scale": 1.0})
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "unheard of"}))
    with pytest.raises(KeyError, match="architecture"):
        ModelConfig(checkpoint_dir=str(tmp_path)).arch()


def test_registry_and_presets(rt):
    from triton_distributed_b200.models import AutoLLM, ModelConfig, VasolixLLM

    m = AutoLLM.from_pretrained(ModelConfig(model_name="tiny-vasolix", dtype=torch.float32, num_layers_override=5))
    assert isinstance(m, VasolixLLM) and len(m.layers) == 5 and m.layers[4].spec == m.layers[1].spec
    with pytest.raises(ValueError, match="bfloat16 or float32"):
        AutoLLM.from_pretrained(ModelConfig(model_name="tiny-vasolix", dtype=torch.float16))


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

    def all_of(i, lo, hi):
        return (i, prompts[i][lo:hi], list(range(hi - lo)))

    got = {i: [] for i in prompts}

    def step(parts):
        z = eng.step([all_of(*p) for p in parts])
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


def test_step_rejects_what_does_not_fit(mixed):
    eng = cases.engine(mixed[0], torch.float32, max_length=10)
    for bad, msg in (([("a", [1, 101], [])], "token ids"), ([("a", [1], [1])], "wanted"), ([("a", [], [])], "at least one"),
                     ([("a", [1], []), ("a", [2], [])], "distinct"), ([("a", [1] * 11, [])], "max_length"), ([], "empty")):
        with pytest.raises(ValueError, match=msg):
            eng.step(bad)
    eng.step([("a", [1] * 10, [])])
    with pytest.raises(ValueError, match="max_length"):
        eng.step([("a", [1], [0])])


def test_cache_slots():
    from triton_distributed_b200.models import HybridCache, StateSpec, TiedKVSpec

    c = HybridCache([TiedKVSpec(2, 8, 16), TiedKVSpec(1, 8, 0), StateSpec(2, 4, 4)], 2, 40, torch.float32, "cpu")
    assert c.layers[0]["k"].shape == (2, 16, 2, 8) and c.layers[1]["k"].shape == (2, 40, 1, 8)
    c.layers[2]["state"][1] = 3.0
    c.advance([0, 1], [5, 9])
    assert c.kv_offset.tolist() == [5, 9] and c.lens == [5, 9]
    s = c.alloc()                                           # grows, keeps what is there
    assert s == 2 and c.capacity == 4 and float(c.layers[2]["state"][1].min()) == 3.0 and c.lens[1] == 9
    c.free(1)
    with pytest.raises(ValueError):
        c.free(1)
    assert c.alloc() == 1 and c.lens[1] == 0 and int(c.kv_offset[1]) == 0
    plan = c.plan([0, 1], [30, 16])                         # positions 5..34 and 0..15, blocks of 16
    b = plan.blocks(TiedKVSpec(2, 8, 16))
    assert b.cu.tolist() == [0, 11, 27, 30, 46] and b.q_pos0.tolist() == [5, 0, 0, 0] and b.kv_lens.tolist() == [16, 16, 3, 16]
    assert b.carry_src.tolist() == [0, 1, 2, 3, 4] and b.home_rows[:27].max() == -1 and b.home_rows[27:30].tolist() == [0, 1, 2]
    with pytest.raises(ValueError, match="max_length"):
        c.plan([0], [36])


# ------------------------------------------------------------------ generation
def test_greedy_generation_through_serve(rt, tmp_path):
    cfg = cases.PLAIN
    w = cases.weights(cfg, seed=3)
    eng = cases.engine(cases.write(tmp_path, cfg, w), torch.float32, max_length=64)
    prompts = [cases.prompt(cfg, 22, s) for s in range(3)]
    want = [cases.greedy(cfg, w, p, 6) for p in prompts]
    assert min(g for _, g in want) > 1e-3
    out = eng.serve(torch.tensor(prompts), 6)
    assert out.tolist() == [t for t, _ in want]
    # unequal prompts, right-padded: the same continuations as alone
    lens = [22, 5, 13]
    short = [cases.greedy(cfg, w, p[:n], 6)[0] for p, n in zip(prompts, lens)]
    assert eng.serve(torch.tensor(prompts), 6, seq_lens=lens).tolist() == short
    with pytest.raises(ValueError, match="seq_lens"):
        eng.serve(torch.tensor(prompts), 2, seq_lens=[22, 0, 1])
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
TP = cases.config([(cases.attention(4, 2, 16, 12), cases.moe(4, 2, 16, 32)), (cases.gla(2, 8, 24, 3.0), cases.moe(4, 1, 16, 0))], 48, 77)


def _tp_rank(rank, world, d, toks):
    import vasolix_cases as cases_
    import vasolix_oracle as oracle_

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
    def no_sink(scores, sink):
        return torch.softmax(scores, 0)

    def edge(i, j, size):                      # blocks one position late
        return j <= i and (not size or (i + 1) // size == (j + 1) // size or i == j)

    def open_edge(i, j, size):                 # one key of the block before
        return j <= i and (not size or i // size == j // size or j == i // size * size - 1)

    def weight_on_output(h, W, p, mlp):
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            for e, we in zip(*oracle.route(h[t], W, p, mlp["router"]["top"])):
                out[t] += we * oracle.expert(h[t], W, f"{p}e{e}.")
            if mlp.get("shared"):
                out[t] += oracle.sigmoid(W[p + "shared.sg"] @ h[t]) * oracle.expert(h[t], W, p + "shared.")
        return out

    def late_decay(q, k, v, alpha, state=None):
        return real(q, k, v, torch.cat([torch.ones_like(alpha[:1]), alpha[:-1]]), state)

    real = oracle.gla_recurrence
    return [("sink_softmax", no_sink), ("visible", edge), ("visible", open_edge), ("moe", weight_on_output), ("gla_recurrence", late_decay)]


@pytest.mark.parametrize("i", range(5))
def test_a_mistake_in_one_mechanism_shows(i, mixed, monkeypatch):
    """A fault of one mechanism moves logits far beyond the tolerances used here and on the GPU."""
    _, w, toks, want = mixed
    name, wrong = _mistakes()[i]
    monkeypatch.setattr(oracle, name, wrong)
    got = oracle.forward(cases.MIXED, w, toks)
    assert cases.rel(got, want) > 0.3, name
