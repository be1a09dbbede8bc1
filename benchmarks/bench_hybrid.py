"""Layered decoder (Vasolix) against the closest existing model (Qwen3-MoE) at equal layer sizes, random weights, one GPU:
prefill and decode throughput of a few layers, and the kernels one by one beside the like kernel of the other model.

    python benchmarks/bench_hybrid.py [--size 30b-a3b,1b] [--parts prefill,decode,kernels]

Model numbers: CUDA events around whole steps (decode: CUDA-graph replays), weights and activations larger than L2.  Kernel
numbers: median of single calls with an L2 flush in between; ``roof_us`` is the slower of bytes / measured copy bandwidth and
FLOPs / measured GEMM rate, ``frac`` = roof / time.
"""
import argparse
import json
import os
import statistics
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

import triton_distributed_b200 as tdb  # noqa: E402
from triton_distributed_b200 import ops  # noqa: E402
from triton_distributed_b200.models import ArchConfig, KV_Cache, ModelConfig, Qwen3MoE, VasolixLLM  # noqa: E402
from triton_distributed_b200.models.vasolix import AttentionSpec, GLASpec, MoESpec, hybrid_stack  # noqa: E402
from triton_distributed_b200.utils import device_time_ms, load_peaks  # noqa: E402

LAYERS, VOCAB, CTX = 4, 32768, 4096
# width, query heads, KV heads, head dim, attention block, GLA heads, GLA dims, experts, top, ff, shared ff
SIZES = {"30b-a3b": (2048, 32, 4, 128, 4096, 16, (128, 128), 128, 8, 768, 768),
         "1b": (1536, 24, 4, 64, 1024, 12, (64, 128), 32, 4, 512, 512)}


def archs(size):
    W, hq, hkv, D, block, gh, (dk, dv), E, top, ff, sff = SIZES[size]
    v = hybrid_stack(f"vasolix-{size}", VOCAB, W, ("GA" * LAYERS)[:LAYERS], AttentionSpec(hq, hkv, D, D ** -0.5, block),
                     GLASpec(gh, dk, dv, 16.0), MoESpec(E, top, ff, sff))
    q = ArchConfig(f"qwen3-moe-{size}", W, ff, LAYERS, hq, hkv, D, VOCAB, num_experts=E, num_experts_per_tok=top, moe_intermediate_size=ff)
    return {"vasolix": v, "qwen3_moe": q}


class Fixed(ModelConfig):
    """A run-time configuration around a given architecture."""

    def arch(self):
        return self._arch


def make(cls, arch, max_length):
    cfg = Fixed(model_name=arch.name, max_length=max_length)
    cfg._arch = arch
    m = cls(cfg)
    if cls is Qwen3MoE:
        m.init_ctx_for("triton_dist_gemm_ar", 8192)
    m.set_fwd("triton_dist_gemm_ar")
    return m


def new_cache(model, B, max_length):
    if hasattr(model, "new_cache"):
        return model.new_cache(B, max_length)
    a = model.arch
    return KV_Cache(a.num_hidden_layers, B, max_length, a.num_key_value_heads, a.head_dim, device=model.device)


def timed(fn, iters, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    s.record()
    for _ in range(iters):
        fn()
    e.record()
    torch.cuda.synchronize()
    return s.elapsed_time(e) / iters


def bench_prefill(model, B, S):
    cache = new_cache(model, B, S)
    ids = torch.randint(0, VOCAB, (B, S), device=model.device)
    pos = torch.arange(S, device=model.device).expand(B, S).contiguous()
    def run():
        cache.clear()
        if not hasattr(model, "new_cache"):
            cache.kv_offset.zero_()
        model.inference(ids, pos, cache)
    return timed(run, 8)


def bench_decode(model, B, ctx):
    cache = new_cache(model, B, ctx + 64)
    cache.rand_fill(ctx)
    ids = torch.randint(0, VOCAB, (B, 1), device=model.device)

    def step():
        model.inference(ids, cache.kv_offset[:B].to(torch.int64).unsqueeze(1), cache)

    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for _ in range(3):
            step()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        step()
    return timed(g.replay, 50)


def bench_models(size, parts):
    out = []
    for name, arch in archs(size).items():
        model = make(VasolixLLM if name == "vasolix" else Qwen3MoE, arch, 16384)
        if "prefill" in parts:
            for B, S in ((1, 2048), (1, 8192), (4, 2048)):
                ms = bench_prefill(model, B, S)
                out.append({"model": name, "size": size, "layers": LAYERS, "phase": "prefill", "batch": B, "tokens": S, "ms": round(ms, 3),
                            "tokens_per_s": round(B * S / ms * 1e3)})
        if "decode" in parts:
            for B in (1, 8, 64):
                ms = bench_decode(model, B, CTX)
                out.append({"model": name, "size": size, "layers": LAYERS, "phase": "decode", "batch": B, "ctx": CTX, "ms": round(ms, 4),
                            "tokens_per_s": round(B / ms * 1e3)})
        model.finalize()
        del model
        torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------ kernels
def bench_kernels(size):
    W, hq, hkv, D, block, gh, (dk, dv), E, top, ff, sff = SIZES[size]
    peaks = load_peaks()
    dev, bf = "cuda", torch.bfloat16
    out = []

    def rec(kernel, like_of, T, fn, nbytes, flops=0.0):
        us = statistics.median(device_time_ms(fn, 15, 3)) * 1e3
        roof = max(nbytes / (peaks["hbm_gbs"] * 1e3), flops / (peaks["bf16_tflops"] * 1e6))
        out.append({"kernel": kernel, "beside": like_of, "size": size, "tokens": T, "us": round(us, 2), "roof_us": round(roof, 2),
                    "frac": round(roof / us, 3)})

    def rnd(*s, dtype=bf):
        return torch.randn(*s, device=dev).to(dtype)

    for T in (8192, 64, 8, 1):
        x, xb, y = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W)
        wf, wb = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=bf)
        rec("postnorm_add", "norm", T, lambda: ops.postnorm_add(x, xb, y, wf, W, 1e-5), T * W * (4 + 4 + 2 + 2))
        rec("rmsnorm + residual (qwen3_moe)", "norm", T, lambda: ops.rmsnorm(y, wb, 1e-5, residual=xb), T * W * 2 * 4)
        # q / k norm and cache write
        nq, nk = hq * D, hkv * D
        qkg, rows = rnd(T, 2 * nq + nk), torch.arange(T, device=dev)
        kc, sc, qw = torch.empty(T, nk, device=dev, dtype=bf), torch.empty(T, device=dev), torch.ones(nq, device=dev)
        rec("qk_norm_tied", "qk norm", T, lambda: ops.qk_norm_tied(qkg, qw, nk, nq, nk, 1e-5, (kc, sc, rows)), T * 2 * 2 * (nq + nk))
        qkv, nw = rnd(T, nq + 2 * nk), torch.ones(D, device=dev, dtype=bf)
        vc = torch.empty_like(kc)
        rec("qk_norm_rope_kv (qwen3_moe)", "qk norm", T,
            lambda: ops.qk_norm_rope_kv(qkv, nw, nw, rows, rows, kc.view(T, hkv, D), vc.view(T, hkv, D), hq, hkv, D), T * 2 * 2 * (nq + 2 * nk))
        # router
        rw, rw1 = rnd(E + 1, W), rnd(E, W)
        rec("sigmoid_router", "router", T, lambda: ops.sigmoid_router(xb, rw, top, True), (T + E) * W * 2, 2.0 * T * E * W)
        rec("gemm + topk_router (qwen3_moe)", "router", T, lambda: ops.topk_router(ops.gemm(xb, rw1).float(), top), (T + E) * W * 2, 2.0 * T * E * W)
        # experts (both with the routing of random tokens)
        ids, wts, gate = ops.sigmoid_router(xb, rw * W ** -0.5, top, True)
        up, down, w13 = rnd(E, ff, W), rnd(E, W, ff), rnd(E, 2 * ff, W)
        used = ids.unique().numel()
        if T <= ops.EXPERT_GEMV_MAX_T:
            su, sd = rnd(sff, W), rnd(W, sff)
            rec("experts gemv (incl. shared)", "experts", T, lambda: ops.relu2_experts_gemv(xb, up, down, ids, wts, su, sd, gate),
                (used * ff + sff) * W * 2 * 2)
        else:
            def grouped():
                srt = ops.sort_topk_ids_align_block_size(ids, E)
                h = ops.relu2(ops.group_gemm_gather(xb, up, srt, a_row_div=top, scatter_out=True), wts.reshape(-1))
                return ops.group_gemm_gather(h, down, srt, a_row_div=1, scatter_out=True)
            rec("experts grouped GEMM (without shared)", "experts", T, grouped, used * ff * W * 4 + T * W * 2 * (1 + top), 4.0 * T * top * ff * W)
            h = rnd(T * top, ff)
            rec("relu2", "activation", T, lambda: ops.relu2(h, wts.reshape(-1)), T * top * ff * 4)
        rs = ops.create_moe_rs_context(max_token_num=T, hidden_dim=W, num_experts=E, topk=top)

        def qwen_moe():
            srt = ops.sort_topk_ids_align_block_size(ids, E)
            hs = ops.silu_mul(ops.group_gemm_gather(xb, w13, srt, a_row_div=top))
            return ops.run_moe_reduce_ar(hs, down, ids, wts, rs, sort=srt)
        rec("experts SwiGLU (qwen3_moe)", "experts", T, qwen_moe, used * ff * W * 6 + T * W * 4, 6.0 * T * top * ff * W)
        del up, down, w13
        # gated linear attention
        N = 1 if T == 8192 else T
        state = torch.zeros(N, gh, dk, dv, device=dev)
        slots, pos0 = torch.arange(N, dtype=torch.int32, device=dev), torch.ones(N, dtype=torch.int64, device=dev)
        qkvg, low = rnd(T, 2 * gh * (dk + dv)), rnd(T, 16, dtype=torch.float32)
        a2, a2b, nwv = rnd(16, gh * dk, dtype=torch.float32), torch.full((gh * dk,), 2.0, device=dev), torch.ones(dv, device=dev)
        io = T * gh * (2 * dk + 3 * dv) * 2
        if T == 8192:
            tabs, cu = ops.gla_chunk_tables([0, T], dev), torch.tensor([0, T], dtype=torch.int32, device=dev)
            fl = T * gh * (4.0 * dk * dv + 64 * (dk + dv))
            rec("gla chunk", "recurrence", T, lambda: ops.gated_linear_attention(qkvg, low, a2, a2b, 16.0, nwv, state, slots, pos0, cu, dv, 0.1, 1e-5, tabs), io, fl)
            q, k, v = rnd(1, T, gh, 128), rnd(1, T, gh, 128) * 0.05, rnd(1, T, gh, 128)
            gg, bt = -torch.rand(1, T, gh, device=dev), torch.rand(1, T, gh, device=dev).to(bf)
            rec("gdn chunk (K = V = 128)", "recurrence", T, lambda: ops.chunk_gated_delta_rule_fwd(q, k, v, gg, bt, 0.1, None, False, cu),
                T * gh * 512 * 2, T * gh * (6.0 * 128 * 128 + 64 * 512))
        else:
            rec("gla decode", "recurrence", T, lambda: ops.gated_linear_attention(qkvg, low, a2, a2b, 16.0, nwv, state, slots, pos0, None, dv, 0.1, 1e-5),
                io + T * gh * dk * dv * 8)
        # attention
        sink = torch.zeros(hq, device=dev)
        if T == 8192:
            from triton_distributed_b200.models import HybridCache, TiedKVSpec
            spec = TiedKVSpec(hkv, D, block)
            bp = HybridCache([spec], 1, T, bf, dev).plan([0], [T]).blocks(spec)
            pages, scale = rnd(bp.pages, bp.page_rows, hkv, D), torch.ones(bp.pages, bp.page_rows, device=dev)
            q = rnd(T, hq, D)
            pairs = (T // block) * block * (block + 1) / 2
            rec("tied block attention", "prefill attention", T,
                lambda: ops.tied_attn_varlen(q, pages, scale, bp.block_table, bp.cu, bp.q_pos0, bp.kv_lens, bp.max_q, bp.max_kv, sink, qkg[:, nq + nk:]),
                T * (3 * nq + nk) * 2, 4.0 * pairs * hq * D)
            # the other model's kernel on the same (sequence, block) pairs
            vp = torch.empty_like(pages)
            rec("flash_attn_varlen (qwen3_moe), same blocks", "prefill attention", T,
                lambda: ops.flash_attn_varlen(q, pages, vp, bp.block_table, bp.cu, bp.kv_lens, bp.max_q, max_kv_len=bp.max_kv),
                T * (2 * nq + 2 * nk) * 2, 4.0 * pairs * hq * D)
        else:
            n = min(block, CTX)
            kk, vv = rnd(T, n, hkv, D), rnd(T, n, hkv, D)
            scale = torch.ones(T, n, device=dev)
            bt = ops.dense_block_table(T, dev)
            lens = torch.full((T,), n, dtype=torch.int32, device=dev)
            q = rnd(T, hq, D)
            sp = ops.pick_kv_splits(T, hkv, (hq // hkv + 15) // 16, n)
            sp2 = ops.pick_tied_splits(T, hkv, (hq // hkv + 15) // 16, n)
            rec("tied decode attention", "decode attention", T, lambda: ops.tied_attn_decode(q, kk, scale, bt, lens, n, sp2, sink, qkg[:, nq + nk:]),
                T * n * (nk * 2 + 4))
            rec("gqa_fwd_batch_decode (qwen3_moe)", "decode attention", T, lambda: ops.gqa_fwd_batch_decode(q, kk, vv, None, None, lens, bt, kv_split=sp),
                T * n * nk * 2 * 2)
        torch.cuda.empty_cache()
    return out


def run(sizes, parts):
    """All records, as dictionaries."""
    out = []
    for s in sizes:
        if "prefill" in parts or "decode" in parts:
            out += bench_models(s, parts)
        if "kernels" in parts:
            out += bench_kernels(s)
    return out


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default=",".join(SIZES))
    ap.add_argument("--parts", default="prefill,decode,kernels")
    args = ap.parse_args()
    tdb.initialize_distributed(seed=0)
    for r in run(args.size.split(","), args.parts.split(",")):
        print(json.dumps(r), flush=True)
    tdb.finalize_distributed()


if __name__ == "__main__":
    main()
