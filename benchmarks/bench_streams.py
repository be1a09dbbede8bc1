"""Tazitar (several residual streams, attention beside a gated delta rule) against the closest existing model (Qwen3 dense) at equal
layer sizes, random weights, one GPU: prefill and decode throughput of a few layers, and the kernels one by one beside the like kernel
of the other models (recurrence: gated linear attention of Vasolix and the bare gated delta rule).

    python benchmarks/bench_streams.py [--size 8b,1b] [--parts prefill,decode,kernels]

Timing and roofline columns as in ``bench_hybrid.py``.
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
from triton_distributed_b200.models import ArchConfig, DenseLLM, TazitarLLM  # noqa: E402
from triton_distributed_b200.models.tazitar import KINDS, DeltaRuleSpec, RotaryAttnSpec, TwinSpec, stream_stack  # noqa: E402
from triton_distributed_b200.utils import device_time_ms, load_peaks  # noqa: E402
from benchmarks import bench_hybrid as hybrid  # noqa: E402
from benchmarks.bench_hybrid import CTX, LAYERS, VOCAB  # noqa: E402

# width, query heads, KV heads, head dim, feed-forward; delta rule: heads, key heads, key and value dims of a head
SIZES = {"8b": (4096, 32, 8, 128, 12288, 32, 16, (128, 128)), "1b": (1536, 24, 4, 64, 4096, 12, 6, (64, 128))}
STREAMS, TAPS, CAP = 4, 4, 50.0


def archs(size):
    W, hq, hkv, D, ff, dh, dg, (dk, dv) = SIZES[size]

    def attn(kind, rot, **kw):
        return RotaryAttnSpec(hq, hkv, D, D, D ** -0.5, 1e6, rot, **kw, **KINDS[kind])

    t = stream_stack(f"tazitar-{size}", VOCAB, W, ("APPB" * LAYERS)[:LAYERS], attn("attention", D, softcap=CAP),
                     TwinSpec(attn("left", D // 4), DeltaRuleSpec(dh, dg, dk, dv, TAPS)),
                     attn("attention_2", D, scaling=ops.YarnScaling(4.0, 8192, 32.0, 1.0)), ff, STREAMS)
    return {"tazitar": (TazitarLLM, t), "qwen3": (DenseLLM, ArchConfig(f"qwen3-{size}", W, ff, LAYERS, hq, hkv, D, VOCAB))}


def bench_models(size, parts):
    out = []
    for name, (cls, a) in archs(size).items():
        model = hybrid.make(cls, a, 16384)
        if cls is DenseLLM:
            model.init_ctx_for("triton_dist_gemm_ar", 8192)
        if "prefill" in parts:
            for B, S in ((1, 2048), (1, 8192), (4, 2048)):
                ms = hybrid.bench_prefill(model, B, S)
                out.append({"model": name, "size": size, "layers": LAYERS, "phase": "prefill", "batch": B, "tokens": S, "ms": round(ms, 3),
                            "tokens_per_s": round(B * S / ms * 1e3)})
        if "decode" in parts:
            for B in (1, 8, 64):
                ms = hybrid.bench_decode(model, B, CTX)
                out.append({"model": name, "size": size, "layers": LAYERS, "phase": "decode", "batch": B, "ctx": CTX, "ms": round(ms, 4),
                            "tokens_per_s": round(B / ms * 1e3)})
        model.finalize()
        del model
        torch.cuda.empty_cache()
    ops.check_attention_errors()
    return out


# ------------------------------------------------------------------ kernels
def bench_kernels(size):
    W, hq, hkv, D, ff, dh, dg, (dk, dv) = SIZES[size]
    S = STREAMS
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
        # between two sublayers
        x, y, y2, xb = rnd(T, S, W, dtype=torch.float32), rnd(T, W), rnd(T, W), rnd(T, W)
        wf, wb = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=bf)
        hc = ops.HyperWeights(torch.full((S,), 1.0 / S, device=dev), torch.ones(S, device=dev), torch.eye(S, device=dev))
        rec("hyper_step", "norm", T, lambda: ops.hyper_step(x, (hc, ops.SublayerOutput(y)), (hc.inp, wf), W, 1e-5, bf), T * W * (8 * S + 2 + 2))
        rec("hyper_step, two branches", "norm", T, lambda: ops.hyper_step(x, (hc, ops.SublayerOutput(y, y2, wf, wf)), (hc.inp, wf), W, 1e-5, bf),
            T * W * (8 * S + 4 + 2))
        rec("rmsnorm + residual (qwen3)", "norm", T, lambda: ops.rmsnorm(y, wb, 1e-5, residual=xb), T * W * 2 * 4)
        x1 = rnd(T, W, dtype=torch.float32)
        rec("postnorm_add (vasolix)", "norm", T, lambda: ops.postnorm_add(x1, xb, y, wf, W, 1e-5), T * W * (4 + 4 + 2 + 2))
        # feed-forward's activation
        h = rnd(T, 2 * ff)
        rec("gated_act (gelu)", "activation", T, lambda: ops.gated_act(h, "gelu"), T * ff * 6)
        rec("silu_mul (qwen3)", "activation", T, lambda: ops.silu_mul(h), T * ff * 6)
        if T <= ops.GEMV_FAST_M and ops.gemv_supported(T, ff):
            wd = rnd(W, ff)
            rec("down projection with gelu", "gemv", T, lambda: ops.gemv_fused(h, wd, silu_mul=True, act="gelu"), (W * ff + T * (2 * ff + W)) * 2)
            rec("down projection with silu (qwen3)", "gemv", T, lambda: ops.gemv_fused(h, wd, silu_mul=True), (W * ff + T * (2 * ff + W)) * 2)
        # q / k preparation and cache write
        nq, nk = hq * D, hkv * D
        qkv, nw, nwf, rows = rnd(T, nq + 2 * nk), torch.ones(D, device=dev, dtype=bf), torch.ones(D, device=dev), torch.arange(T, device=dev)
        kc, vc = rnd(T, hkv, D), rnd(T, hkv, D)
        io = T * 2 * 2 * (nq + 2 * nk)
        tab = ops.rope_table(1e6, D, D, max(CTX, T), dev)
        rec("head_prep, weighted norms, halves", "q / k preparation", T,
            lambda: ops.head_prep(qkv, hq, hkv, D, D, nwf, nwf, False, 1e-5, tab, D, False, rows, kc, vc, rows), io)
        rec("head_prep, unit norms, neighbours", "q / k preparation", T,
            lambda: ops.head_prep(qkv, hq, hkv, D, D, None, None, True, 1e-5, tab, D, True, rows, kc, vc, rows), io)
        rec("qk_norm_rope_kv (qwen3)", "q / k preparation", T, lambda: ops.qk_norm_rope_kv(qkv, nw, nw, rows, rows, kc, vc, hq, hkv, D), io)
        # recurrence
        N = 1 if T == 8192 else T
        C, Hv = 2 * dg * dk + dh * dv, dh * dv
        z, ab = rnd(T, C + Hv), rnd(T, 2 * dh, dtype=torch.float32)
        conv_w, alog, dt = rnd(C, TAPS, dtype=torch.float32), torch.zeros(dh, device=dev), torch.full((dh,), -2.0, device=dev)
        nwv, state = torch.ones(dv, device=dev), torch.zeros(N, dh, dk, dv, device=dev)
        ring = torch.zeros(N, TAPS, C, device=dev, dtype=bf)
        slots, pos0 = torch.arange(N, dtype=torch.int32, device=dev), torch.full((N,), 64, dtype=torch.int64, device=dev)
        args = (z, ab, conv_w, alog, dt, nwv, state, ring, slots, pos0)
        qkvg, low = rnd(T, 2 * dh * (dk + dv)), rnd(T, 16, dtype=torch.float32)
        a2, a2b = rnd(16, dh * dk, dtype=torch.float32), torch.full((dh * dk,), 2.0, device=dev)
        dio, gio = T * (C + 2 * Hv) * 2, T * dh * (2 * dk + 3 * dv) * 2
        if T == 8192:
            tabs, cu = ops.gla_chunk_tables([0, T], dev), torch.tensor([0, T], dtype=torch.int32, device=dev)
            rec("delta rule, chunks (with convolutions)", "recurrence", T, lambda: ops.gated_delta_rule(*args, cu, dg, dv, dk ** -0.5, 1e-5, tabs), dio,
                T * dh * (6.0 * dk * dv + 64 * (dk + dv)))
            rec("gla chunk (vasolix)", "recurrence", T, lambda: ops.gated_linear_attention(qkvg, low, a2, a2b, 16.0, nwv, state, slots, pos0, cu, dv, 0.1,
                                                                                           1e-5, tabs), gio, T * dh * (4.0 * dk * dv + 64 * (dk + dv)))
            q, k, v = rnd(1, T, dh, 128), rnd(1, T, dh, 128) * 0.05, rnd(1, T, dh, 128)
            gg, bt = -torch.rand(1, T, dh, device=dev), torch.rand(1, T, dh, device=dev).to(bf)
            rec("gdn chunk (K = V = 128, bf16 state, recurrence only)", "recurrence", T,
                lambda: ops.chunk_gated_delta_rule_fwd(q, k, v, gg, bt, 0.1, None, False, cu), T * dh * 512 * 2, T * dh * (6.0 * 128 * 128 + 64 * 512))
            del q, k, v
        else:
            rec("delta rule, decode (with convolutions)", "recurrence", T, lambda: ops.gated_delta_rule(*args, None, dg, dv, dk ** -0.5, 1e-5),
                dio + T * (dh * dk * dv * 8 + C * 2 * TAPS))
            rec("gla decode (vasolix)", "recurrence", T, lambda: ops.gated_linear_attention(qkvg, low, a2, a2b, 16.0, nwv, state, slots, pos0, None, dv, 0.1, 1e-5),
                gio + T * dh * dk * dv * 8)
        # attention
        sink = torch.zeros(hq, device=dev)
        if T == 8192:
            kk, vv, q = rnd(1, T, hkv, D), rnd(1, T, hkv, D), rnd(T, hq, D)
            i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=dev)   # noqa: E731
            cu, kl, bt = i32(0, T), i32(T), ops.dense_block_table(1, dev)
            for name, kw in (("attention with soft cap", {"softcap": CAP}), ("attention with soft cap, large scores", {"softcap": 2.0}),
                             ("attention with sink", {"sink": sink}), ("attention (qwen3)", {})):
                rec(name, "prefill attention", T, lambda: ops.flash_attn_varlen(q, kk, vv, bt, cu, kl, T, max_kv_len=T, **kw),
                    T * (2 * nq + 2 * nk) * 2, 2.0 * T * (T + 1) * hq * D)
        else:
            kk, vv, q = rnd(T, CTX, hkv, D), rnd(T, CTX, hkv, D), rnd(T, hq, D)
            bt, lens = ops.dense_block_table(T, dev), torch.full((T,), CTX, dtype=torch.int32, device=dev)
            for name, kw in (("attention with soft cap", {"soft_cap": CAP}), ("attention with sink", {"sink": sink}), ("attention (qwen3)", {})):
                rec(name, "decode attention", T, lambda: ops.gqa_fwd_batch_decode(q, kk, vv, None, None, lens, bt, **kw), T * CTX * nk * 2 * 2)
        torch.cuda.empty_cache()
    ops.check_attention_errors()
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
    for rec in run(args.size.split(","), args.parts.split(",")):
        print(json.dumps(rec), flush=True)
    tdb.finalize_distributed()


if __name__ == "__main__":
    main()
