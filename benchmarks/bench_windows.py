"""Bagasun (sandwiched sublayers, sliding windows with sigmoid and differential attention, state space layers) against the closest existing
model (Qwen3 dense) at equal layer sizes, random weights, one GPU: prefill and decode throughput of a few layers, and the kernels one by
one beside the like kernel of the other models (recurrence: gated linear attention of Vasolix, gated delta rule of Tazitar).

    python benchmarks/bench_windows.py [--size 8b,1b] [--parts prefill,decode,kernels]

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
from triton_distributed_b200.models import ArchConfig, BagasunLLM, DenseLLM  # noqa: E402
from triton_distributed_b200.models.bagasun import DifferentialAttnSpec, SigmoidAttnSpec, StateSpaceSpec, sandwich_stack  # noqa: E402
from triton_distributed_b200.utils import device_time_ms, load_peaks  # noqa: E402
from benchmarks import bench_hybrid as hybrid  # noqa: E402
from benchmarks.bench_hybrid import CTX, LAYERS, VOCAB  # noqa: E402

# width, query heads, KV heads, head dim, feed-forward, window; differential: heads, KV heads, dim of a map, vdim; state space: heads, groups, state, vdim
SIZES = {"8b": (4096, 32, 8, 128, 12288, 4096, (32, 8, 64, 128), (128, 8, 128, 64)), "1b": (1536, 24, 4, 64, 4096, 1024, (12, 4, 64, 128), (48, 1, 128, 64))}
TAPS = 4


def archs(size):
    W, hq, hkv, D, ff, win, (dh, dg, dd, ddv), (sh, sg, sn, sv) = SIZES[size]
    b = sandwich_stack(f"bagasun-{size}", VOCAB, W, ("MDMA" * LAYERS)[:LAYERS], SigmoidAttnSpec(hq, hkv, D, D, D ** -0.5, win),
                       DifferentialAttnSpec(dh, dg, dd, ddv, dd ** -0.5, 0.8, 1e6, dd, ops.BandScaling(4.0, 8192, 1.0, 4.0), win),
                       StateSpaceSpec(sh, sg, sn, sv, TAPS, sg), ff)
    return {"bagasun": (BagasunLLM, b), "qwen3": (DenseLLM, ArchConfig(f"qwen3-{size}", W, ff, LAYERS, hq, hkv, D, VOCAB))}


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
def pairs(T, window):
    """Visible (query, key) pairs of a prompt."""
    full = min(T, window)
    return full * (full + 1) / 2 + (T - full) * window


def bench_kernels(size):
    W, hq, hkv, D, ff, win, (dh, dg, dd, ddv), (sh, sg, sn, sv) = SIZES[size]
    peaks = load_peaks()
    dev, bf, f32 = "cuda", torch.bfloat16, torch.float32
    out = []

    def rec(kernel, like_of, T, fn, nbytes, flops=0.0):
        us = statistics.median(device_time_ms(fn, 15, 3)) * 1e3
        roof = max(nbytes / (peaks["hbm_gbs"] * 1e3), flops / (peaks["bf16_tflops"] * 1e6))
        out.append({"kernel": kernel, "beside": like_of, "size": size, "tokens": T, "us": round(us, 2), "roof_us": round(roof, 2),
                    "frac": round(roof / us, 3)})

    def rnd(*s, dtype=bf):
        return torch.randn(*s, device=dev).to(dtype)

    def i32(*v):
        return torch.tensor(v, dtype=torch.int32, device=dev)

    nq, nk = hq * D, hkv * D
    for T in (8192, 64, 8, 1):
        # between two sublayers
        x, y, xb, one, wb = rnd(T, W, dtype=f32), rnd(T, W), rnd(T, W), torch.ones(1, device=dev), torch.ones(W, device=dev, dtype=bf)
        rec("sandwich_step", "norm", T, lambda: ops.sandwich_step(x, (y, one), one, W, 1e-5, bf), T * W * (8 + 2 + 2))
        rec("rmsnorm + residual (qwen3)", "norm", T, lambda: ops.rmsnorm(y, wb, 1e-5, residual=xb), T * W * 2 * 4)
        # queries, keys, values
        pos, rows = torch.arange(T, device=dev), torch.arange(T, device=dev)
        tab = ops.rope_table(1e6, D, D, max(CTX, T), dev)
        qkv, nw = rnd(T, nq + 2 * nk), torch.ones(D, device=dev, dtype=bf)
        kc, vc = rnd(T, hkv, D), rnd(T, hkv, D)
        io = T * 2 * 2 * (nq + 2 * nk)
        bias, qw, kw = rnd(nq + 2 * nk, dtype=f32), torch.ones(nq, device=dev), torch.ones(nk, device=dev)
        rec("qkv_prep, biases and whole norms", "q / k preparation", T,
            lambda: ops.qkv_prep(qkv, hq, hkv, hkv, D, D, bias, (qw, kw, nq, nk), 1e-5, None, 0, pos, (kc, vc, rows)), io)
        dz = rnd(T, 2 * (dh + dg) * dd + dg * ddv + 8)
        dk, dv_ = rnd(T, dg, 2 * dd), rnd(T, dg, ddv)
        dtab = ops.rope_table(1e6, dd, dd, max(CTX, T), dev)
        rec("qkv_prep, rotation", "q / k preparation", T,
            lambda: ops.qkv_prep(dz, 2 * dh, 2 * dg, dg, dd, ddv, None, None, 1e-5, dtab, dd, pos, (dk, dv_, rows)), T * 4 * (2 * (dh + dg) * dd + dg * ddv))
        rec("qk_norm_rope_kv (qwen3)", "q / k preparation", T, lambda: ops.qk_norm_rope_kv(qkv, nw, nw, rows, rows, kc, vc, hq, hkv, D), io)
        # recurrence
        N = 1 if T == 8192 else T
        slots, pos0 = torch.arange(N, dtype=torch.int32, device=dev), torch.full((N,), 64, dtype=torch.int64, device=dev)
        inner, C = sh * sv, sh * sv + 2 * sg * sn
        z = rnd(T, inner + C + sh)
        w = ops.SsdWeights(rnd(C, TAPS, dtype=f32), rnd(C, dtype=f32), torch.zeros(sh, device=dev), torch.full((sh,), -2.0, device=dev), torch.ones(sh, device=dev))
        state, ring = torch.zeros(N, sh, sn, sv, device=dev), torch.zeros(N, TAPS, C, device=dev, dtype=bf)
        args = (z[:, inner:], C, w, state, ring, slots, pos0)
        sio, slike = T * (C + sh + inner) * 2, T * sh * (4.0 * sn * sv + 64 * sv) + T * sg * 64.0 * sn
        gh, gk, gv = (16, 128, 128) if size == "8b" else (12, 64, 128)
        qkvg, low = rnd(T, 2 * gh * (gk + gv)), rnd(T, 16, dtype=f32)
        a2, a2b, nwv, gstate = rnd(16, gh * gk, dtype=f32), torch.full((gh * gk,), 2.0, device=dev), torch.ones(gv, device=dev), torch.zeros(N, gh, gk, gv, device=dev)
        gargs, gio = (qkvg, low, a2, a2b, 16.0, nwv, gstate, slots, pos0), T * gh * (2 * gk + 3 * gv) * 2
        if T == 8192:
            tabs, cu = ops.gla_chunk_tables([0, T], dev), i32(0, T)
            rec("state space, chunks (with convolutions)", "recurrence", T, lambda: ops.state_space(*args, cu, sg, tabs), sio, slike)
            rec("gla chunk (vasolix)", "recurrence", T, lambda: ops.gated_linear_attention(*gargs, cu, gv, 0.1, 1e-5, tabs), gio, T * gh * (4.0 * gk * gv + 64 * (gk + gv)))
        else:
            rec("state space, decode (with convolutions)", "recurrence", T, lambda: ops.state_space(*args, None, sg), sio + T * (sh * sn * sv * 8 + C * 2 * TAPS))
            rec("gla decode (vasolix)", "recurrence", T, lambda: ops.gated_linear_attention(*gargs, None, gv, 0.1, 1e-5), gio + T * gh * gk * gv * 8)
        yy, gw = rnd(T, inner), torch.ones(inner, device=dev)
        rec("gate and norm over groups", "activation", T, lambda: ops.gated_group_norm(yy, z, gw, sh, sv, sg, 1e-5), T * inner * 6)
        h = rnd(T, 2 * ff)
        rec("silu_mul (qwen3)", "activation", T, lambda: ops.silu_mul(h), T * ff * 6)
        # attention
        sig = ops.SigmoidWeights(ops.distance_table(torch.full((hq,), 0.3), torch.full((hq,), 0.5), torch.full((hq,), -3.0), max(T, CTX)).to(dev))
        diff = ops.DifferentialWeights(0.6, 0.5, 1e-5, ddv)
        if T == 8192:
            q, kk, vv = rnd(T, hq, D), rnd(T, hkv, D), rnd(T, hkv, D)
            cu, zero, kl, bt = i32(0, T), i32(0), i32(T), ops.dense_block_table(1, dev)
            rec("attention (qwen3)", "prompt attention", T, lambda: ops.flash_attn_varlen(q, kk[None], vv[None], bt, cu, kl, T, max_kv_len=T),
                T * (2 * nq + 2 * nk) * 2, 4.0 * pairs(T, T) * hq * D)
            dq, dkk, dvv, gate = rnd(T, 2 * dh, dd), rnd(T, 2 * dg, dd), rnd(T, dg, ddv), rnd(T, dh)
            for window in (0, 4096, 1024):
                p = pairs(T, window or T)
                rec(f"sigmoid attention, window {window or 'none'}", "prompt attention", T,
                    lambda: ops.window_attention_prompt(q, kk, vv, sig, D ** -0.5, None, cu, zero, zero, T, window), T * (2 * nq + 2 * nk) * 2, 4.0 * p * hq * D)
                rec(f"differential attention, window {window or 'none'}", "prompt attention", T,
                    lambda: ops.window_attention_prompt(dq, dkk, dvv, diff, dd ** -0.5, gate, cu, zero, zero, T, window),
                    T * (2 * dh * dd + dh * ddv + 2 * dg * dd + dg * ddv) * 2, 4.0 * p * dh * (dd + ddv))
        else:
            R = CTX
            q, kk, vv = rnd(T, hq, D), rnd(T, R, hkv, D), rnd(T, R, hkv, D)
            at = torch.full((T,), 3 * R + 100, dtype=torch.int64, device=dev)
            bt, lens, sl = ops.dense_block_table(T, dev), torch.full((T,), R, dtype=torch.int32, device=dev), torch.arange(T, dtype=torch.int32, device=dev)
            rec("attention (qwen3)", "decode attention", T, lambda: ops.gqa_fwd_batch_decode(q, kk, vv, None, None, lens, bt), T * R * nk * 2 * 2)
            rec("sigmoid attention", "decode attention", T, lambda: ops.window_attention_decode(q, kk, vv, sig, D ** -0.5, None, sl, at), T * R * nk * 2 * 2)
            dq, dkk, dvv, gate = rnd(T, 2 * dh, dd), rnd(T, R, 2 * dg, dd), rnd(T, R, dg, ddv), rnd(T, dh)
            rec("differential attention", "decode attention", T, lambda: ops.window_attention_decode(dq, dkk, dvv, diff, dd ** -0.5, gate, sl, at),
                T * R * dg * (2 * dd + ddv) * 2)
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
