"""Lisenex (latent attention, parallel layers) against the closest existing model (Vasolix) at equal layer sizes, random weights,
one GPU: prefill and decode throughput of a few layers, and the kernels one by one beside the like kernel of the other model.

    python benchmarks/bench_latent.py [--size 30b-a3b,1b] [--parts prefill,decode,kernels]

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
from triton_distributed_b200.models import LisenexLLM, VasolixLLM  # noqa: E402
from triton_distributed_b200.models.lisenex import DenseSpec, LatentAttnSpec, RoutedSpec, latent_stack  # noqa: E402
from triton_distributed_b200.utils import device_time_ms, load_peaks  # noqa: E402
from benchmarks import bench_hybrid as hybrid  # noqa: E402
from benchmarks.bench_hybrid import CTX, LAYERS, VOCAB  # noqa: E402

# unrotated, rotated and value dimensions of a head, latent size; groups of router outputs, identity experts.  The rest (width,
# heads, experts) is that of the other model's sizes.
SIZES = {"30b-a3b": (128, 64, 128, 512, (8, 4), 8), "1b": (64, 32, 64, 256, (4, 2), 4)}


def arch(size):
    W, hq, _, _, _, _, _, E, top, ff, sff = hybrid.SIZES[size]
    d, r, dv, R, groups, ident = SIZES[size]
    attn = LatentAttnSpec(hq, d, r, dv, R, (d + r) ** -0.5, 1e6)
    # every other layer uses the rows of the one before; the router has as many outputs as the other model's
    return latent_stack(f"lisenex-{size}", VOCAB, W, ("Mm" * LAYERS)[:LAYERS], attn, DenseSpec(3 * W), RoutedSpec(E - ident, top, ff, sff, ident, *groups))


def bench_models(size, parts):
    out = []
    models = {"lisenex": (LisenexLLM, arch(size)), "vasolix": (VasolixLLM, hybrid.archs(size)["vasolix"])}
    for name, (cls, a) in models.items():
        model = hybrid.make(cls, a, 16384)
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
    ops.check_latent_errors()
    return out


# ------------------------------------------------------------------ kernels
def bench_kernels(size):
    W, H, hkv, D, block, _, _, E, top, ff, sff = hybrid.SIZES[size]
    d, r, dv, R, groups, ident = SIZES[size]
    n_exp = E - ident
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
        # stream
        x, mix, y, sh = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T * top, W), rnd(T, W)
        xb, wf = rnd(T, W), torch.ones(W, device=dev)
        rec("parallel_add + two norms", "norm", T, lambda: ops.parallel_add(x, mix, ops.FeedForward(xb), wf, wf, W, 1e-5, bf), T * W * (4 + 4 + 4 * 2))
        rec("postnorm_add (vasolix)", "norm", T, lambda: ops.postnorm_add(x, xb, mix, wf, W, 1e-5), T * W * (4 + 4 + 2 + 2))
        # router
        rw, corr = rnd(E, W), torch.zeros(E, device=dev)
        rec("softmax_router", "router", T, lambda: ops.softmax_router(xb, rw, corr, top, *groups), (T + E) * W * 2, 2.0 * T * E * W)
        rec("sigmoid_router (vasolix)", "router", T, lambda: ops.sigmoid_router(xb, rw, top), (T + E) * W * 2, 2.0 * T * E * W)
        ids, wts = ops.softmax_router(xb, rw * W ** -0.5, corr, top, *groups)
        if T == 8192:
            ff_rows = ops.FeedForward(y, top, ids, wts, n_exp, xb, sh)
            rec("parallel_add + two norms, expert rows", "norm", T, lambda: ops.parallel_add(x, mix, ff_rows, wf, wf, W, 1e-5, bf),
                T * W * (4 + 4 + 3 * 2 + 2 * (top + 1)))
            rec("postnorm_add, expert rows (vasolix)", "norm", T, lambda: ops.postnorm_add(x, xb, y, wf, W, 1e-5, top, sh, wts[:, 0].contiguous()),
                T * W * (4 + 4 + 2 + 2 * (top + 1)))
        # experts
        up, down = rnd(n_exp, 2 * ff, W), rnd(n_exp, W, ff)
        used = int((ids.unique() < n_exp).sum())
        pairs = int((ids < n_exp).sum())
        ids2, wts2, gate2 = ops.sigmoid_router(xb, rnd(E + 1, W) * W ** -0.5, top, True)
        used2 = ids2.unique().numel()
        up2, down2 = rnd(E, ff, W), rnd(E, W, ff)
        if T <= ops.EXPERT_GEMV_MAX_T:
            su, sd = rnd(2 * sff, W), rnd(W, sff)
            rec("gated experts gemv (incl. shared)", "experts", T, lambda: ops.gated_experts_gemv(xb, up, down, ids, wts, su, sd, ident),
                (used * ff + sff) * W * 2 * 3)
            rec("squared-ReLU experts gemv (vasolix)", "experts", T, lambda: ops.relu2_experts_gemv(xb, up2, down2, ids2, wts2, su[:sff], sd, gate2),
                (used2 * ff + sff) * W * 2 * 2)
        else:
            def grouped():
                srt = ops.sort_topk_ids_align_block_size(ids, n_exp)
                h = ops.silu_mul(ops.group_gemm_gather(xb, up, srt, a_row_div=top, scatter_out=True))
                return ops.group_gemm_gather(h, down, srt, a_row_div=1, scatter_out=True, row_weight=wts)

            def grouped2():
                srt = ops.sort_topk_ids_align_block_size(ids2, E)
                h = ops.relu2(ops.group_gemm_gather(xb, up2, srt, a_row_div=top, scatter_out=True), wts2.reshape(-1))
                return ops.group_gemm_gather(h, down2, srt, a_row_div=1, scatter_out=True)
            rec("gated experts grouped GEMM (without shared)", "experts", T, grouped, used * ff * W * 6 + T * W * 2 * (1 + top), 6.0 * pairs * ff * W)
            rec("squared-ReLU experts grouped GEMM (vasolix)", "experts", T, grouped2, used2 * ff * W * 4 + T * W * 2 * (1 + top), 4.0 * T * top * ff * W)
        del up, down, up2, down2
        # dense feed-forward's activation
        h, hb = rnd(T, 3 * W), torch.zeros(3 * W, device=dev)
        rec("relu2 with bias", "activation", T, lambda: ops.relu2(h, None, hb), T * 3 * W * 4)
        rec("relu2 (vasolix)", "activation", T, lambda: ops.relu2(h, None), T * 3 * W * 4)
        # what stands around the attention
        nq, nk = H * D, hkv * D
        z = rnd(T, H * (d + r) + R + r + H * dv)
        gate = z[:, H * (d + r) + R + r:]
        tab, rows = ops.rope_table(1e6, r, r, max(CTX, T), dev), torch.arange(T, device=dev)
        nw, cache1 = torch.ones(R, device=dev), torch.empty(T, R + r, device=dev, dtype=bf)
        qkg = rnd(T, 2 * nq + nk)
        kc, sc, qw = torch.empty(T, nk, device=dev, dtype=bf), torch.empty(T, device=dev), torch.ones(nq, device=dev)
        uk_t, uv = rnd(H, R, d), rnd(H, dv, R)
        if T == 8192:
            ctx = torch.empty(T, R + r, device=dev, dtype=bf)
            rec("latent_rotate", "q / k preparation", T, lambda: ops.latent_rotate(z, H, d, r, nw, R, R, 1e-5, tab, rows, (cache1, rows), (ctx, rows)),
                T * 2 * (2 * H * r + 3 * (R + r)))
            rec("qk_norm_tied (vasolix)", "q / k preparation", T, lambda: ops.qk_norm_tied(qkg, qw, nk, nq, nk, 1e-5, (kc, sc, rows), (kc, sc, rows)),
                T * 2 * (2 * nq + 3 * nk))
        else:
            rec("latent_absorb", "q / k preparation", T, lambda: ops.latent_absorb(z, uk_t, r, nw, R, 1e-5, tab, rows, (cache1, rows)),
                2 * (H * R * d + T * (H * (d + r) + H * (R + r) + 2 * (R + r))))
            rec("qk_norm_tied (vasolix)", "q / k preparation", T, lambda: ops.qk_norm_tied(qkg, qw, nk, nq, nk, 1e-5, (kc, sc, rows)), T * 2 * 2 * (nq + nk))
        # attention
        sink = torch.zeros(H, device=dev)
        from triton_distributed_b200.models import HybridCache, TiedKVSpec
        if T == 8192:
            k, vt, lens = rnd(T, H * d), rnd(H * dv, T), [T]
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)   # noqa: E731
            cu, zero, kl = i32([0, T]), i32([0]), i32(lens)
            rec("latent prompt attention", "prefill attention", T,
                lambda: ops.latent_prefill(z, k, ctx, vt, cu, zero, kl, zero, T, H, d, r, dv, (d + r) ** -0.5, gate),
                T * 2 * (H * (2 * d + r + 3 * dv) + r), T * (T + 1.0) * H * (d + r + dv))
            rec("keys and values of the prompt (two GEMMs)", "expansion", T, lambda: (torch.matmul(ctx[:, :R], uk_t.view(H * d, R).t()),
                                                                                     torch.matmul(uv.view(H * dv, R), ctx[:, :R].t())),
                T * 2 * (H * (d + dv) + 2 * R), 2.0 * T * R * H * (d + dv))
            spec = TiedKVSpec(hkv, D, block)
            bp = HybridCache([spec], 1, T, bf, dev).plan([0], [T]).blocks(spec)
            pages, scale, q = rnd(bp.pages, bp.page_rows, hkv, D), torch.ones(bp.pages, bp.page_rows, device=dev), rnd(T, H, D)
            kv_pairs = (T // block) * block * (block + 1) / 2
            rec("tied block attention (vasolix)", "prefill attention", T,
                lambda: ops.tied_attn_varlen(q, pages, scale, bp.block_table, bp.cu, bp.q_pos0, bp.kv_lens, bp.max_q, bp.max_kv, sink, qkg[:, nq + nk:]),
                T * (3 * nq + nk) * 2, 4.0 * kv_pairs * H * D)
        else:
            cache = rnd(T, CTX, R + r)
            slots, kl = torch.arange(T, dtype=torch.int32, device=dev), torch.full((T,), CTX, dtype=torch.int32, device=dev)
            q = rnd(T, H, R + r)
            o, ml = ops.latent_decode(q, cache, slots, kl, R, (d + r) ** -0.5)
            rec("latent decode attention", "decode attention", T, lambda: ops.latent_decode(q, cache, slots, kl, R, (d + r) ** -0.5),
                T * CTX * (R + r) * 2, 2.0 * T * CTX * H * (2 * R + r))
            rec("latent_out (merge, W_uv, gate)", "decode attention", T, lambda: ops.latent_out(o, ml, uv, gate), 2 * H * R * dv + T * H * (4 * R * o.shape[2] + 4 * dv))
            n = min(block, CTX)
            kk, scale, qd = rnd(T, n, hkv, D), torch.ones(T, n, device=dev), rnd(T, H, D)
            bt, lens = ops.dense_block_table(T, dev), torch.full((T,), n, dtype=torch.int32, device=dev)
            sp = ops.pick_tied_splits(T, hkv, (H // hkv + 15) // 16, n)
            rec("tied decode attention (vasolix)", "decode attention", T, lambda: ops.tied_attn_decode(qd, kk, scale, bt, lens, n, sp, sink, qkg[:, nq + nk:]),
                T * n * (nk * 2 + 4))
        torch.cuda.empty_cache()
    ops.check_latent_errors()
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
