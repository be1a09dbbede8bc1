"""Small, self-terminating workloads for Nsight Compute captures of single kernels (one GPU, a few launches).

  python benchmarks/ncu_case.py gemm      # tcgen05 GEMM 8192 x 4096 x 4096 (inputs + output ~160 MB > L2)
  python benchmarks/ncu_case.py skinny    # decode GEMM 32 x 5120 x 3200, split-K
  python benchmarks/ncu_case.py decode    # split-KV decode attention, 16 seqs x 4096 tokens, 8 q heads / 1 kv head
  python benchmarks/ncu_case.py gemv      # decode GEMV 1 x 6400 x 5120 (65 MB of weights per launch, 4 weight copies)
  python benchmarks/ncu_case.py gemm_fp8  # block-scaled e4m3 GEMM 8192 x 3584 x 8192 (pair kernel, ~150 MB)
  python benchmarks/ncu_case.py moe       # grouped GEMM with in-kernel row gather: 8192 tokens, top-2 of 16 experts, 2048 x 2048
  python benchmarks/ncu_case.py gdn       # chunk-parallel gated delta rule, 8192 tokens x 16 heads
  python benchmarks/ncu_case.py gla       # chunk-parallel gated linear attention, 8192 tokens x 16 heads, 128 x 128 states
  python benchmarks/ncu_case.py delta     # chunk-parallel gated delta rule with convolutions, 8192 tokens x 16 heads, 128 x 128 states
  python benchmarks/ncu_case.py hyper     # pass over 4 residual streams between two sublayers, 8192 tokens, width 2048
  python benchmarks/ncu_case.py ssd       # chunk-parallel state space layer with convolutions, 8192 tokens x 64 heads, 128 x 64 states
  python benchmarks/ncu_case.py sandwich  # sublayer between two norms, 8192 tokens, width 4096
  python benchmarks/ncu_case.py sigmoid   # sigmoid prompt attention, 8192 tokens, window 4096, 32 heads / 8 kv heads of 128
  python benchmarks/ncu_case.py differential  # differential prompt attention, 8192 tokens, window 4096, 32 heads / 8 kv heads of 2 x 64 / 128
  python benchmarks/ncu_case.py window_decode  # sigmoid decode attention over full rings, 64 seqs x 4096 positions, 32 heads / 8 kv heads of 128
  python benchmarks/ncu_case.py tied      # tied-KV block decode attention, 64 seqs x 4096 positions, 32 q heads / 4 kv heads
  python benchmarks/ncu_case.py latent_decode   # latent decode attention, 64 seqs x 4096 tokens, 32 heads, rows of 512 + 64
  python benchmarks/ncu_case.py latent_prefill  # latent prompt attention, 8192 tokens, 8 heads of 128 + 64 / 128
"""
import sys

import torch

sys.path.insert(0, __import__("os").path.dirname(__import__("os").path.dirname(__import__("os").path.abspath(__file__))))

from triton_distributed_b200 import ops  # noqa: E402


def main():
    case = sys.argv[1] if len(sys.argv) > 1 else "gemm"
    if case == "gemm":
        a = torch.randn(8192, 4096, device="cuda", dtype=torch.bfloat16)
        b = (torch.randn(4096, 4096, device="cuda") * 0.02).to(torch.bfloat16)
        out = torch.empty(8192, 4096, device="cuda", dtype=torch.bfloat16)
        for _ in range(3):
            ops.gemm(a, b, out=out)
    elif case == "skinny":
        a = torch.randn(32, 3200, device="cuda", dtype=torch.bfloat16)
        b = (torch.randn(5120, 3200, device="cuda") * 0.02).to(torch.bfloat16)
        for _ in range(3):
            ops.skinny_gemm(a, b)
    elif case == "gemv":
        ws = [(torch.randn(6400, 5120, device="cuda") * 0.02).to(torch.bfloat16) for _ in range(4)]
        x = torch.randn(1, 5120, device="cuda", dtype=torch.bfloat16)
        out = torch.empty(1, 6400, device="cuda", dtype=torch.bfloat16)
        for w in ws:
            ops.gemv_fused(x, w, out=out)
    elif case == "gemm_fp8":
        a = torch.randn(8192, 8192, device="cuda", dtype=torch.bfloat16)
        b = (torch.randn(3584, 8192, device="cuda") * 0.02).to(torch.bfloat16)
        a_q, a_s = ops.quantize_act_1x128(a)
        b_q, b_s = ops.quantize_weight_128x128(b)
        for _ in range(3):
            ops.gemm_fp8_blockscaled(a_q, a_s, b_q, b_s)
    elif case == "moe":
        T, E, k, H, N = 8192, 16, 2, 2048, 2048
        x = torch.randn(T, H, device="cuda", dtype=torch.bfloat16)
        w = (torch.randn(E, N, H, device="cuda") * 0.02).to(torch.bfloat16)
        ids = torch.randint(0, E, (T, k), device="cuda", dtype=torch.int32)
        srt = ops.sort_topk_ids_align_block_size(ids, E)
        for _ in range(3):
            ops.group_gemm_gather(x, w, srt, k)
    elif case == "gdn":
        import torch.nn.functional as F
        T, H, K, V = 8192, 16, 128, 128
        q = torch.randn(1, T, H, K, device="cuda", dtype=torch.bfloat16)
        kk = F.normalize(torch.randn(1, T, H, K, device="cuda"), dim=-1).to(torch.bfloat16)
        v = torch.randn(1, T, H, V, device="cuda", dtype=torch.bfloat16)
        beta = torch.rand(1, T, H, device="cuda").to(torch.bfloat16)
        g = F.logsigmoid(torch.rand(1, T, H, device="cuda"))
        for _ in range(2):
            ops.chunk_gated_delta_rule_fwd(q, kk, v, g, beta, K ** -0.5, impl="chunk")
    elif case == "gla":
        T, H, dk, dv = 8192, 16, 128, 128
        qkvg = torch.randn(T, 2 * H * (dk + dv), device="cuda", dtype=torch.bfloat16)
        low, a2 = torch.randn(T, 16, device="cuda"), torch.randn(16, H * dk, device="cuda")
        bias, norm = torch.full((H * dk,), 2.0, device="cuda"), torch.ones(dv, device="cuda")
        state = torch.zeros(1, H, dk, dv, device="cuda")
        slot, pos0 = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int64, device="cuda")
        cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
        tabs = ops.gla_chunk_tables([0, T], "cuda")
        for _ in range(2):
            ops.gated_linear_attention(qkvg, low, a2, bias, 16.0, norm, state, slot, pos0, cu, dv, dk ** -0.5, 1e-5, tabs)
    elif case == "delta":
        T, H, dk, dv, taps = 8192, 16, 128, 128, 4
        C = H * (2 * dk + dv)
        z, ab = torch.randn(T, C + H * dv, device="cuda", dtype=torch.bfloat16), torch.randn(T, 2 * H, device="cuda")
        conv_w, norm = torch.randn(C, taps, device="cuda"), torch.ones(dv, device="cuda")
        alog, dt = torch.zeros(H, device="cuda"), torch.full((H,), -2.0, device="cuda")
        state, ring = torch.zeros(1, H, dk, dv, device="cuda"), torch.zeros(1, taps, C, device="cuda", dtype=torch.bfloat16)
        slot, pos0 = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int64, device="cuda")
        cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
        tabs = ops.gla_chunk_tables([0, T], "cuda")
        for _ in range(2):
            ops.gated_delta_rule(z, ab, conv_w, alog, dt, norm, state, ring, slot, pos0, cu, H, dv, dk ** -0.5, 1e-5, tabs)
    elif case == "hyper":
        T, S, W = 8192, 4, 2048
        x, y = torch.randn(T, S, W, device="cuda"), torch.randn(T, W, device="cuda", dtype=torch.bfloat16)
        one = torch.ones(S, device="cuda")
        hc = ops.HyperWeights(one / S, one, torch.eye(S, device="cuda"))
        for _ in range(3):
            ops.hyper_step(x, (hc, ops.SublayerOutput(y)), (hc.inp, torch.ones(W, device="cuda")), W, 1e-5, torch.bfloat16)
    elif case == "ssd":
        T, H, G, N, dv, taps = 8192, 64, 8, 128, 64, 4
        C = H * dv + 2 * G * N
        z = torch.randn(T, C + H, device="cuda", dtype=torch.bfloat16)
        w = ops.SsdWeights(torch.randn(C, taps, device="cuda"), torch.randn(C, device="cuda"), torch.zeros(H, device="cuda"), torch.full((H,), -2.0, device="cuda"),
                           torch.ones(H, device="cuda"))
        state, ring = torch.zeros(1, H, N, dv, device="cuda"), torch.zeros(1, taps, C, device="cuda", dtype=torch.bfloat16)
        slot, pos0 = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int64, device="cuda")
        cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
        tabs = ops.gla_chunk_tables([0, T], "cuda")
        for _ in range(2):
            ops.state_space(z, C, w, state, ring, slot, pos0, cu, G, tabs)
    elif case == "sandwich":
        T, W = 8192, 4096
        x, y, one = torch.randn(T, W, device="cuda"), torch.randn(T, W, device="cuda", dtype=torch.bfloat16), torch.ones(1, device="cuda")
        for _ in range(3):
            ops.sandwich_step(x, (y, one), one, W, 1e-5, torch.bfloat16)
    elif case in ("sigmoid", "differential", "window_decode"):
        T, H, G, window = (64 if case == "window_decode" else 8192), 32, 8, 4096
        m, dk, dv = (2, 64, 128) if case == "differential" else (1, 128, 128)
        w = ops.DifferentialWeights(0.6, 0.5, 1e-5, dv)
        if m == 1:
            w = ops.SigmoidWeights(ops.distance_table(torch.full((H,), 0.3), torch.full((H,), 0.5), torch.full((H,), -3.0), window).cuda())
        rows = (T, window) if case == "window_decode" else (T,)
        q, k, v = (torch.randn(*s, device="cuda", dtype=torch.bfloat16) for s in ((T, H * m, dk), (*rows, G * m, dk), (*rows, G, dv)))
        i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device="cuda")   # noqa: E731
        for _ in range(3):
            if case == "window_decode":
                ops.window_attention_decode(q, k, v, w, dk ** -0.5, None, i32(*range(T)), torch.full((T,), 3 * window, dtype=torch.int64, device="cuda"))
            else:
                ops.window_attention_prompt(q, k, v, w, dk ** -0.5, None, i32(0, T), i32(0), i32(0), T, window)
        ops.check_attention_errors()
    elif case == "tied":
        B, Hq, Hkv, D, L = 64, 32, 4, 128, 4096
        k = torch.randn(B, L, Hkv, D, device="cuda", dtype=torch.bfloat16)
        scale = torch.ones(B, L, device="cuda")
        q = torch.randn(B, Hq, D, device="cuda", dtype=torch.bfloat16)
        bt, lens = ops.dense_block_table(B, "cuda"), torch.full((B,), L, dtype=torch.int32, device="cuda")
        sink = torch.zeros(Hq, device="cuda")
        for _ in range(3):
            ops.tied_attn_decode(q, k, scale, bt, lens, L, ops.pick_tied_splits(B, Hkv, 1, L), sink)
    elif case == "latent_decode":
        B, H, R, r, L = 64, 32, 512, 64, 4096
        cache = torch.randn(B, L, R + r, device="cuda", dtype=torch.bfloat16)
        q = torch.randn(B, H, R + r, device="cuda", dtype=torch.bfloat16)
        slots, lens = torch.arange(B, dtype=torch.int32, device="cuda"), torch.full((B,), L, dtype=torch.int32, device="cuda")
        for _ in range(3):
            ops.latent_decode(q, cache, slots, lens, R, (R + r) ** -0.5)
        ops.check_latent_errors()
    elif case == "latent_prefill":
        T, H, d, r, dv, R = 8192, 8, 128, 64, 128, 512
        z = torch.randn(T, H * (d + r + dv), device="cuda", dtype=torch.bfloat16)
        k, vt = (torch.randn(*s, device="cuda", dtype=torch.bfloat16) for s in ((T, H * d), (H * dv, T)))
        ctx = torch.randn(T, R + r, device="cuda", dtype=torch.bfloat16)
        i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device="cuda")   # noqa: E731
        for _ in range(3):
            ops.latent_prefill(z, k, ctx, vt, i32(0, T), i32(0), i32(T), i32(0), T, H, d, r, dv, (d + r) ** -0.5, z[:, H * (d + r):])
        ops.check_latent_errors()
    elif case == "decode":
        B, Hq, Hkv, D, L = 16, 8, 1, 128, 4096
        k = torch.randn(B, L, Hkv, D, device="cuda", dtype=torch.bfloat16)
        v = torch.randn(B, L, Hkv, D, device="cuda", dtype=torch.bfloat16)
        q = torch.randn(B, Hq, D, device="cuda", dtype=torch.bfloat16)
        bt = ops.dense_block_table(B, "cuda")
        lens = torch.full((B,), L, dtype=torch.int32, device="cuda")
        for _ in range(3):
            ops.gqa_fwd_batch_decode(q, k, v, None, None, lens, bt)
    torch.cuda.synchronize()
    print("done", case)


if __name__ == "__main__":
    main()
