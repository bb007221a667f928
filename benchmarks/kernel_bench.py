"""Micro-benchmarks of the hot kernels, one case per invocation (also the workload for
``ncu`` captures: each case launches its kernel a handful of times on inputs larger than
L2 but of at most a few GB).

    python benchmarks/kernel_bench.py --case gemm_prefill   [--iters 20]
    python benchmarks/kernel_bench.py --case attn_decode --no-time   # for ncu: 3 launches only

Timing: CUDA events around each launch, median reported, with achieved TFLOP/s or GB/s
against the measured peaks in MEASURED_PEAKS.json when present. Before the first event of an
iteration the stream is given ~200 us of busy-waiting to chew on, so that the host has queued
the event pair and the launch by the time the device reaches them: the interval is then the
device's own time for the kernel, not the host's launch path (which for a 10 us decode kernel
would otherwise be most of the number). Every case keeps several
copies of its large operand (weights, KV cache, activations) whose total exceeds twice the
L2 capacity and rotates through them, so each timed launch reads its operands from HBM
without the write-back traffic that a dirty flush buffer would add to the measurement.
"""

import argparse
import json
import math
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from arcticinference_b200 import ops  # noqa: E402

DEV = "cuda:0"


def peaks():
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return d.get("hbm_gbs", 6650.0), d.get("bf16_tflops", 1590.0), "measured"
    return 6650.0, 1590.0, "fallback"


def R(*s):
    return (torch.randn(*s, device=DEV) * 0.05).to(torch.bfloat16)


ROTATE_BYTES = 320 << 20      # > 2 x the 126 MB L2


def copies_for(nbytes: int) -> int:
    return max(1, min(64, -(-ROTATE_BYTES // max(int(nbytes), 1))))


def timeit(fn, iters, warm=3, copies=1):
    """``fn(i)`` launches the case on operand copy ``i % copies`` (``fn()`` when copies == 1:
    such a case must stream more than L2 by itself)."""
    call = (lambda i: fn()) if copies == 1 else (lambda i: fn(i % copies))
    for i in range(max(warm, copies)):
        call(i)
    torch.cuda.synchronize()
    ts = []
    for i in range(iters):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda._sleep(400000)     # head start for the host (~200 us of device time)
        e0.record()
        call(i)
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1))
    ts.sort()
    return ts[len(ts) // 2]


def paged(q_lens, kv_lens, Hq=32, Hkv=8, D=128, bs=64):
    T = sum(q_lens)
    nblk = [(k + bs - 1) // bs for k in kv_lens]
    bt = torch.zeros(len(q_lens), max(nblk), dtype=torch.int32)
    o = 1
    for i, n in enumerate(nblk):
        bt[i, :n] = torch.arange(o, o + n)
        o += n
    q, kc, vc = R(T, Hq * D), R(o, Hkv, bs, D), R(o, Hkv, bs, D)
    meta = ops.build_attention_metadata(q_lens, kv_lens, bt.to(DEV), Hq // Hkv, Hq, D, DEV)
    return q, kc, vc, meta


CASES = {
    # decode in latent space: heads, latent width, sequences, cached tokens
    "latent_512": ("latent", (16, 512, 128, 2000)),
    "latent_256": ("latent", (40, 256, 128, 2000)),
    "latent_128": ("latent", (16, 128, 128, 2000)),
    # mixture of experts (gate / up with the activation): tokens, width, ff, experts, per token
    "experts_prefill": ("experts", (8192, 2048, 1408, 64, 6)),
    "experts_decode": ("experts", (128, 2048, 1408, 64, 6)),
    "route_prefill": ("route", (8192, 2048, 64, 6)),
    "route_decode": ("route", (128, 2048, 64, 6)),
    "stream_norm": ("stream_norm", (8192, 4096)),
    "latent_norm_cache": ("latent_norm", (8192, 512)),
    # attention with sink, output gate and a mask (kind, positions): query and cached lengths
    "masked_prefill_4x2048": ("masked", ([2048] * 4, [2048] * 4, "chunk", 4096)),
    "masked_prefill_chunks_1024": ("masked", ([2048] * 4, [2048] * 4, "chunk", 1024)),
    "masked_decode_128": ("masked", ([1] * 128, [2000] * 128, "chunk", 4096)),
    "masked_decode_window_128": ("masked", ([1] * 128, [2000] * 128, "window", 128)),
    # expanded latents with a rotated part: keys of 192, values of 128
    "expanded_192_4x2048": ("expanded", (32, [2048] * 4, 4096)),
    # decode in latent space with 64 key-only columns under a window
    "latent_rot_512": ("latent_rot", (32, 512, 128, 2000, 4096)),
    "latent_rot_512_window_128": ("latent_rot", (32, 512, 128, 2000, 128)),
    # query / key norms, rotation, cache write: tokens, heads, K/V heads, dimensions, rotated
    "head_rope": ("head_rope", (8192, 32, 8, 128, 32)),
    "head_rope_64": ("head_rope", (8192, 40, 8, 64, 16)),
    "latent_rope": ("latent_rope", (8192, 32, 128, 64, 512)),
    "stream_sandwich": ("sandwich", (8192, 4096)),
    # name: (kind, params)
    "gemm_prefill": ("gemm", (8192, 28672, 4096)),
    "gemm_prefill_qkv": ("gemm", (8192, 6144, 4096)),
    "gemm_prefill_down": ("gemm", (8192, 4096, 14336)),
    "gemm_decode": ("gemm", (32, 28672, 4096)),
    "gemm_decode_128": ("gemm", (128, 28672, 4096)),
    "gemm_decode_128_down": ("gemm", (128, 4096, 14336)),
    "gemm_decode_o": ("gemm", (32, 4096, 4096)),
    "gemm_decode_down": ("gemm", (32, 4096, 14336)),
    "gemm_mid": ("gemm", (512, 28672, 4096)),
    "gemm_fp8_prefill": ("gemm_fp8", (8192, 28672, 4096)),
    "gemm_fp8_mid": ("gemm_fp8", (256, 28672, 4096)),
    "gemm_fp8_decode": ("gemm_fp8", (32, 28672, 4096)),
    "gemm_fp8_decode_128": ("gemm_fp8", (128, 28672, 4096)),
    "gemm_fp8_decode_o": ("gemm_fp8", (32, 4096, 4096)),
    "gemm_fp8_decode_down": ("gemm_fp8", (32, 4096, 14336)),
    # W8A8 with per-token / per-feature scales (activations already quantised, as the fused
    # norm / SiLU kernels hand them over); "*_w8a8_block" is the block-scaled kernel itself
    "gemm_fp8row_prefill": ("gemm_fp8row", (8192, 28672, 4096)),
    "gemm_fp8row_prefill_qkv": ("gemm_fp8row", (8192, 6144, 4096)),
    "gemm_fp8row_prefill_down": ("gemm_fp8row", (8192, 4096, 14336)),
    "gemm_fp8row_mid": ("gemm_fp8row", (512, 28672, 4096)),
    "gemm_fp8row_decode": ("gemm_fp8row", (32, 28672, 4096)),
    "gemm_fp8row_decode_128": ("gemm_fp8row", (128, 28672, 4096)),
    "gemm_fp8row_decode_128_down": ("gemm_fp8row", (128, 4096, 14336)),
    "gemm_fp8row_decode_o": ("gemm_fp8row", (32, 4096, 4096)),
    "gemm_fp8row_decode_128_tiled": ("gemm_fp8row_tiled", (128, 28672, 4096)),
    "gemm_fp8row_decode_128_down_tiled": ("gemm_fp8row_tiled", (128, 4096, 14336)),
    "gemm_fp8row_prefill_tiled": ("gemm_fp8row_tiled", (8192, 28672, 4096)),
    "gemm_fp8row_decode_qkv": ("gemm_fp8row", (128, 6144, 4096)),
    "gemm_w8a8_block_prefill": ("gemm_fp8blk", (8192, 28672, 4096)),
    "attn_prefill": ("attn", ([8192], [8192])),
    "attn_prefill_4x2048": ("attn", ([2048] * 4, [2048] * 4)),
    "attn_decode": ("attn", ([1] * 32, [2000] * 32)),
    "attn_decode_128": ("attn", ([1] * 128, [2000] * 128)),
    "attn_decode_128_short": ("attn", ([1] * 128, [144] * 128)),
    "attn_decode_long": ("attn", ([1] * 8, [8000] * 8)),
    "attn_verify": ("attn", ([4] * 32, [2000] * 32)),
    "rmsnorm": ("rmsnorm", (8192, 4096)),
    "rmsnorm_quant": ("rmsnorm_q", (8192, 4096)),
    "silu_mul": ("silu", (8192, 14336)),
    "silu_mul_quant": ("silu_q", (8192, 14336)),
    "quant_fp8_row": ("quant_row", (8192, 4096)),
    # recurrent layers (keys and values of 128; the matrix memory's keys of 64): heads, sequences, tokens
    "delta_prefill_4x2048": ("delta", (32, 4, 2048)),
    "delta_prefill_4x256": ("delta", (32, 4, 256)),
    "delta_decode_128": ("delta", (32, 128, 1)),
    "delta_decode_64": ("delta", (32, 64, 1)),
    "forget_prefill_4x2048": ("forget", (32, 4, 2048)),
    "forget_prefill_4x256": ("forget", (32, 4, 256)),
    "forget_decode_128": ("forget", (32, 128, 1)),
    "poly_norm_prefill": ("poly", (8192, 21504)),
    "poly_norm_prefill_9600": ("poly", (8192, 9600)),
    "poly_norm_decode": ("poly", (128, 21504)),
    "soft_cap_decode": ("soft_cap", (128, 128256)),
    "stream_pre": ("pre", (8192, 4096)),
    "memory_prefill_4x2048": ("memory", (16, 4, 2048)),
    "memory_decode_128": ("memory", (16, 128, 1)),
}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--case", required=True,
                    help="one of: %s (or several, comma-separated; 'all' for every case)"
                         % ", ".join(sorted(CASES)))
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--no-time", action="store_true", help="three plain launches (for ncu)")
    ap.add_argument("--splits", type=int, default=0,
                    help="force the split-K factor of the bf16 GEMM cases (0 = the kernel's choice)")
    ap.add_argument("--tile-keys", type=int, default=0,
                    help="force the key-tile size (64 or 128) of the attention cases")
    a = ap.parse_args()
    names = sorted(CASES) if a.case == "all" else a.case.split(",")
    for name in names:
        if name not in CASES:
            raise SystemExit("unknown case %r" % name)
        run_case(a, name)
        torch.cuda.empty_cache()


def run_case(a, case):
    hbm, tf, src = peaks()
    kind, prm = CASES[case]
    if kind == "gemm":
        M, N, K = prm
        nc = copies_for(2 * N * K)
        x, ws = R(M, K), [R(N, K) for _ in range(nc)]
        fn = lambda i=0: ops.linear(x, ws[i], force_splits=a.splits)
        flops, byts = 2.0 * M * N * K, 2.0 * (M * K + N * K + M * N)
    elif kind == "gemm_fp8":
        from arcticinference_b200.models import quant
        M, N, K = prm
        nc = copies_for(N * K)
        x, ws = R(M, K), [quant.quantize_weight_fp8(R(N, K)) for _ in range(nc)]
        fn = lambda i=0: ops.linear(x, ws[i])
        flops, byts = 2.0 * M * N * K, 2.0 * (M * K + M * N) + 1.0 * N * K
    elif kind in ("gemm_fp8row", "gemm_fp8row_tiled"):
        from arcticinference_b200.models import quant
        M, N, K = prm
        nc = copies_for(N * K)
        xq = ops.quant_fp8_row(R(M, K))
        tiled = kind != "gemm_fp8row"     # the "_tiled" cases store 16-row x 128-byte tiles
        ws = [quant.quantize_weight_fp8_row(R(N, K), tiled=tiled) for _ in range(nc)]
        for w_ in ws:
            ops.mark_static(w_)      # parameters, as in a loaded model
        fn = lambda i=0: ops.linear(xq, ws[i], force_splits=a.splits)
        flops, byts = 2.0 * M * N * K, 1.0 * (M * K + N * K) + 2.0 * M * N
    elif kind == "gemm_fp8blk":
        from arcticinference_b200.models import quant
        M, N, K = prm
        nc = copies_for(N * K)
        x, ws = R(M, K), [quant.quantize_weight_fp8(R(N, K)) for _ in range(nc)]
        fn = lambda i=0: ops.linear_fp8(x, ws[i], mode="w8a8")
        flops, byts = 2.0 * M * N * K, 2.0 * (M * K + M * N) + 1.0 * N * K
    elif kind == "attn":
        ql, kl = prm
        byts = sum(b_ * 8 * 128 * 2 * 2.0 for b_ in kl) + 2.0 * sum(ql) * 32 * 128 * 2
        nc = copies_for(byts)
        sets = [paged(ql, kl) for _ in range(nc)]
        if a.tile_keys:
            for st in sets:
                st[3].tile_keys = a.tile_keys
        fn = lambda i=0: ops.attention(sets[i][0], sets[i][1], sets[i][2], sets[i][3], 32, 8, 128)
        flops = sum(4.0 * a_ * (b_ - a_ / 2.0) * 32 * 128 for a_, b_ in zip(ql, kl))
    elif kind == "latent":
        from arcticinference_b200.ops import latent_ops as lat
        H, rank, n, kl = prm
        byts = 2.0 * n * kl * rank + 4.0 * n * H * rank
        nc = copies_for(byts)
        nb = n * (-(-kl // 64)) + 1
        bt = torch.arange(1, nb, dtype=torch.int32, device=DEV).view(n, -1)
        shape = lat.LatentShape.of(H, rank, torch.bfloat16)
        meta = lat.build_plan(shape, [1] * n, [kl] * n, bt, 64, DEV)
        sets = [(R(n, H * rank), R(nb, 1, 64, rank)) for _ in range(nc)]
        fn = lambda i=0: lat.latent_attention(sets[i][0], sets[i][1], meta, shape, 0.1)
        flops = 4.0 * n * kl * H * rank
    elif kind == "masked":
        from arcticinference_b200.config import MaskSpec
        from arcticinference_b200.ops import head_ops as hd
        ql, kl, name, size = prm
        shape = hd.HeadShape.of(32, 8, 128, 128, torch.bfloat16, MaskSpec(name, size))
        pairs = sum(p - shape.mask.first_key(p) + 1 for n, k in zip(ql, kl) for p in range(k - n, k))
        keys = sum(k - shape.mask.first_key(k - n) for n, k in zip(ql, kl))
        flops, byts = 4.0 * pairs * 32 * 128, 4.0 * keys * 8 * 128 + 6.0 * sum(ql) * 32 * 128
        nc = copies_for(byts)
        sink, sets = torch.zeros(32, device=DEV), []
        for _ in range(nc):
            q, kc, vc, meta = paged(ql, kl)
            sets.append((q, kc, vc, hd.build_plan(shape, ql, kl, meta.block_tables, 64, DEV), R(*q.shape)))
        fn = lambda i=0: hd.head_attention(*sets[i][:4], shape, 0.09, sink, sets[i][4])
    elif kind == "expanded":
        from arcticinference_b200.config import MaskSpec
        H, ql, size = prm
        mask, T = MaskSpec("window", size), sum(ql)
        starts = [sum(ql[:i]) for i in range(len(ql))]
        meta = ops.build_attention_metadata(ql, ql, None, 1, H, 128, DEV, Hkv=H, seq_rows=starts,
                                            allow_split=False, mask=mask)
        q, kv = R(T, H * 192), R(T, H * 320)
        fn = lambda i=0: ops.attention_masked(q, kv[:, :H * 192], kv[:, H * 192:], meta, H, H, 128,
                                              0.07, mask, paged=False, Dk=192)
        nc = 1
        pairs = sum(p - mask.first_key(p) + 1 for n in ql for p in range(n))
        flops, byts = 2.0 * pairs * H * 320, 2.0 * T * H * (192 + 320 + 128)
    elif kind == "latent_rot":
        from arcticinference_b200.config import MaskSpec
        from arcticinference_b200.ops import latent_ops as lat
        H, rank, n, kl, size = prm
        seen = min(kl, size)
        byts = 2.0 * n * seen * (rank + 64) + 2.0 * n * H * (2 * rank + 64)
        nc = copies_for(byts)
        nb = n * (-(-kl // 64)) + 1
        bt = torch.arange(1, nb, dtype=torch.int32, device=DEV).view(n, -1)
        shape = lat.LatentShape.of(H, rank, torch.bfloat16, 64, MaskSpec("window", size))
        meta = lat.build_plan(shape, [1] * n, [kl] * n, bt, 64, DEV)
        sets = [(R(n, H * (rank + 64)), R(nb, 1, 64, rank + 64)) for _ in range(nc)]
        fn = lambda i=0: lat.latent_attention(sets[i][0], sets[i][1], meta, shape, 0.1)
        flops = 2.0 * n * seen * H * (2 * rank + 64)
    elif kind == "head_rope":
        from arcticinference_b200.ops import head_ops as hd
        T, H, G, D, dims = prm
        shape = hd.HeadShape.of(H, G, D, D, torch.bfloat16)
        byts = 2.0 * T * D * (2 * (H + G) + 2 * G)
        nc = copies_for(byts)
        sets = [(R(T, (H + 2 * G) * D), *(R(T // 64, G, 64, D) for _ in range(2))) for _ in range(nc)]
        w, freq = torch.ones(D, device=DEV), torch.rand(dims // 2, device=DEV)
        at = torch.arange(T, device=DEV)
        table = hd.rotary_table(at, freq)
        fn = lambda i=0: hd.head_rope_cache(sets[i][0], shape, D, w, w, table, 1e-6, at, *sets[i][1:])
        flops = 0.0
    elif kind == "latent_rope":
        from arcticinference_b200.ops import head_ops as hd
        from arcticinference_b200.ops import latent_ops as lat
        T, H, dim, rot, rank = prm
        nq = H * (dim + rot)
        byts = 4.0 * T * (H * rot + rank + rot)
        nc = copies_for(byts)
        sets = [(R(T, nq + rank + rot), R(T // 64, 1, 64, rank + rot)) for _ in range(nc)]
        w, freq = torch.ones(rank, device=DEV), torch.rand(rot // 2, device=DEV)
        at = torch.arange(T, device=DEV)
        table = hd.rotary_table(at, freq)
        fn = lambda i=0: lat.latent_rope_cache(sets[i][0], sets[i][0][:, nq:], H, dim + rot, dim, w,
                                               rank, table, 1e-6, at, sets[i][1], rank)
        flops = 0.0
    elif kind in ("delta", "memory"):
        import numpy as np
        from arcticinference_b200.ops import state_ops as states
        H, nseq, n = prm
        T, dv, d = nseq * n, 128, 128 if kind == "delta" else 64
        nk, nv, bf16 = H * d, H * dv, torch.bfloat16
        rnd = lambda *s: torch.randn(*s, device=DEV)
        step = states.StateStep.build(np.asarray([(i * n, n, i + 1, 0 if n > 1 else 5, 0)
                                                  for i in range(nseq)], dtype=np.int32), DEV)
        cols = dv if kind == "delta" else dv + 4
        byts = 2.0 * T * (2 * nk + 3 * nv + (nk if kind == "delta" else 0)) + \
            4.0 * nseq * H * d * cols * (1 if n > 1 else 2)
        flops = (6.0 if kind == "delta" else 4.0) * T * H * d * dv
        nc = copies_for(byts)
        if kind == "delta":
            sh = states.DeltaShape(H, H, d, dv, 4, 0, nk, 2 * nk, 2 * nk + nv)
            w = (rnd(4, sh.channels), torch.rand(H, device=DEV) + 0.5, rnd(nk) * 0.5 - 4, rnd(dv))
            sets = [(R(T, 2 * nk + nv + H), R(T, nk + nv), rnd(nseq + 1, H, d, cols),
                     rnd(nseq + 1, 2, 3, sh.channels).to(bf16)) for _ in range(nc)]
            fn = lambda i=0: states.delta_scan(sets[i][0], sets[i][1], sets[i][1][:, nk:], *w, sh,
                                               *sets[i][2:], step, 1e-6)
        else:
            sh = states.MemoryShape(H, d, dv, 15.0, 0, nk, 2 * nk, 2 * nk + nv, 2 * nk + nv + H)
            w = (rnd(H), rnd(H) + 4, rnd(nv))
            sets = [(R(T, 2 * nk + nv + 2 * H), R(T, nv), rnd(nseq + 1, H, d, cols), rnd(nseq + 1, 2, H))
                    for _ in range(nc)]
            fn = lambda i=0: states.memory_scan(*sets[i][:2], *w, sh, *sets[i][2:], step, 1e-6)
    elif kind == "forget":
        import numpy as np
        from arcticinference_b200.ops import state_ops as states
        H, nseq, n = prm
        T, d = nseq * n, 128
        step = states.StateStep.build(np.asarray([(i * n, n, i + 1, 0 if n > 1 else 5, 0)
                                                  for i in range(nseq)], dtype=np.int32), DEV)
        byts = 2.0 * T * H * 4 * d + 4.0 * nseq * H * d * d * (1 if n > 1 else 2)
        flops = 4.0 * T * H * d * d
        nc = copies_for(byts)
        sh = states.ForgetShape(H, d, d, 0, H * d, 2 * H * d)
        w = (torch.rand(H * d, device=DEV) * 4, torch.rand(H * d, device=DEV) * 0.9, torch.ones(d, device=DEV))
        sets = [(R(T, 3 * H * d), torch.randn(nseq + 1, H, d, d, device=DEV)) for _ in range(nc)]
        fn = lambda i=0: states.forget_scan(sets[i][0], *w, sh, sets[i][1], step, 1e-6)
    elif kind == "poly":
        from arcticinference_b200.ops import stream_ops as st
        T, ff = prm
        nc = copies_for(4 * T * ff)
        zs, bias, coef = [R(T, ff) for _ in range(nc)], R(ff), torch.ones(4, device=DEV)
        fn = lambda i=0: st.poly_norm(zs[i], bias, coef, ff, 1e-6)
        flops, byts = 0.0, 4.0 * T * ff
    elif kind == "soft_cap":
        from arcticinference_b200.ops import stream_ops as st
        T, V = prm
        nc = copies_for(6 * T * V)
        zs = [R(T, V) for _ in range(nc)]
        fn = lambda i=0: st.soft_cap(zs[i], 30.0)
        flops, byts = 0.0, 6.0 * T * V
    elif kind == "pre":
        from arcticinference_b200.ops import stream_ops as st
        T, W = prm
        nc = copies_for(8 * T * W)
        sets = [(torch.randn(T, W, device=DEV), R(T, W), R(T, W)) for _ in range(nc)]
        w = torch.ones(1, device=DEV)
        fn = lambda i=0: st.stream_pre(sets[i][0], 0.5, 1e-6, y=sets[i][1], w_in=w, act=sets[i][2])
        flops, byts = 0.0, 12.0 * T * W
    elif kind == "sandwich":
        from arcticinference_b200.ops import stream_ops as st
        T, W = prm
        nc = copies_for(8 * T * W)
        sets = [(torch.randn(T, W, device=DEV), R(T, W), R(T, W)) for _ in range(nc)]
        w = torch.ones(W, device=DEV)
        fn = lambda i=0: st.stream_sandwich(sets[i][0], sets[i][1], w, None, w, sets[i][2], eps=1e-6)
        flops, byts = 0.0, 12.0 * T * W
    elif kind == "experts":
        from arcticinference_b200.ops import stream_ops as st
        T, W, ff, E, top = prm
        x = torch.randn(T, W, device=DEV)
        r, rows = st.route(x, x.to(torch.bfloat16), R(E, W), torch.zeros(E, device=DEV), top)
        nc = copies_for(4 * E * W * ff)
        ws = [R(E, 2 * ff, W) for _ in range(nc)]
        fn = lambda i=0: st.grouped_linear(rows, ws[i], r, act="silu")
        flops = 4.0 * T * top * W * ff
        byts = 4.0 * E * W * ff + 2.0 * T * top * (W + ff)
    elif kind == "route":
        from arcticinference_b200.ops import stream_ops as st
        T, W, E, top = prm
        nc = copies_for(6 * T * W)
        sets = [(torch.randn(T, W, device=DEV), R(T, W)) for _ in range(nc)]
        w, b = R(E, W), torch.zeros(E, device=DEV)
        fn = lambda i=0: st.route(sets[i][0], sets[i][1], w, b, top)
        flops, byts = 2.0 * T * W * E, T * W * (6.0 + 2.0 * top)
    elif kind == "latent_norm":
        from arcticinference_b200.ops import latent_ops as lat
        T, rank = prm
        nc = copies_for(4 * T * rank)
        sets = [(R(T, rank), R(T // 64, 1, 64, rank)) for _ in range(nc)]
        w, slots = torch.ones(rank, device=DEV), torch.arange(T, device=DEV)
        fn = lambda i=0: lat.latent_norm_cache(sets[i][0], w, rank, 1e-6, slots, sets[i][1])
        flops, byts = 0.0, 4.0 * T * rank
    elif kind == "stream_norm":
        from arcticinference_b200.ops import stream_ops as st
        T, W = prm
        nc = copies_for(8 * T * W)
        sets = [(torch.randn(T, W, device=DEV), R(T, W), R(T, W)) for _ in range(nc)]
        w = torch.zeros(W, device=DEV)
        fn = lambda i=0: st.stream_norm(sets[i][0], sets[i][1], sets[i][2], w, 1.5, 1e-6)
        flops, byts = 0.0, 12.0 * T * W
    elif kind == "rmsnorm":
        T, H = prm
        nc = copies_for(4 * T * H)
        xs, w, rs = [R(T, H) for _ in range(nc)], R(H), [R(T, H) for _ in range(nc)]
        fn = lambda i=0: ops.rmsnorm(xs[i], w, 1e-5, residual=rs[i])
        flops, byts = 0.0, 4.0 * T * H * 2
    elif kind == "rmsnorm_q":
        T, H = prm
        nc = copies_for(4 * T * H)
        xs, w, rs = [R(T, H) for _ in range(nc)], R(H), [R(T, H) for _ in range(nc)]
        fn = lambda i=0: ops.rmsnorm(xs[i], w, 1e-5, residual=rs[i], quant=True)
        flops, byts = 0.0, 3.0 * T * H * 2 + T * H
    elif kind == "quant_row":
        T, H = prm
        nc = copies_for(2 * T * H)
        xs = [R(T, H) for _ in range(nc)]
        fn = lambda i=0: ops.quant_fp8_row(xs[i])
        flops, byts = 0.0, 3.0 * T * H
    elif kind == "silu_q":
        T, I = prm
        nc = copies_for(4 * T * I)
        gs = [R(T, 2 * I) for _ in range(nc)]
        fn = lambda i=0: ops.silu_mul_blocked(gs[i], 1, quant=True)
        flops, byts = 0.0, 2.0 * T * I * 2 + T * I
    else:
        T, I = prm
        nc = copies_for(4 * T * I)
        gs = [R(T, 2 * I) for _ in range(nc)]
        fn = lambda i=0: ops.silu_mul(gs[i])
        flops, byts = 0.0, 3.0 * T * I * 2
    if a.no_time:
        for i in range(3):
            fn(i % nc)
        torch.cuda.synchronize()
        ops.check_status()
        print("ran", case)
        return
    ms = timeit(fn, a.iters, copies=nc)
    ops.check_status()
    t = ms / 1e3
    print(json.dumps({"case": case, "splits": a.splits, "us": ms * 1e3, "tflops": flops / t / 1e12,
                      "gbs": byts / t / 1e9, "frac_of_%s_bf16" % src: flops / t / 1e12 / tf,
                      "frac_of_%s_hbm" % src: byts / t / 1e9 / hbm}))


if __name__ == "__main__":
    main()
