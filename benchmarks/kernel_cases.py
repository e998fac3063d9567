#!/usr/bin/env python
"""One hot kernel at a time, on one GPU, at a size that is larger than L2 but small enough to profile.

    python benchmarks/kernel_cases.py --case gemm            # one case
    python benchmarks/kernel_cases.py --case all             # every case, one JSON line each
    ncu --set full --clock-control none -k regex:gemm_bf16_kernel -s 3 -c 1 -o prof \
        python benchmarks/kernel_cases.py --case gemm --iters 1

Every case warms up, then times ``--iters`` launches with CUDA events (an L2 flush between launches) and prints
the achieved rate next to the measured peak it is bounded by (copy bandwidth / cuBLAS bf16 rate of this machine,
given with --hbm-gbs / --bf16-tflops or a JSON file named by --peaks-file / $TESSERACT_PEAKS_FILE). The fused tensor-parallel kernels run here as
an emulation of two ranks on one GPU: all buffers local, the gather kernel split into its push half and its
multiply half so that no launch waits for a later one.
Shapes follow the reference's microbenchmarks where it has one (benchmarks/bench_cuda_matmul.cpp,
bench_cuda_fused_attention.cpp, bench_cuda_moe.cpp, bench_cuda_mamba_scaling.cpp, bench_cuda_fp8_gemm.cpp).
"""
from __future__ import annotations

import argparse
import ctypes
import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

import torch  # noqa: E402


_PEAKS = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "src": "default"}


def set_peaks(hbm_gbs=None, bf16_tflops=None, peaks_file=None):
    """The denominators of the reported fractions: --hbm-gbs / --bf16-tflops, or a JSON file with the keys
    ``hbm_gbs`` and ``bf16_tflops`` (--peaks-file or $TESSERACT_PEAKS_FILE), else 6650 GB/s and 1590 TFLOP/s."""
    path = peaks_file or os.environ.get("TESSERACT_PEAKS_FILE", "")
    if path:
        d = json.load(open(path))
        _PEAKS.update(hbm_gbs=float(d["hbm_gbs"]), bf16_tflops=float(d["bf16_tflops"]), src="measured")
    if hbm_gbs:
        _PEAKS.update(hbm_gbs=float(hbm_gbs), src="given")
    if bf16_tflops:
        _PEAKS.update(bf16_tflops=float(bf16_tflops), src="given")


def peaks():
    return _PEAKS["hbm_gbs"], _PEAKS["bf16_tflops"], _PEAKS["src"]


class Bench:
    def __init__(self, iters: int):
        self.dev = torch.device("cuda", 0)
        self.iters = iters
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=self.dev)
        self.gen = torch.Generator(device=self.dev).manual_seed(0)

    def randn(self, *shape, scale=1.0):
        return (torch.randn(*shape, device=self.dev, generator=self.gen) * scale).bfloat16()

    def time(self, fn, warmup=2):
        for _ in range(warmup):
            fn()
        torch.cuda.synchronize()
        total = 0.0
        for _ in range(self.iters):
            self.flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            total += e0.elapsed_time(e1)
        return total / self.iters


def report(name, ms, flops=None, bytes_=None, **extra):
    hbm, tf, src = peaks()
    out = {"case": name, "ms": round(ms, 4)}
    if flops:
        out["tflops"] = round(flops / ms / 1e9, 1)
        out["frac_of_bf16_peak"] = round(flops / ms / 1e9 / tf, 3)
    if bytes_:
        out["gbs"] = round(bytes_ / ms / 1e6, 1)
        out["frac_of_hbm_peak"] = round(bytes_ / ms / 1e6 / hbm, 3)
    out["peaks"] = src
    out.update(extra)
    print(json.dumps(out), flush=True)


# ------------------------------------------------------------------------------------------------- cases
def case_gemm(b: Bench):
    from tesseract_b200.ops import gemm_bf16
    M = N = K = 8192
    a, w = b.randn(M, K), b.randn(N, K, scale=0.02)
    out = torch.empty(M, N, device=b.dev, dtype=torch.bfloat16)
    ms = b.time(lambda: gemm_bf16(a, w, out=out))
    report("gemm", ms, flops=2.0 * M * N * K, shape=[M, N, K])


def case_gemm_wgrad(b: Bench):
    from tesseract_b200.ops import gemm_bf16
    T, N, K = 16384, 4096, 4096
    dy, x = b.randn(T, N), b.randn(T, K)
    dw = torch.zeros(N, K, device=b.dev, dtype=torch.float32)
    ms = b.time(lambda: gemm_bf16(dy, x, a_mn=True, b_mn=True, out=dw, accumulate=True))
    report("gemm_wgrad", ms, flops=2.0 * T * N * K, shape=[N, K, T])


def case_gemm_fp8(b: Bench):
    from tesseract_b200.ops import fp8
    M = N = K = 8192
    qa, sa = fp8.quantize_act(b.randn(M, K))
    qb, sb = fp8.quantize_weight(b.randn(N, K, scale=0.02))
    ms = b.time(lambda: fp8.fp8_gemm(qa, sa, qb, sb))
    report("gemm_fp8", ms, flops=2.0 * M * N * K, shape=[M, N, K], note="fractions are of the bf16 peak")


def case_gemm_fp8_pertensor(b: Bench):
    """The reference's FP8 benchmark shape family (square, one scale per operand); its bar is FP8 >= 1.3 x FP16
    (benchmarks/bench_cuda_fp8_gemm.cpp:156-159): the 16-bit product of the same shape is timed next to it."""
    from tesseract_b200.ops import fp8, gemm_bf16
    for n in (4096, 8192):
        x, w = b.randn(n, n), b.randn(n, n, scale=0.02)
        qa, sa = fp8.quantize_tensor(x)
        qb, sb = fp8.quantize_tensor(w)
        ms8 = b.time(lambda: fp8.fp8_gemm_pertensor(qa, sa, qb, sb))
        out = torch.empty(n, n, device=b.dev, dtype=torch.bfloat16)
        ms16 = b.time(lambda: gemm_bf16(x, w, out=out))
        report(f"gemm_fp8_pertensor_{n}", ms8, flops=2.0 * n ** 3, shape=[n, n, n], bf16_ms=round(ms16, 4),
               fp8_over_bf16=round(ms16 / ms8, 3), note="fractions are of the bf16 peak")


def case_decode_gemm(b: Bench):
    """Weight-streaming GEMMs of one decode step (Llama-8B layer shapes) at 64 and 256 rows."""
    from tesseract_b200 import ops
    for M in (64, 256):
        tot_ms, tot_bytes = 0.0, 0
        for name, N, K in (("qkv", 6144, 4096), ("o_proj", 4096, 4096), ("gate_up", 28672, 4096), ("down", 4096, 14336)):
            x, w = b.randn(M, K), b.randn(N, K, scale=0.02)
            ms = b.time(lambda: ops.decode_linear(x, w))
            tot_ms += ms
            tot_bytes += N * K * 2
            report(f"decode_gemm_{name}_M{M}", ms, bytes_=N * K * 2, shape=[M, N, K])
        report(f"decode_gemm_layer_M{M}", tot_ms, bytes_=tot_bytes)


def case_stream_linear(b: Bench):
    """The weight-streaming decode GEMM (bf16 and block-scaled fp8 weights) on the layer shapes of one decode step,
    next to the cluster split-K kernel it replaces; bytes = the weight matrix once."""
    from tesseract_b200 import ops
    from tesseract_b200.ops import fp8
    for M in (16, 64, 141, 256):
        tot = {"bf16": [0.0, 0], "fp8": [0.0, 0], "old": [0.0, 0]}
        for name, N, K in (("qkv", 6144, 4096), ("o_proj", 4096, 4096), ("gate_up", 28672, 4096), ("down", 4096, 14336)):
            x, w = b.randn(M, K), b.randn(N, K, scale=0.02)
            q, sc = fp8.quantize_weight(w)
            ms_old = b.time(lambda: ops.decode_linear(x, w))
            ms_bf = b.time(lambda: ops.stream_linear(x, w))
            ms_f8 = b.time(lambda: ops.stream_linear(x, q, sc))
            for key, ms, nbytes in (("old", ms_old, N * K * 2), ("bf16", ms_bf, N * K * 2), ("fp8", ms_f8, N * K)):
                tot[key][0] += ms
                tot[key][1] += nbytes
            report(f"stream_linear_bf16_{name}_M{M}", ms_bf, bytes_=N * K * 2, shape=[M, N, K], cluster_splitk_ms=round(ms_old, 4))
            report(f"stream_linear_fp8_{name}_M{M}", ms_f8, bytes_=N * K, shape=[M, N, K])
        for key in ("old", "bf16", "fp8"):
            report(f"stream_linear_layer_{key}_M{M}", tot[key][0], bytes_=tot[key][1])


def case_gemm_mx(b: Bench):
    """Block-scaled fp8 GEMM on the tensor core's own block scaling (E4M3 x E4M3, power-of-two scales, persistent
    128 x 192 tiles), next to the bf16 GEMM of the same shape; the activation quantiser is timed separately."""
    import os

    from tesseract_b200.ops import fp8, gemm_bf16
    shapes = ((8192, 8192, 8192), (16384, 4096, 4096), (16384, 28672, 4096), (16384, 4096, 14336))
    if os.environ.get("TESSERACT_KERNEL_CASES_SMALL", "0") == "1":
        shapes = shapes[:1]                                   # one shape for a profiler capture
    for M, N, K in shapes:
        a, w = b.randn(M, K), b.randn(N, K, scale=0.02)
        wq, ws = fp8.quantize_weight(w, pow2=True)
        q, sf = fp8.quantize_act_mx(a, atoms=True)
        wa = fp8.weight_scale_atoms(ws)
        out = torch.empty(M, N, device=b.dev, dtype=torch.bfloat16)
        ms = b.time(lambda: fp8.mx_linear(q, sf, wq, ws, out=out, w_atoms=wa))
        ms_bf = b.time(lambda: gemm_bf16(a, w, out=out))
        ms_q = b.time(lambda: fp8.quantize_act_mx(a, out=(q, sf), atoms=True))
        report(f"gemm_mx_{M}x{N}x{K}", ms, flops=2.0 * M * N * K, shape=[M, N, K], bf16_gemm_ms=round(ms_bf, 4),
               speedup_over_bf16=round(ms_bf / ms, 3), quantiser_ms=round(ms_q, 4))


def case_mx_linear(b: Bench):
    """The block-scaled fp8 decode GEMM on tcgen05.mma kind::mxf8f6f4 (E4M3 activations and weights, power-of-two
    scales applied by the tensor core) on the layer shapes of one decode step; bytes = the fp8 weight matrix once.
    ``with_quant`` adds the stand-alone activation quantiser in front (the serving engine fuses it into RMSNorm /
    SwiGLU instead); ``TESSERACT_KERNEL_CASES_SMALL=1`` runs one shape only (a profiler capture)."""
    import os

    from tesseract_b200.ops import fp8
    small = os.environ.get("TESSERACT_KERNEL_CASES_SMALL", "0") == "1"
    shapes = (("qkv", 6144, 4096), ("o_proj", 4096, 4096), ("gate_up", 28672, 4096), ("down", 4096, 14336))
    for M in ((32,) if small else (16, 32, 64, 128, 256)):
        tot = [0.0, 0.0, 0]
        for name, N, K in (shapes[2:3] if small else shapes):
            x, w = b.randn(M, K), b.randn(N, K, scale=0.02)
            wq, ws = fp8.quantize_weight(w, pow2=True)
            q, sf = fp8.quantize_act_mx(x)
            ms = b.time(lambda: fp8.mx_linear(q, sf, wq, ws))
            # (not in the small profiler case: it launches with the programmatic-serialisation attribute)
            ms_q = ms if small else b.time(lambda: fp8.mx_linear(*fp8.quantize_act_mx(x, out=(q, sf)), wq, ws, pdl=True))
            tot[0] += ms
            tot[1] += ms_q
            tot[2] += N * K
            bn, split, stages, _ = fp8.mx_linear_plan(M, N, K)
            report(f"mx_linear_{name}_M{M}", ms, bytes_=N * K, shape=[M, N, K], with_quant_ms=round(ms_q, 4),
                   tile=bn, k_split=split, stages=stages)
        report(f"mx_linear_layer_M{M}", tot[0], bytes_=tot[2], with_quant_ms=round(tot[1], 4))


def case_grouped_gemm(b: Bench):
    from tesseract_b200.ops import moe
    E, N, K, per = 8, 4096, 4096, 2048
    offsets = torch.arange(E + 1, device=b.dev, dtype=torch.int32) * per
    a, w = b.randn(E * per, K), b.randn(E, N, K, scale=0.02)
    ms = b.time(lambda: moe.grouped_gemm_rows(a, w[0], N * K, offsets, E))
    report("grouped_gemm", ms, flops=2.0 * E * per * N * K, shape=[E, per, N, K])


def _qkv(b: Bench, B, S, H, Hkv, D):
    return b.randn(B, S, H + 2 * Hkv, D)


def case_flash_fwd(b: Bench):
    from tesseract_b200.ops import flash_attention_packed
    B, S, H, Hkv, D = 2, 4096, 32, 8, 128
    qkv = _qkv(b, B, S, H, Hkv, D)
    with torch.no_grad():
        ms = b.time(lambda: flash_attention_packed(qkv, H, Hkv, causal=True))
    report("flash_fwd", ms, flops=4.0 * B * H * S * S * D / 2, shape=[B, S, H, Hkv, D])


def case_flash_bwd(b: Bench):
    from tesseract_b200.ops import flash_attention_packed
    B, S, H, Hkv, D = 2, 4096, 32, 8, 128
    qkv = _qkv(b, B, S, H, Hkv, D).requires_grad_(True)
    o = flash_attention_packed(qkv, H, Hkv, causal=True)
    do = torch.randn_like(o)

    def run():
        qkv.grad = None
        o.backward(do, retain_graph=True)
    ms = b.time(run)
    report("flash_bwd", ms, flops=10.0 * B * H * S * S * D / 2, shape=[B, S, H, Hkv, D])


def _paged(b: Bench, A, L, int8):
    H, Hkv, D, bs = 32, 8, 128, 16
    mb = (L + bs - 1) // bs
    nb = A * mb + 1
    if int8:
        k = torch.randint(-127, 127, (nb, Hkv, bs, D), device=b.dev, dtype=torch.int8)
        v = torch.randint(-127, 127, (nb, Hkv, bs, D), device=b.dev, dtype=torch.int8)
        ks, vs = torch.rand(nb, Hkv, bs, device=b.dev), torch.rand(nb, Hkv, bs, device=b.dev)
    else:
        k, v, ks, vs = b.randn(nb, Hkv, bs, D), b.randn(nb, Hkv, bs, D), None, None
    tables = torch.randperm(nb - 1, device=b.dev)[:A * mb].view(A, mb).int()
    lens = torch.full((A,), L, device=b.dev, dtype=torch.int32)
    q = b.randn(A, H, D)
    return q, k, v, tables, lens, ks, vs, A * L * Hkv * D * 2 * (1 if int8 else 2)


def case_decode(b: Bench):
    from tesseract_b200 import ops
    q, k, v, tables, lens, ks, vs, nbytes = _paged(b, 256, 1400, False)
    ms = b.time(lambda: ops.paged_decode_attention(q, k, v, tables, lens, None, ks, vs, max_len_hint=2560))
    report("decode", ms, bytes_=nbytes, shape=[256, 1400])


def case_decode_int8(b: Bench):
    from tesseract_b200 import ops
    q, k, v, tables, lens, ks, vs, nbytes = _paged(b, 256, 1400, True)
    ms = b.time(lambda: ops.paged_decode_attention(q, k, v, tables, lens, None, ks, vs, max_len_hint=2560))
    report("decode_int8", ms, bytes_=nbytes, shape=[256, 1400])


def case_rmsnorm(b: Bench):
    from tesseract_b200 import ops
    x, w = b.randn(32768, 4096), torch.ones(4096, device=b.dev, dtype=torch.bfloat16)
    with torch.no_grad():
        ms = b.time(lambda: ops.rms_norm(x, w, 1e-5))
    report("rmsnorm", ms, bytes_=2 * x.numel() * 2, shape=list(x.shape))


def case_swiglu(b: Bench):
    from tesseract_b200 import ops
    x = b.randn(16384, 2 * 14336)
    with torch.no_grad():
        ms = b.time(lambda: ops.swiglu(x))
    report("swiglu", ms, bytes_=x.numel() * 2 * 1.5, shape=list(x.shape))


def case_swiglu_bwd(b: Bench):
    from tesseract_b200.ops import fused
    x = b.randn(16384, 2 * 14336)
    d = b.randn(16384, 14336)
    ms = b.time(lambda: fused.swiglu_backward(x, d))
    report("swiglu_bwd", ms, bytes_=d.numel() * 2 * 5, shape=list(x.shape))


def case_adam(b: Bench):
    from tesseract_b200 import _native
    from tesseract_b200.optim import optimizers  # noqa: F401  (registers the signatures of loss_optim.cu)
    n = 256 << 20
    p = torch.zeros(n, device=b.dev, dtype=torch.bfloat16)
    g = torch.zeros(n, device=b.dev, dtype=torch.bfloat16)
    m = torch.zeros(n, device=b.dev, dtype=torch.float32)
    v = torch.zeros(n, device=b.dev, dtype=torch.float32)
    s = torch.cuda.current_stream().cuda_stream
    lib = _native.lib()
    ms = b.time(lambda: _native.check(lib.tsb_adam_flat(p.data_ptr(), g.data_ptr(), m.data_ptr(), v.data_ptr(), None, n,
                                                        1e-4, 0.9, 0.999, 1e-8, 0.1, 0.001, 0.0, None, 1, 1, s),
                                      "tsb_adam_flat"))
    report("adam", ms, bytes_=n * (2 + 2 + 4 + 4 + 2 + 4 + 4), shape=[n])


def case_ce(b: Bench):
    from tesseract_b200 import ops
    T, V = 4096, 128256
    logits = b.randn(T, V)
    tgt = torch.randint(0, V, (T,), device=b.dev)
    ms = b.time(lambda: ops.ce_stats(logits, tgt))
    report("ce_stats", ms, bytes_=T * V * 2, shape=[T, V])


def case_scan(b: Bench):
    from tesseract_b200.ops import ssm
    B, L, D, N = 4, 4096, 4096, 16
    u = torch.randn(B, L, D, device=b.dev, generator=b.gen)
    delta = torch.rand(B, L, D, device=b.dev, generator=b.gen) * 0.1
    A = -torch.rand(D, N, device=b.dev, generator=b.gen)
    Bm = torch.randn(B, L, N, device=b.dev, generator=b.gen)
    C = torch.randn(B, L, N, device=b.dev, generator=b.gen)
    Dv = torch.ones(D, device=b.dev)
    with torch.no_grad():
        ms = b.time(lambda: ssm.selective_scan(u, delta, A, Bm, C, Dv))
    report("selective_scan", ms, bytes_=3 * B * L * D * 4, shape=[B, L, D, N])


def case_gemv(b: Bench):
    from tesseract_b200 import quant
    N, K = 14336, 4096
    w = torch.randn(N, K, device=b.dev, generator=b.gen)
    q8, s8 = (t.to(b.dev) for t in quant.pack_int8_symmetric(w))     # the packer works on the host
    x = b.randn(1, K)
    ms = b.time(lambda: quant.dequantize_matmul_int8(x, q8, s8))
    report("gemv_w8", ms, bytes_=N * K, shape=[1, N, K])


def _ptrs(ts):
    return (ctypes.c_void_p * len(ts))(*[t.data_ptr() for t in ts])


def case_gemm_rs_emul(b: Bench):
    from tesseract_b200 import _native
    from tesseract_b200.parallel import fused_tp  # noqa: F401
    lib = _native.lib()
    world, rpr, N, K = 2, 4096, 4096, 2048
    M = world * rpr
    x, w = b.randn(M, K), b.randn(N, K, scale=0.02)
    staging = [torch.empty(world, rpr, N, device=b.dev, dtype=torch.bfloat16) for _ in range(world)]
    pa = _ptrs(staging)
    s = torch.cuda.current_stream().cuda_stream
    ms = b.time(lambda: _native.check(lib.tsb_gemm_rs(x.data_ptr(), w.data_ptr(), pa, M, N, K, x.stride(0), w.stride(0),
                                                      0, rpr, 0, world, s), "tsb_gemm_rs"))
    report("gemm_rs_emul", ms, flops=2.0 * M * N * K, shape=[M, N, K], note="rank 0 of 2, peers on the same GPU")


def case_ag_gemm_emul(b: Bench):
    from tesseract_b200 import _native
    from tesseract_b200.parallel import fused_tp  # noqa: F401
    lib = _native.lib()
    world, rpr, N, K = 2, 4096, 3072, 4096
    M = world * rpr
    shards = [b.randn(rpr, K) for _ in range(world)]
    w = b.randn(N, K, scale=0.02)
    lands = [torch.empty(M, K, device=b.dev, dtype=torch.bfloat16) for _ in range(world)]
    flags = [torch.zeros(world, dtype=torch.int32, device=b.dev) for _ in range(world)]
    y = torch.empty(M, N, device=b.dev, dtype=torch.bfloat16)
    pl, pf = _ptrs(lands), _ptrs(flags)
    s = torch.cuda.current_stream().cuda_stream
    calls = [0]

    def call(rank, mask):
        _native.check(lib.tsb_gemm_ag(shards[rank].data_ptr(), pl, pf, None, w.data_ptr(), y.data_ptr(), calls[0], 1,
                                      mask, M, N, K, w.stride(0), y.stride(0), 0, rpr, rank, world, None, s),
                      "tsb_gemm_ag")

    def push_all():
        calls[0] += 1
        for r in range(world):
            call(r, 1)
    push_all()
    ms_mult = b.time(lambda: call(0, 2))
    ms_push = b.time(push_all) / world
    report("ag_gemm_emul", ms_mult, flops=2.0 * M * N * K, shape=[M, N, K], push_ms=round(ms_push, 4),
           note="multiply half of rank 0 of 2 after both ranks' push halves; push_ms = one rank's push half alone")


# ---- hybrid decoders: 4096-wide layers, 16 key / 32 value heads of 128 x 128 (delta), 32 / 8 heads of 128 (attention)
class _Step:
    """A ragged batch of ``n`` sequences bringing ``rows`` tokens each, after ``past`` tokens."""

    def __init__(self, b, run, n, rows, past=0, chunks=(), block=16, tiles=()):
        from tesseract_b200.nn.ragged import HybridCache, HybridSequence, RaggedBatch
        blocks = n * ((past + rows + block - 1) // block)
        self.cache = HybridCache([run], blocks, block, n, past + rows + block, torch.bfloat16, b.dev)
        seqs = [HybridSequence(self.cache) for _ in range(n)]
        for s in seqs:
            if past:
                s.reserve(past)
                s.advance(past)
        self.batch = RaggedBatch(self.cache, [(s, [0] * rows) for s in seqs], None, chunks, 0, tiles)


def _delta_case(b, n, rows, past):
    from tesseract_b200.nn.ragged import StateRun
    from tesseract_b200.ops.delta import DeltaGeometry, DeltaWeights, gated_delta
    g = DeltaGeometry(16, 32, 128, 128, 4)
    st = _Step(b, StateRun((g.heads, g.dim, g.vdim_pad), (g.taps - 1, g.conv_cols)), n, rows, past)
    proj = b.randn(n * rows, g.cols)
    f = lambda *sh: torch.randn(*sh, device=b.dev, generator=b.gen)   # noqa: E731
    w = DeltaWeights(f(g.taps, g.conv_cols), f(g.heads), f(g.heads), f(g.vdim), 1e-5)
    ms = b.time(lambda: gated_delta(proj, g, w, *st.cache.runs[0], st.batch))
    return g, ms


def case_delta_prefill(b: Bench):
    """All four launches; bound by the fp32 multiply-adds of the recurrence (8 flops per state element and token)."""
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        g, ms = _delta_case(b, n, rows, 0)
        fl = 8.0 * g.heads * g.dim * g.vdim * n * rows
        peak = 148 * 128 * 2 * 1.965e9 / 1e12
        print(json.dumps({"case": "delta_prefill", "ms": round(ms, 4), "fp32_tflops": round(fl / ms / 1e9, 2),
                          "frac_of_nominal_fp32": round(fl / ms / 1e9 / peak, 3), "ns_per_token": round(ms * 1e6 / (n * rows), 1),
                          "shape": [n, rows]}))


def case_delta_step(b: Bench):
    for n in (256, 32):
        g, ms = _delta_case(b, n, 1, 7)
        report("delta_step", ms, bytes_=n * (2.0 * g.heads * g.dim * g.vdim * 4 + 2 * (2 * g.taps - 1) * g.conv_cols), shape=[n])


def _chunk_attn(b, n, rows, past, chunk):
    from tesseract_b200 import ops
    from tesseract_b200.nn.ragged import PagedRun
    H, G, D = 32, 8, 128
    st = _Step(b, PagedRun(G, D), n, rows, past, (chunk,))
    qkv, bias = b.randn(n * rows, (H + 2 * G) * D), torch.zeros((H + 2 * G) * D, device=b.dev)
    return b.time(lambda: ops.ragged_attention(qkv, bias, *st.cache.runs[0], st.batch, H, G, D ** -0.5, chunk))


def case_chunk_attn(b: Bench):
    """Append + attention. Prompts: two sequences of 4096 in chunks of 4096 (the flash_fwd case) and of 1024; decode: 256
    sequences at 1400 tokens of one chunk (the decode case)."""
    from tesseract_b200 import ops
    for chunk in (4096, 1024):
        ms = _chunk_attn(b, 2, 4096, 0, chunk)
        report("chunk_attn_prefill", ms, flops=2 * 4096 * chunk * 32 * 128 * 2.0, shape=[2, 4096, chunk])
        n = 2 * 4096 // chunk                       # the plain kernel over as many sequences of the chunk's length
        qkv = b.randn(n, chunk, 48, 128)
        with torch.no_grad():
            ms = b.time(lambda: ops.flash_attention_packed(qkv, 32, 8))
        report("flash_fwd_same_lengths", ms, flops=2 * 4096 * chunk * 32 * 128 * 2.0, shape=[n, chunk])
    ms = _chunk_attn(b, 256, 1, 1399, 4096)
    report("chunk_attn_decode", ms, bytes_=256 * 1400 * 8 * 128 * 2 * 2, shape=[256, 1400])


def case_dyn_tanh(b: Bench):
    from tesseract_b200 import ops
    T, W = 16384, 4096
    x, y = torch.randn(T, W, device=b.dev, generator=b.gen), b.randn(T, W)
    v = lambda: torch.randn(W, device=b.dev, generator=b.gen)   # noqa: E731
    post, nxt = (0.5, v(), v()), (0.5, v() * 0.01, v() * 0.01)
    ms = b.time(lambda: ops.dyn_tanh_residual(x, y, None, post, next_norm=nxt))
    report("dyn_tanh_residual", ms, bytes_=T * W * 12, shape=[T, W])


def case_clamped_glu(b: Bench):
    from tesseract_b200 import ops
    x, bias = b.randn(16384, 2 * 14336), torch.zeros(2 * 14336, device=b.dev)
    ms = b.time(lambda: ops.clamped_glu(x, bias, 7.0))
    report("clamped_glu", ms, bytes_=x.numel() * 2 * 1.5, shape=list(x.shape))


# ---- the mixers of 4096-wide layers with 32 heads: retention 128 x 128, latent 64 + 64 / 128 / 512, recurrence 4096 in blocks of 256
def _mixer_case(b, block, n, rows, past=0):
    """Time of a mixer's core (everything between its two products)."""
    st = _Step(b, block.run_spec(), n, rows, past, block.masks or (0,), tiles=block.tiles)
    proj = b.randn(n * rows, block.cols)
    return b.time(lambda: block.core(proj, st.cache.runs[0], st.batch))


def case_retention(b: Bench):
    """Prompts: bytes of q, k, v, gate and the result; decode: the state read and written once."""
    from tesseract_b200.nn.hybrid import Retention
    from tesseract_b200.ops.rotary import Rotary
    H = 32
    blk = Retention(64, H, 128, 128, [1.0 - 2.0 ** (-5 - 7 * i / H) for i in range(H)], Rotary(128, 1e4), 1e-6, torch.bfloat16, b.dev)
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        ms = _mixer_case(b, blk, n, rows)
        report("retention_prefill", ms, bytes_=n * rows * H * 128 * 5 * 2.0, shape=[n, rows])
    for n in (256, 32):
        report("retention_step", _mixer_case(b, blk, n, 1, 7), bytes_=n * 2.0 * H * 128 * 128 * 4, shape=[n])


def case_latent(b: Bench):
    """Prompts: flops of the written-out form (expansion of the latents and causal attention); decode: bytes of the cached rows."""
    from tesseract_b200.nn.hybrid import LatentAttention
    from tesseract_b200.ops.rotary import Rotary
    H = 32
    blk = LatentAttention(64, H, 64, 64, 128, 512, 128 ** -0.5, Rotary(64, 1e6), 1e-6, torch.bfloat16, b.dev)
    for n, rows in ((2, 4096), (8, 1024)):
        ms = _mixer_case(b, blk, n, rows)
        report("latent_prefill", ms, flops=n * rows * (rows * H * 128 * 2.0 + 2.0 * 512 * H * 192), shape=[n, rows])
    for n, past in ((256, 1399), (32, 1399), (32, 8191)):
        ms = _mixer_case(b, blk, n, 1, past)
        report("latent_decode", ms, bytes_=n * (past + 1) * 576 * 2.0, flops=n * (past + 1.0) * H * 2 * (576 + 512), shape=[n, past + 1])


def case_rglru(b: Bench):
    """Prompts: bytes of x, y and the result; decode: the gate matrices, x, y, the states and the result."""
    from tesseract_b200.nn.hybrid import RGLRU
    W = 4096
    blk = RGLRU(64, W, W // 256, 4, torch.bfloat16, b.dev)
    blk.w.ra.normal_(std=0.06)
    blk.w.ri.normal_(std=0.06)
    blk.w.decay.fill_(0.2)
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        report("rglru_prefill", _mixer_case(b, blk, n, rows), bytes_=n * rows * W * 3 * 2.0, shape=[n, rows])
    for n in (256, 32):
        report("rglru_step", _mixer_case(b, blk, n, 1, 7), bytes_=2.0 * 256 * W * 2 + n * W * (2 * 4 + 5 * 2 + 3 * 2.0), shape=[n])


def case_depth_residual(b: Bench):
    from tesseract_b200 import ops
    T, W = 16384, 4096
    hist = torch.randn(5, T, W, device=b.dev, generator=b.gen)
    x, y, avg = torch.randn(T, W, device=b.dev, generator=b.gen), b.randn(T, W), torch.randn(5, device=b.dev, generator=b.gen)
    for depth in (1, 4):
        a = avg[:depth + 1].contiguous()
        ms = b.time(lambda: ops.depth_residual(x, y, 0.5, history=hist, depth=depth, average=a, eps=1e-6))
        report("depth_residual", ms, bytes_=T * W * (4 * (depth + 3) + 4), shape=[T, W, depth])


def case_silu_glu(b: Bench):
    from tesseract_b200 import ops
    x = b.randn(16384, 2 * 14336)
    report("silu_glu", b.time(lambda: ops.silu_glu(x, 0.9)), bytes_=x.numel() * 2 * 1.5, shape=list(x.shape))


# ---- the mixers of 4096-wide post-normed layers: 32 / 8 heads of 128 (attention), 64 heads of 64 (time mixing), 128 heads of 64 with a
# state of 128 (state-space duality)
def _shaped(b, window):
    from tesseract_b200.nn.hybrid import ShapedAttention
    from tesseract_b200.ops.masks import Window
    from tesseract_b200.ops.ragged import ScoreForm
    from tesseract_b200.ops.rotary import Rotary
    H, G, D, bf = 32, 8, 128, torch.bfloat16
    if window:
        form = ScoreForm(D ** -0.5, Window(window), slopes=torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]))
        return ShapedAttention(64, H, G, D, D, form, 1e-6, bf, b.dev, bias=True, keys_as_values=True, norm="unit", learned_sink=True, gate="head")
    form = ScoreForm(D ** -0.5, 0, 30.0, None, torch.zeros(H))
    blk = ShapedAttention(64, H, G, D, D, form, 1e-6, bf, b.dev, norm="head", rotary=Rotary(D, 1e4, neighbours=True), gate="element")
    blk.w.q_norm.fill_(1.0)
    blk.w.k_norm.fill_(1.0)
    return blk


def case_shaped_attn(b: Bench):
    """Norms, rotation, append, attention and gate; the counts are those of chunk_attn (two sequences of 4096, or as many rows in
    shorter ones; 256 sequences at 1400 tokens)."""
    for n, rows, window in ((2, 4096, 0), (8, 1024, 0), (2, 4096, 1024)):
        seen = rows * (rows + 1) / 2 if not window else window * (rows - window / 2)
        ms = _mixer_case(b, _shaped(b, window), n, rows)
        report("shaped_attn_prefill", ms, flops=4.0 * n * seen * 32 * 128, shape=[n, rows, window])
    for n, window in ((256, 0), (32, 0), (256, 1024)):
        ms = _mixer_case(b, _shaped(b, window), n, 1, 1399)
        report("shaped_attn_decode", ms, bytes_=n * (window or 1400) * 8 * 128 * 2 * 2.0, shape=[n, 1400, window])


def case_attn_prepare(b: Bench):
    """What comes before attention, alone: biases, norms, rotation, append to the pool and to the key axis (bytes of q, k, v in and out,
    k and v twice), beside the plain append of chunk_attn."""
    from tesseract_b200 import ops
    from tesseract_b200.nn.ragged import PagedRun
    from tesseract_b200.ops import ragged
    n, rows, H, G, D = 4, 4096, 32, 8, 128
    saved, ragged._attend = ragged._attend, lambda *a: None
    try:
        for name, window in (("capped", 0), ("window", 1024)):
            ms = _mixer_case(b, _shaped(b, window), n, rows)
            report("attn_prepare_" + name, ms, bytes_=n * rows * D * 2.0 * (2 * H + (5 if window else 6) * G), shape=[n, rows])
        st = _Step(b, PagedRun(G, D), n, rows, 0, (0,))
        qkv, bias = b.randn(n * rows, (H + 2 * G) * D), torch.zeros((H + 2 * G) * D, device=b.dev)
        ms = b.time(lambda: ops.ragged_attention(qkv, bias, *st.cache.runs[0], st.batch, H, G, D ** -0.5, 0))
        report("ragged_append", ms, bytes_=n * rows * D * 2.0 * (2 * H + 6 * G), shape=[n, rows])
    finally:
        ragged._attend = saved


def case_time_mix(b: Bench):
    """Prompts: bytes of r, k, v, gate and the result; decode: the state read and written once."""
    from tesseract_b200.nn.hybrid import TimeMix
    H, D = 64, 64
    blk = TimeMix(64, H, D, 64, 1e-6, torch.bfloat16, b.dev)
    blk.w.w0.uniform_(-6.0, -1.0)
    blk.w.u.uniform_(0.0, 1.0)
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        report("time_mix_prefill", _mixer_case(b, blk, n, rows), bytes_=n * rows * H * D * 5 * 2.0, shape=[n, rows])
    for n in (256, 32):
        report("time_mix_step", _mixer_case(b, blk, n, 1, 7), bytes_=n * 2.0 * H * D * D * 4, shape=[n])


def case_ssd(b: Bench):
    """Prompts: bytes of z, x, B, C and the result (convolution and norm included); decode: the state read and written once."""
    from tesseract_b200.nn.hybrid import SSD
    H, E, N = 128, 64, 128
    blk = SSD(64, H, E, N, 1, 4, 1, 1e-6, torch.bfloat16, b.dev)
    blk.w.conv.uniform_(-0.5, 0.5)
    blk.w.dt_bias.uniform_(-4.0, -2.0)
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        report("ssd_prefill", _mixer_case(b, blk, n, rows), bytes_=n * rows * (3 * H * E + 2 * N) * 2.0, shape=[n, rows])
    for n in (256, 32):
        report("ssd_step", _mixer_case(b, blk, n, 1, 7), bytes_=n * 2.0 * H * E * N * 4, shape=[n])


def case_post_norm(b: Bench):
    from tesseract_b200 import ops
    T, W = 16384, 4096
    x, y, gain = torch.randn(T, W, device=b.dev, generator=b.gen), b.randn(T, W), torch.ones(W, device=b.dev)
    report("post_norm_step", b.time(lambda: ops.post_norm_step(x, y, gain, 1e-6)), bytes_=T * W * 12.0, shape=[T, W])


def case_token_side(b: Bench):
    """The side input of 4096-wide layers, 128 columns per layer: bytes of the normed input, the looked-up row, x in and out."""
    from tesseract_b200 import ops
    from tesseract_b200.nn.hybrid import TokenSide
    W, V, dim = 4096, 32768, 128
    side = TokenSide(W, dim, 1e-6, torch.bfloat16, b.dev)
    side.w_gate.normal_(std=0.02)
    side.w_proj.normal_(std=0.02)
    table = b.randn(V, dim)
    for T in (16384, 256, 32):
        toks = torch.randint(0, V, (T,), device=b.dev, generator=b.gen, dtype=torch.int32)
        x, h = torch.randn(T, W, device=b.dev, generator=b.gen), b.randn(T, W)
        ms = b.time(lambda: ops.post_norm_step(x, side.forward(h, toks, table, 0), side.norm.gain, 1e-6))
        report("token_side", ms, bytes_=T * (W * 12.0 + dim * 2) + 2 * W * dim * 2.0, shape=[T, W, dim])


def case_token_shift(b: Bench):
    from tesseract_b200.nn.hybrid import TimeMix
    from tesseract_b200.ops.timemix import token_shift
    W = 4096
    blk = TimeMix(W, 64, 64, 64, 1e-6, torch.bfloat16, b.dev)
    st = _Step(b, blk.run_spec(), 4, 4096)
    h = b.randn(4 * 4096, W)
    ms = b.time(lambda: token_shift(h, blk.mu, st.cache.runs[0][0], st.batch, keep=True))
    report("token_shift", ms, bytes_=h.numel() * 2.0 * 7, shape=[4, 4096, W])


def case_project_inputs(b: Bench):
    """One product over six inputs (the first of 6272 columns) against the same product over one."""
    from tesseract_b200 import ops
    starts = (0, 6400, 10496, 14592, 18688, 22784)
    w = b.randn(22848, 4096, scale=0.02)
    for M in (16384, 256, 32):
        xs = b.randn(6, M, 4096)
        kw = dict(flops=2.0 * M * w.shape[0] * 4096) if M > 256 else dict(bytes_=w.numel() * 2.0)
        report("project_inputs", b.time(lambda: ops.project_inputs(xs, w, starts)), shape=[M, w.shape[0], 4096], **kw)
        report("project_one", b.time(lambda: ops.project(xs[0], w)), shape=[M, w.shape[0], 4096], **kw)


# ---- 4096-wide pre-normed layers: 32 heads of 128 x 128 (delta rule, decays per channel), 64 heads of 64 (gated linear attention), 32 / 8
# heads of 128 (attention), 6 of 32 experts of 3584
def case_channel_delta(b: Bench):
    """All launches, the two products of low rank included; counted like delta_prefill and delta_step."""
    from tesseract_b200.nn.hybrid import GatedDelta
    H, D = 32, 128
    blk = GatedDelta(64, H, H, D, D, 4, 1e-6, torch.bfloat16, b.dev, 128, 128)
    blk.w.conv.uniform_(-0.5, 0.5)
    blk.w.dt_bias.uniform_(-6.0, -1.0)
    blk.w.w_decay.normal_(std=0.05)
    blk.w.w_gate.normal_(std=0.05)
    peak = 148 * 128 * 2 * 1.965e9 / 1e12
    for n, rows in ((4, 4096), (1, 4096), (32, 512)):
        ms = _mixer_case(b, blk, n, rows)
        fl = 8.0 * H * D * D * n * rows
        print(json.dumps({"case": "channel_delta_prefill", "ms": round(ms, 4), "fp32_tflops": round(fl / ms / 1e9, 2),
                          "frac_of_nominal_fp32": round(fl / ms / 1e9 / peak, 3), "ns_per_token": round(ms * 1e6 / (n * rows), 1),
                          "shape": [n, rows]}), flush=True)
    for n in (256, 32):
        report("channel_delta_step", _mixer_case(b, blk, n, 1, 7), bytes_=n * 2.0 * H * D * D * 4, shape=[n])


def case_gated_linear(b: Bench):
    """Prompts: bytes of q, k, v, gate and the result; decode: the state read and written once."""
    from tesseract_b200.nn.hybrid import GatedLinear
    for H, D in ((64, 64), (32, 128)):
        blk = GatedLinear(64, H, D, D, 64, 16.0, 1e-6, torch.bfloat16, b.dev)
        blk.w.w2.normal_(std=0.1)
        for n, rows in ((4, 4096), (1, 4096), (32, 512)):
            report("gated_linear_prefill", _mixer_case(b, blk, n, rows), bytes_=n * rows * H * D * 5 * 2.0, shape=[n, rows, H, D])
        for n in (256, 32):
            report("gated_linear_step", _mixer_case(b, blk, n, 1, 7), bytes_=n * 2.0 * H * D * D * 4, shape=[n, H, D])


def case_growing_attn(b: Bench):
    """Counts of shaped_attn."""
    from tesseract_b200.nn.hybrid import ShapedAttention
    from tesseract_b200.ops.ragged import ScoreForm
    blk = ShapedAttention(64, 32, 8, 128, 128, ScoreForm(128 ** -0.5), 1e-6, torch.bfloat16, b.dev, bias=True, gate="element", q_temp=(0.1, 512.0))
    for n, rows in ((2, 4096), (8, 1024)):
        report("growing_attn_prefill", _mixer_case(b, blk, n, rows), flops=4.0 * n * rows * (rows + 1) / 2 * 32 * 128, shape=[n, rows])
    for n in (256, 32):
        report("growing_attn_decode", _mixer_case(b, blk, n, 1, 1399), bytes_=n * 1400 * 8 * 128 * 2 * 2.0, shape=[n, 1400])


def case_pre_norm(b: Bench):
    """The step between two products: bytes of x and y in, x and h out (mixed: the chosen rows)."""
    from tesseract_b200.nn.ragged import StateRun
    from tesseract_b200.ops.moe import Mixed
    from tesseract_b200.ops.pre_norm import Shift, pre_norm_step
    W = 4096
    for n, rows in ((4, 4096), (256, 1), (32, 1)):
        T = n * rows
        st = _Step(b, StateRun((0,), (1, W)), n, rows, 7 if rows == 1 else 0)
        x, y, one = torch.randn(T, W, device=b.dev, generator=b.gen), b.randn(T, W), torch.ones(W, device=b.dev)
        mixed = Mixed(b.randn(T * 6, W), torch.randperm(T * 6, device=b.dev).int().view(T, 6), torch.rand(T, 6, device=b.dev))
        shift = Shift(0.5 * one, st.cache.runs[0][0])
        for name, yy, sh, by in (("plain", y, None, 12), ("shift", y, shift, 12), ("mixed_shift", mixed, shift, 22)):
            ms = b.time(lambda: pre_norm_step(st.batch, W, one, 2, 1e-6, x, yy, one, one, shift=sh, out_dtype=torch.bfloat16))
            report("pre_norm_" + name, ms, bytes_=T * W * float(by), shape=[n, rows, W])


def case_experts(b: Bench):
    """Choice, layout, gather and both products (router and weighted sum not included): prompts by FLOPs, decoded tokens by the bytes
    of the experts that are taken."""
    from tesseract_b200.ops.moe import Choice, relu2_experts
    W, F, c = 4096, 3584, Choice(32, 6, 4, 2, 1.0)
    up, down = b.randn(32, F, W, scale=0.02), b.randn(32, W, F, scale=0.02)
    corr = torch.zeros(32, device=b.dev)
    for T in (16384, 2048, 256, 32, 1):
        h, z = b.randn(T, W), torch.randn(1, T, 32, device=b.dev, generator=b.gen)
        ms = b.time(lambda: relu2_experts(h, z, corr, c, up, down))
        from tesseract_b200.ops.moe import choose_experts_torch
        taken = choose_experts_torch(z[0], corr, c)[0].unique().numel()
        kw = dict(flops=4.0 * T * 6 * W * F) if T > 256 else dict(bytes_=taken * 2 * W * F * 2.0)
        report("experts", ms, shape=[T, 32, 6, W, F], **kw)


def case_gelu_glu(b: Bench):
    from tesseract_b200 import ops
    x = b.randn(16384, 2 * 14336)
    report("gelu_glu", b.time(lambda: ops.gelu_glu(x)), bytes_=x.numel() * 2 * 1.5, shape=list(x.shape))


CASES = {"gemm": case_gemm, "gemm_fp8": case_gemm_fp8, "gemm_fp8_pertensor": case_gemm_fp8_pertensor, "decode_gemm": case_decode_gemm, "gemm_wgrad": case_gemm_wgrad, "grouped_gemm": case_grouped_gemm,
         "flash_fwd": case_flash_fwd, "flash_bwd": case_flash_bwd, "decode": case_decode,
         "decode_int8": case_decode_int8, "rmsnorm": case_rmsnorm, "swiglu": case_swiglu, "swiglu_bwd": case_swiglu_bwd, "adam": case_adam,
         "ce_stats": case_ce, "selective_scan": case_scan, "gemv_w8": case_gemv, "gemm_rs_emul": case_gemm_rs_emul,
         "ag_gemm_emul": case_ag_gemm_emul, "stream_linear": case_stream_linear, "mx_linear": case_mx_linear, "gemm_mx": case_gemm_mx,
         "delta_prefill": case_delta_prefill, "delta_step": case_delta_step, "chunk_attn": case_chunk_attn,
         "dyn_tanh": case_dyn_tanh, "clamped_glu": case_clamped_glu, "retention": case_retention, "latent": case_latent, "rglru": case_rglru,
         "depth_residual": case_depth_residual, "silu_glu": case_silu_glu, "shaped_attn": case_shaped_attn, "attn_prepare": case_attn_prepare, "time_mix": case_time_mix,
         "ssd": case_ssd, "post_norm": case_post_norm, "token_side": case_token_side, "token_shift": case_token_shift,
         "project_inputs": case_project_inputs, "channel_delta": case_channel_delta, "gated_linear": case_gated_linear,
         "growing_attn": case_growing_attn, "pre_norm": case_pre_norm, "experts": case_experts, "gelu_glu": case_gelu_glu}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--case", default="all", choices=["all"] + sorted(CASES))
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--hbm-gbs", type=float, default=0.0, help="measured copy bandwidth of this GPU (GB/s)")
    ap.add_argument("--bf16-tflops", type=float, default=0.0, help="measured library bf16 GEMM rate of this GPU")
    ap.add_argument("--peaks-file", default="", help="JSON file with hbm_gbs and bf16_tflops")
    a = ap.parse_args()
    set_peaks(a.hbm_gbs, a.bf16_tflops, a.peaks_file)
    from tesseract_b200 import _native
    names = sorted(CASES) if a.case == "all" else [a.case]
    for n in names:
        CASES[n](Bench(a.iters))
        torch.cuda.synchronize()
    status = _native.read_status(torch.cuda.current_stream().cuda_stream)
    if status:
        print(json.dumps({"kernel_status": status}))
        sys.exit(1)


if __name__ == "__main__":
    main()
