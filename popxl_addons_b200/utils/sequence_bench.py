"""Kernels of the sequence models (minGRU, differential and sliding-window attention, Dynamic Tanh, RMS norms, small-M linears)
against the roofline, beside the like kernels of the GPT-J / Llama path: `python -m popxl_addons_b200.utils.sequence_bench`.

Device times come from replayed CUDA graphs of back-to-back launches. Every row walks round-robin through enough operand sets
to exceed L2, so operands stream from HBM as inside a step.
"""
import argparse
import json
import os

import torch

from .kernel_bench import graph_time_ms

BF = torch.bfloat16


def _rotating(make, nbytes, fn):
    """`fn(operands)` over operand sets that together exceed L2: `(callable, number of sets)`."""
    n = max(1, min(12, -(-300_000_000 // max(1, nbytes))))
    sets = [make() for _ in range(n)]
    state = {"i": 0}

    def call():
        s = sets[state["i"] % n]
        state["i"] += 1
        return fn(*s)

    return call, n


class Bench:
    def __init__(self, peaks, only=None):
        self.peaks, self.only, self.rows = peaks, only, []

    def row(self, name, make, fn, nbytes=0, flops=0):
        if self.only and self.only not in name:
            return
        call, n = _rotating(make, nbytes, fn)
        ms = graph_time_ms(call, reps=max(n, 24 // n * n))
        t_mem, t_mma = nbytes / self.peaks["hbm_gbs"] / 1e6, flops / self.peaks["bf16_tflops"] / 1e9
        self.rows.append(dict(kernel=name, ms=ms, gbs=nbytes / ms / 1e6, tflops=flops / ms / 1e9, roofline_ms=max(t_mem, t_mma),
                              frac=max(t_mem, t_mma) / ms, bound="memory" if t_mem >= t_mma else "tensor"))
        torch.cuda.empty_cache()


def randn(*shape, dtype=BF):
    return torch.randn(*shape, device="cuda", dtype=dtype)


def prompt_rows(b, nat, ns, T=4096, C=4096, F=11008):
    f32 = torch.float32
    norm = (torch.full((1,), 0.5, device="cuda"), randn(C, dtype=f32), randn(C, dtype=f32))
    b.row(f"stream_dyt {T}x{C}", lambda: (randn(T, C, dtype=f32), randn(T, C)),
          lambda x, y: ns.stream_dyt(x, y, 0.7, None, None, norm, BF), T * C * 12)
    w, bias = randn(C), randn(C)
    b.row(f"  like: layer_norm {T}x{C}", lambda: (randn(T, C),), lambda x: nat.layer_norm_cuda(x, w, bias, 1e-5), T * C * 4)
    b.row(f"  like: rms_norm {T}x{C}", lambda: (randn(T, C),), lambda x: nat.rms_norm_cuda(x, w, 1e-5), T * C * 4)
    y = torch.empty(T, F, device="cuda", dtype=BF)
    b.row(f"swiglu_packed {T}x{F}", lambda: (randn(T, 2 * F),),
          lambda gu: ns._swiglu_packed(gu.data_ptr(), y.data_ptr(), T, F, 2, nat._stream()), T * F * 6)
    b.row(f"  like: swiglu {T}x{F}", lambda: (randn(T, F), randn(T, F)), lambda g, u: nat.swiglu_cuda(g, u), T * F * 6)
    b.row(f"stream_rms {T}x{C}", lambda: (randn(T, C, dtype=f32), randn(T, C)),
          lambda x, d: ns.stream_rms(x, d, 1.0, None, None, norm[1], 1e-6, BF), T * C * 12)
    wide = 6144 + 2 * F  # [plain | gate | up] rows
    b.row(f"clamped_glu {T}x{F}", lambda: (randn(T, wide),),
          lambda p: ns._clamped_glu(p.data_ptr() + 2 * 6144, wide, y.data_ptr(), F, T, F, 7.0, 1.702, 1.0, 2, nat._stream()),
          T * F * 6)
    for width in (C, 1024):
        bz, bx, st = randn(width, dtype=f32) - 3, randn(width, dtype=f32), torch.zeros(1, width, device="cuda")
        pos, cnt = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.full((1,), T, dtype=torch.int32, device="cuda")
        out = torch.empty(T, width, device="cuda", dtype=BF)
        pairs = torch.empty(ns._min_gru_scratch(1, T, width), device="cuda")
        b.row(f"min_gru scan {T}x{width}", lambda: (randn(T, 3 * width),),
              lambda z: ns._min_gru(z.data_ptr(), bz.data_ptr(), bx.data_ptr(), st.data_ptr(), out.data_ptr(), pairs.data_ptr(),
                                    pos.data_ptr(), cnt.data_ptr(), 1, T, width, 2, nat._stream()), T * width * 8)


def attention_rows(b, nat, ns):
    err = nat.gemm_error_flag(torch.device("cuda"))
    for T, H, G, d, dv, chunk in ((4096, 32, 8, 64, 128, 0), (4096, 32, 8, 64, 128, 1024), (4096, 32, 8, 64, 128, 128),
                                  (4096, 16, 16, 128, 128, 0), (2048, 16, 4, 64, 128, 0)):
        ld, cols = (H + G) * 2 * d + G * dv, H * dv
        kc, vc = randn(1, G, 2, T, d), randn(1, G, T, dv)
        pos, cnt = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.full((1,), T, dtype=torch.int32, device="cuda")
        lam, out = torch.full((1,), 0.6, device="cuda"), torch.empty(T, cols, device="cuda", dtype=BF)
        size = chunk or T
        pairs = T * size / 2  # visible (query, key) pairs, half of every chunk's square
        b.row(f"diff_attn {T} tokens H={H} G={G} 2x{d}/{dv} chunk={chunk}", lambda: (randn(T, ld),),
              lambda q: ns._diff_tcgen05(q.data_ptr(), ld, kc.data_ptr(), vc.data_ptr(), out.data_ptr(), cols, pos.data_ptr(),
                                         cnt.data_ptr(), lam.data_ptr(), 1, T, H, G, d, dv, T, chunk, d ** -0.5, 1e-6, 0.4,
                                         err.data_ptr(), nat._stream()),
              T * (H * 2 * d + cols) * 2, 2 * 2 * (d + dv) * pairs * H)
        cos = torch.rand(T, d // 2, device="cuda")
        b.row(f"diff_rope_append {T} tokens H={H} G={G} 2x{d}/{dv}", lambda: (randn(T, ld),),
              lambda q: ns._rope_append(q.data_ptr(), ld, cos.data_ptr(), cos.data_ptr(), kc.data_ptr(), vc.data_ptr(),
                                        pos.data_ptr(), cnt.data_ptr(), 1, T, H, G, d, dv, d, T, 2, nat._stream()),
              T * (2 * H * 2 * d + 2 * G * (2 * d + dv)) * 2)
    for T, H, G, d, dv, window, keep in ((4096, 32, 8, 128, 128, 0, 0), (4096, 32, 8, 128, 128, 1024, 4),
                                         (4096, 64, 8, 64, 64, 128, 4), (4096, 64, 8, 64, 64, 0, 0), (2048, 16, 16, 128, 128, 0, 0)):
        plain, cols = (H + G) * d + G * dv, H * dv
        ld = plain + cols
        kc, vc = randn(1, G, T, d), randn(1, G, T, dv)
        pos, cnt = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.full((1,), T, dtype=torch.int32, device="cuda")
        out, wq = torch.empty(T, cols, device="cuda", dtype=BF), torch.ones(d, device="cuda")
        pairs = sum(min(i + 1, window + min(keep, max(0, i - window + 1))) if window else i + 1 for i in range(T))
        name = f"{T} tokens H={H} G={G} {d}/{dv}"
        b.row(f"window_attn {name} window={window}+{keep}", lambda: (randn(T * H, d), randn(T, ld)),
              lambda q, p: ns._window_tcgen05(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), p.data_ptr() + 2 * plain, ld,
                                              out.data_ptr(), cols, pos.data_ptr(), cnt.data_ptr(), 1, T, H, G, d, dv, T, window,
                                              keep, d ** -0.5, 0.0, err.data_ptr(), nat._stream()),
              T * (H * d + 2 * cols) * 2, 2 * (d + dv) * pairs * H)
        if window == 0:
            b.row(f"qk_norm_append {name}", lambda: (randn(T, ld), randn(T * H, d)),
                  lambda p, q: ns._qk_norm_append(p.data_ptr(), ld, wq.data_ptr(), wq.data_ptr(), q.data_ptr(), kc.data_ptr(),
                                                  vc.data_ptr(), pos.data_ptr(), cnt.data_ptr(), 1, T, H, G, d, dv, T, 1e-6, 2,
                                                  nat._stream()), T * 2 * plain * 2)
    for S, H, D in ((4096, 32, 128), (4096, 16, 256), (2048, 16, 128), (2048, 16, 256)):
        hd = H * D
        b.row(f"  like: attention {S} tokens H={H} D={D}", lambda: (randn(S, 3 * hd),),
              lambda q: nat.flash_attention_fwd(q, 0, hd, 2 * hd, 1, S, H, D, D ** -0.5, True), S * 4 * hd * 2,
              2 * 2 * S * S * D * H / 2)
    S, H, D = 4096, 32, 128
    sc = torch.rand(1, S, D // 2, device="cuda", dtype=BF)
    b.row(f"  like: rotary {S} tokens H={H} D={D}", lambda: (randn(1, H, S, D),),
          lambda x: nat.rotary_launch(x, sc, sc, x, D, False), S * H * D * 4)


def decode_rows(b, nat, ns, C=4096, F=11008, M=16):
    f32 = torch.float32
    norm = (torch.full((1,), 0.5, device="cuda"), randn(C, dtype=f32), randn(C, dtype=f32))
    a, af = randn(M, C), randn(M, F)
    x = randn(M, C, dtype=f32)
    kw = dict(mult=0.7, has_norm=True, has_inject=False)
    b.row(f"small_m store {C}x6144 M={M}", lambda: (randn(6144, C),), lambda w: ns.linear_rows_cuda(a, w, out_dtype=BF), 6144 * C * 2)
    b.row(f"small_m swiglu 2x{F}x{C} M={M}", lambda: (randn(2 * F, C),), lambda w: ns.linear_swiglu_cuda(a, w), 2 * F * C * 2)
    b.row(f"small_m residual {C}x{F} M={M}", lambda: (randn(C, F),),
          lambda w: ns.linear_residual_dyt_cuda(x, af, w, *norm, **kw), F * C * 2)
    b.row(f"small_m residual {C}x{C} M={M}", lambda: (randn(C, C),),
          lambda w: ns.linear_residual_dyt_cuda(x, a, w, *norm, **kw), C * C * 2)
    sq = torch.rand(M, C // 64, device="cuda")
    b.row(f"small_m split_glu (6144 + 2x{F})x{C} M={M}", lambda: (randn(6144 + 2 * F, C),),
          lambda w: ns.linear_split_glu_cuda(a, w, sq, cols=6144, lead=C, limit=7.0, slope=1.702, shift=1.0, eps=1e-6),
          (6144 + 2 * F) * C * 2)
    joint = randn(M, C + F)
    b.row(f"small_m residual rms {C}x{C + F} M={M}", lambda: (randn(C, C + F),),
          lambda w: ns.linear_residual_rms_cuda(x, joint, w, norm[1], mult=1.0, eps=1e-6, deferred=True), (C + F) * C * 2)
    b.row("small_m head 32000x4096 fp32, deferred norm", lambda: (randn(32000, C),),
          lambda w: ns.linear_rows_cuda(a, w, sq, out_dtype=f32, eps=1e-6), 32000 * C * 2)
    bz, bx, st = randn(C, dtype=f32), randn(C, dtype=f32), torch.zeros(M, C, device="cuda")
    one = torch.ones(M, dtype=torch.int32, device="cuda")
    b.row(f"small_m min_gru 3x{C}x{C} M={M}", lambda: (randn(3 * C, C),),
          lambda w: ns.min_gru_cuda(a, w, bz, bx, st, one, one, 1), 3 * C * C * 2)
    b.row("small_m head 32000x4096 fp32", lambda: (randn(32000, C),), lambda w: ns.linear_rows_cuda(a, w, out_dtype=f32),
          32000 * C * 2)
    from ..layers.linear_gq import interleave_scale_zero
    from ..models.generator import quantize_rows

    def gq(N, K):
        packed, scale, zero = quantize_rows(torch.randn(N, K, device="cuda") * 0.02, 64)
        return packed.view(torch.uint16), interleave_scale_zero(scale.half(), zero.half())

    b.row(f"  like: int4 gemm 28672x{C} M={M}", lambda: gq(28672, C), lambda p, s: nat.gq_gemm_small_m(a, p, s, None, None),
          28672 * C // 2 + 28672 * C // 64 * 4)
    b.row(f"  like: int4 gemm {C}x{C} M={M}", lambda: gq(C, C), lambda p, s: nat.gq_gemm_small_m(a, p, s, None, None),
          C * C // 2 + C * C // 64 * 4)
    for B, H, G, d, dv, n in ((16, 32, 8, 64, 128, 2048), (16, 16, 16, 64, 128, 576), (1, 32, 8, 64, 128, 8192),
                              (16, 32, 8, 64, 128, 132)):
        ld, smax = (H + G) * 2 * d + G * dv, n + 64
        cos, lam = torch.rand(smax, d // 2, device="cuda"), torch.full((1,), 0.6, device="cuda")
        pos, cnt = torch.full((B,), n - 1, dtype=torch.int32, device="cuda"), torch.ones(B, dtype=torch.int32, device="cuda")
        q = randn(B, ld)
        b.row(f"diff_attn_decode B={B} H={H} G={G} 2x{d}/{dv} len={n}", lambda: (randn(B, G, 2, smax, d), randn(B, G, smax, dv)),
              lambda kc, vc: ns.diff_attention_cuda(q, cos, cos, kc, vc, pos, cnt, lam, 1, H, d, 0, d ** -0.5, 1e-6, 0.4),
              B * G * n * (2 * d + dv) * 2)
    for B, H, G, d, dv, window, keep, n in ((16, 32, 8, 128, 128, 0, 0, 2048), (16, 64, 8, 64, 64, 0, 0, 2048),
                                            (16, 16, 16, 128, 128, 0, 0, 576), (16, 64, 8, 64, 64, 128, 4, 4096),
                                            (16, 32, 8, 128, 128, 1024, 4, 4096), (1, 32, 8, 128, 128, 0, 0, 8192)):
        ld, smax = (H + G) * d + (G + H) * dv, n + 64
        wq, joint = torch.ones(d, device="cuda"), torch.empty(B, H * dv, dtype=BF, device="cuda")
        pos, cnt = torch.full((B,), n - 1, dtype=torch.int32, device="cuda"), torch.ones(B, dtype=torch.int32, device="cuda")
        q = randn(B, ld)
        b.row(f"window_attn_decode B={B} H={H} G={G} {d}/{dv} window={window}+{keep} len={n}",
              lambda: (randn(B, G, smax, d), randn(B, G, smax, dv)),
              lambda kc, vc: ns.window_attention_cuda(q, wq, wq, kc, vc, pos, cnt, joint, 1, H, window, keep, d ** -0.5, 0.0, 1e-6),
              B * G * (min(n, window + keep) if window else n) * (d + dv) * 2)
    for B, H, D, n in ((16, 16, 128, 576), (16, 8, 128, 2048), (16, 8, 128, 132), (1, 8, 128, 8192)):
        qkv, p = randn(B, 3 * H * D), torch.tensor(n - 1, dtype=torch.int32, device="cuda")
        b.row(f"  like: attn_decode B={B} H={H} D={D} len={n}", lambda: (randn(B, H, n + 64, D), randn(B, H, n + 64, D)),
              lambda kc, vc: nat.attention_decode_packed_cuda(qkv, kc, vc, p, H, D, D ** -0.5), 2 * B * H * n * D * 2)


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--peaks", default=os.path.join(os.path.dirname(__file__), "..", "..", "MEASURED_PEAKS.json"))
    ap.add_argument("--only", default=None, help="run only the rows whose name contains this text")
    a = ap.parse_args(argv)
    peaks, src = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}, "fallback"
    if os.path.exists(a.peaks):
        peaks.update(json.load(open(a.peaks)))
        src = "measured"
    from ..ops import native as nat, native_sequence as ns

    b = Bench(peaks, a.only)
    prompt_rows(b, nat, ns)
    attention_rows(b, nat, ns)
    decode_rows(b, nat, ns)
    nat.check_gemm_errors()
    print(f"peaks ({src}): hbm {peaks['hbm_gbs']} GB/s, bf16 {peaks['bf16_tflops']} TFLOP/s")
    for r in b.rows:
        print(f"{r['kernel']:64s} {r['ms'] * 1e3:9.1f} us {r['gbs']:8.0f} GB/s {r['tflops']:8.1f} TF  "
              f"{r['frac'] * 100:5.1f}% of the {r['bound']} roofline ({src})")


if __name__ == "__main__":
    main()
