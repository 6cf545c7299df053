"""Kernel micro-benchmarks (one B200): device-timed with CUDA events after warm-up, with an L2
flush between timed launches, reported against the measured peaks of the box.

    python -m omegalax_b200.ops.microbench gemm --m 16384 --n 6144 --k 4096
    python -m omegalax_b200.ops.microbench attn --batch 8 --seq 4096 --heads 32 --kv-heads 8
    python -m omegalax_b200.ops.microbench gdn --batch 2 --seq 8192 --heads 64 --k-heads 16
    python -m omegalax_b200.ops.microbench decode --batch 32 --ctx 4096
    python -m omegalax_b200.ops.microbench elementwise --rows 32768 --cols 4096
    python -m omegalax_b200.ops.microbench ce --rows 8192 --vocab 151936
    python -m omegalax_b200.ops.microbench serving --batch 2 --seq 8192 --ctx 4096
    python -m omegalax_b200.ops.microbench window --batch 2 --seq 8192 --cols 2048 --kv-heads 4

``--iters 0 --warmup N`` only launches the kernels N times (for a profiler capture of a small
case); ``--baseline`` also times the library counterpart (cuBLAS / SDPA) for comparison.
"""
from __future__ import annotations

import argparse
import json
import os

import torch

from . import kernels as K
from . import lib

bf16 = torch.bfloat16


def _peaks():
    here = os.path.dirname(os.path.abspath(__file__))
    p = os.path.join(os.path.dirname(os.path.dirname(here)), "MEASURED_PEAKS.json")
    try:
        d = json.load(open(p))
        return float(d.get("bf16_tflops", 1590.0)), float(d.get("hbm_gbs", 6650.0)), "measured"
    except Exception:
        return 1590.0, 6650.0, "fallback"


def timeit(fn, iters: int, warmup: int, flush=None):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    if iters <= 0:
        return None
    total = 0.0
    for _ in range(iters):
        if flush is not None:
            flush.add_(1.0)           # 256 MB written: larger than L2
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        total += e0.elapsed_time(e1)
    return total / iters


def _report(name, ms, flops=None, bytes_=None, **extra):
    tf_peak, bw_peak, which = _peaks()
    out = {"kernel": name, "ms": ms, **extra}
    if ms:
        if flops:
            out["tflops"] = flops / ms / 1e9
            out[f"frac_of_{which}_bf16_burst"] = out["tflops"] / tf_peak
        if bytes_:
            out["gbs"] = bytes_ / ms / 1e6
            out[f"frac_of_{which}_hbm"] = out["gbs"] / bw_peak
    print(json.dumps(out), flush=True)


def bench_gemm(a, dev, flush):
    m, n, k = a.m, a.n, a.k
    x = torch.randn(m, k, device=dev).to(bf16)
    w = torch.randn(n, k, device=dev).to(bf16)
    dy = torch.randn(m, n, device=dev).to(bf16)
    acc = torch.zeros(n, k, device=dev)
    fl = 2.0 * m * n * k
    by = 2.0 * (m * k + n * k + m * n)
    _report("gemm fprop  y=x w^T", timeit(lambda: K.gemm(x, w), a.iters, a.warmup, flush), fl, by, m=m, n=n, k=k)
    _report("gemm dgrad  dx=dy w", timeit(lambda: K.gemm(dy, w, b_mn=True), a.iters, a.warmup, flush), fl, by, m=m, n=n, k=k)
    _report("gemm wgrad  dw+=dy^T x (fp32 accumulate)",
            timeit(lambda: K.gemm(dy, x, a_mn=True, b_mn=True, out=acc, accumulate=True), a.iters, a.warmup, flush),
            fl, None, m=m, n=n, k=k)
    for nm, fn in (("fprop", lambda: K.gemm(x, w, pair=True)), ("dgrad", lambda: K.gemm(dy, w, b_mn=True, pair=True)),
                   ("wgrad fp32 accumulate", lambda: K.gemm(dy, x, a_mn=True, b_mn=True, out=acc, accumulate=True, pair=True))):
        _report(f"gemm {nm}, CTA pairs (256x256 tiles)", timeit(fn, a.iters, a.warmup, flush), fl, None, m=m, n=n, k=k)
    if a.baseline:
        _report("cuBLAS fprop", timeit(lambda: torch.matmul(x, w.t()), a.iters, a.warmup, flush), fl, by)
        _report("cuBLAS dgrad", timeit(lambda: torch.matmul(dy, w), a.iters, a.warmup, flush), fl, by)
        _report("cuBLAS wgrad", timeit(lambda: torch.matmul(dy.t(), x), a.iters, a.warmup, flush), fl, None)


def bench_attn(a, dev, flush):
    B, T, H, G, HD = a.batch, a.seq, a.heads, a.kv_heads, a.head_dim
    q = torch.randn(B * T, H, HD, device=dev).to(bf16)
    k = torch.randn(B * T, G, HD, device=dev).to(bf16)
    v = torch.randn(B * T, G, HD, device=dev).to(bf16)
    do = torch.randn_like(q)
    cu = torch.arange(B + 1, device=dev, dtype=torch.int32) * T
    sc = HD ** -0.5
    o, lse = K.attn_fwd(q, k, v, cu, T, sc, True)
    fl = 4.0 * B * T * T * H * HD / 2
    _report("attention fwd (causal, GQA)", timeit(lambda: K.attn_fwd(q, k, v, cu, T, sc, True), a.iters, a.warmup, flush),
            fl, None, batch=B, seq=T, heads=H, kv_heads=G, head_dim=HD)
    if HD in (128, 256):
        _report("attention bwd (causal, GQA)",
                timeit(lambda: K.attn_bwd(q, k, v, o, lse, do, cu, T, sc, True), a.iters, a.warmup, flush), 2.5 * fl, None)
    if a.baseline:
        import torch.nn.functional as F

        q4, k4, v4 = (t.view(B, T, -1, HD).transpose(1, 2) for t in (q, k, v))
        _report("SDPA fwd", timeit(lambda: F.scaled_dot_product_attention(q4, k4, v4, is_causal=True, enable_gqa=True),
                                   a.iters, a.warmup, flush), fl, None)


def bench_gdn(a, dev, flush):
    B, T, H, Hk, A, U = a.batch, a.seq, a.heads, a.k_heads, 128, a.head_dim
    q = torch.nn.functional.normalize(torch.randn(B, T, Hk, A, device=dev), dim=-1) * A ** -0.5
    k = torch.nn.functional.normalize(torch.randn(B, T, Hk, A, device=dev), dim=-1)
    v = torch.randn(B, T, H, U, device=dev)
    g = -torch.rand(B, T, H, device=dev) * 0.3
    beta = torch.sigmoid(torch.randn(B, T, H, device=dev))
    do = torch.randn_like(v)
    o, n_out, states, _ = K.gdn_fwd(q, k, v, g, beta)
    J = T // 64
    macs_f = B * H * J * (2 * 64 * 64 * A + 2 * 64 * A * U + 64 * 64 * U + A * 64 * U)
    _report("gated delta rule fwd (fp32)", timeit(lambda: K.gdn_fwd(q, k, v, g, beta), a.iters, a.warmup, flush),
            2.0 * macs_f, None, batch=B, seq=T, heads=H, k_heads=Hk, head_dim_v=U)
    _report("gated delta rule bwd (fp32)",
            timeit(lambda: K.gdn_bwd(q, k, v, g, beta, n_out, states, do), a.iters, a.warmup, flush), None, None)
    x = torch.randn(B, T, 2 * Hk * A + H * U, device=dev).to(bf16)
    w = torch.randn(x.shape[-1], 4, device=dev).to(bf16)
    by = 2.0 * x.numel() * 2
    _report("causal conv1d+SiLU fwd", timeit(lambda: K.causal_conv1d_fwd(x, w), a.iters, a.warmup, flush), None, by)
    dw = torch.zeros(w.shape, device=dev)
    _report("causal conv1d+SiLU bwd", timeit(lambda: K.causal_conv1d_bwd(x, w, x, dw), a.iters, a.warmup, flush), None, 1.5 * by)


def bench_decode(a, dev, flush):
    B, H, G, HD, ctx, page = a.batch, a.heads, a.kv_heads, 128, a.ctx, 64
    blocks = -(-(ctx + 1) // page)
    k_pages = torch.randn(B * blocks, page, G, HD, device=dev).to(bf16)
    v_pages = torch.randn(B * blocks, page, G, HD, device=dev).to(bf16)
    table = torch.randperm(B * blocks, device=dev).to(torch.int32).view(B, blocks)
    lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
    q = torch.randn(B, H, HD, device=dev).to(bf16)
    by = 2.0 * B * ctx * G * HD * 2
    _report("paged decode attention (split-KV, GQA)",
            timeit(lambda: K.decode_attn(q, k_pages, v_pages, table, lens, page, HD ** -0.5), a.iters, a.warmup, flush),
            None, by, batch=B, ctx=ctx, heads=H, kv_heads=G)


def bench_elementwise(a, dev, flush):
    M, D = a.rows, a.cols
    x = torch.randn(M, D, device=dev).to(bf16)
    w = torch.ones(D, device=dev).to(bf16)
    by = 2.0 * M * D * 2
    _report("rmsnorm fwd", timeit(lambda: K.rmsnorm_fwd(x, w, 1e-6), a.iters, a.warmup, flush), None, by, rows=M, cols=D)
    H, G, Kd = 32, 8, 128
    qkv = torch.randn(M, (H + 2 * G) * Kd, device=dev).to(bf16)
    qw, kw = torch.ones(Kd, device=dev).to(bf16), torch.ones(Kd, device=dev).to(bf16)
    ang = torch.rand(M, Kd // 2, device=dev) * 6.28
    cos, sin = ang.cos().contiguous(), ang.sin().contiguous()
    q, k = K.qknorm_rope_fwd(qkv, qw, kw, cos, sin, H, G, Kd, Kd, 1e-6)
    qb = 2.0 * M * (H + G) * Kd * 2
    _report("qk-norm + rope fwd", timeit(lambda: K.qknorm_rope_fwd(qkv, qw, kw, cos, sin, H, G, Kd, Kd, 1e-6),
                                         a.iters, a.warmup, flush), None, qb, rows=M, heads=H, kv_heads=G)
    dqkv = torch.zeros_like(qkv)
    dqw, dkw = torch.zeros(Kd, device=dev), torch.zeros(Kd, device=dev)
    _report("qk-norm + rope bwd",
            timeit(lambda: K.qknorm_rope_bwd(qkv, qw, kw, cos, sin, q, k, dqkv, dqw, dkw, H, G, Kd, Kd, 1e-6),
                   a.iters, a.warmup, flush), None, 1.5 * qb)
    gu = torch.randn(M, 2 * D, device=dev).to(bf16)
    _report("swiglu fwd", timeit(lambda: K.swiglu_fwd(gu), a.iters, a.warmup, flush), None, 3.0 * M * D * 2)


def bench_ce(a, dev, flush):
    from . import functional as Fn

    M, V, D = a.rows, a.vocab, a.cols
    h = (torch.randn(M, D, device=dev) * 0.5).to(bf16).requires_grad_(True)
    w = (torch.randn(V, D, device=dev) * 0.02).to(bf16).requires_grad_(True)
    y = torch.randint(0, V, (M,), device=dev)
    mask = torch.ones(M, device=dev)

    def step():
        loss = Fn.linear_cross_entropy(h, w, y.to(torch.int32), mask, 1.0 / M)
        loss.backward()
        h.grad = None
        w.grad = None

    _report("fused linear + cross-entropy fwd+bwd", timeit(step, a.iters, a.warmup, flush), 6.0 * M * V * D, None,
            rows=M, vocab=V, hidden=D)


def bench_serving(a, dev, flush):
    """The forward-only serving kernels, each next to the training / Qwen3 kernel it resembles."""
    from . import serving as S

    it = lambda fn: timeit(fn, a.iters, a.warmup, flush)  # noqa: E731
    rn = lambda *s: torch.randn(*s, device=dev).to(bf16)  # noqa: E731
    B, T, D, H = a.batch, a.seq, a.cols, a.heads
    N = B * T
    # row ops
    x, w, xb, FF = torch.randn(N, D, device=dev), rn(D), rn(N, D), 4 * D
    _report("layer norm rows fp32 -> bf16", it(lambda: S.layernorm_rows(x, w, w, 1e-5)), None, N * D * 6.0, rows=N, cols=D)
    _report("  like: rmsnorm bf16", it(lambda: K.rmsnorm_fwd(xb, w, 1e-5, want_rstd=False)), None, N * D * 4.0)
    up = rn(N, FF)
    _report("squared relu", it(lambda: S.relu_squared(up)), None, N * FF * 4.0)
    _report("  like: swiglu", it(lambda: K.swiglu_fwd(up)), None, N * FF * 3.0)
    ids = torch.randint(0, 32000, (N,), device=dev, dtype=torch.int32)
    tab = rn(32000, D)
    _report("embedding rows fp32", it(lambda: S.embed_rows(ids, tab)), None, N * D * 6.0)
    _report("  like: embedding bf16", it(lambda: K.embedding_fwd(ids, tab)), None, N * D * 4.0)
    wq = rn(D, D)
    _report("projection added to fp32 rows", it(lambda: S.project(xb, wq, into=x)), 2.0 * N * D * D, None)
    _report("  like: projection + bf16 residual", it(lambda: K.gemm(xb, wq, residual=xb)), 2.0 * N * D * D, None)
    del x, xb, up, ids, tab, wq
    # prompt attention: 128 + 64 query/key channels, 128 value channels
    d1, d2, vd, R = 128, 64, 128, 512
    q, k2, kv = rn(N, H * (d1 + d2)), rn(N, R + d2), rn(N, H * (d1 + vd))
    cu = torch.arange(B + 1, device=dev, dtype=torch.int32) * T
    _report("latent attention, prompt (192 / 128 channels)",
            it(lambda: S.attn_two_part(q, kv, k2[:, R:], kv[:, H * d1:], cu, T, H, d1, d2, vd, 0.07)),
            float(B) * T * T * H * (d1 + d2 + vd), None, batch=B, seq=T, heads=H)
    q8, k8 = rn(N, H, 128), rn(N, a.kv_heads, 128)
    _report("  like: attention fwd 128 channels", it(lambda: K.attn_fwd(q8, k8, k8, cu, T, 0.09, True, want_lse=False)),
            2.0 * B * T * T * H * 128, None)
    proj = rn(N, H * (d1 + d2) + R + d2)
    pos = (torch.arange(N, device=dev) % T).to(torch.int32)
    row = torch.arange(N, device=dev, dtype=torch.int32)
    cos = torch.randn(T, d2 // 2, device=dev)
    nw, cache, packed = rn(R), rn(N, R + d2), rn(N, R + d2)
    _report("latent prepare (rotate q and key part, norm, store)",
            it(lambda: S.latent_prepare(proj, pos, row, cos, cos, H, d1, d2, R, dkv_off=H * (d1 + d2), norm_w=nw, cache=cache, packed=packed, eps=1e-5)),
            None, N * (2.0 * 2 * H * d2 + 2.0 * 3 * (R + d2)))
    qkv, one, c3 = rn(N, (H + 2 * a.kv_heads) * 128), rn(128), torch.randn(N, 64, device=dev)
    _report("  like: qk-norm + rope", it(lambda: K.qknorm_rope_fwd(qkv, one, one, c3, c3, H, a.kv_heads, 128, 128, 1e-6)), None,
            4.0 * N * (H + a.kv_heads) * 128)
    del q, k2, kv, q8, k8, proj, cache, packed, qkv, c3
    # recurrence
    Kd = V = 128
    pr, z, bias = rn(N, 2 * H * (Kd + V)), torch.randn(N, H * Kd, device=dev), rn(H * Kd)
    st, hist = torch.zeros(max(B, a.decode_batch), H, Kd, V, device=dev), torch.zeros(B, dtype=torch.int32, device=dev)
    alpha = S.gla_decay_(z.clone(), bias, 16.0)
    _report("gla decay", it(lambda: S.gla_decay_(z, bias, 16.0)), None, 8.0 * N * H * Kd)
    fl = 6.0 * N * H * Kd * V
    by = N * H * (2.0 * (2 * Kd + V) + 4.0 * (Kd + V))
    _report("gla scan", it(lambda: S.gla_scan(pr, alpha, st, cu, hist, H, Kd, V, 0.09)), fl, by, batch=B, seq=T, heads=H)
    Tg = T - T % 64
    g4 = [torch.randn(B, Tg, H, 128, device=dev) for _ in range(3)]
    gb = -torch.rand(B, Tg, H, device=dev)
    _report("  like: gated delta rule fwd", it(lambda: K.gdn_fwd(g4[0], g4[1] * 0.05, g4[2], gb, gb.exp(), save=False)), None,
            B * Tg * H * 128 * 16.0)
    del g4
    o = S.gla_scan(pr, alpha, st, cu, hist, H, Kd, V, 0.09)
    _report("gla norm + gate", it(lambda: S.gla_norm_gate(o, pr[:, 2 * H * Kd + H * V:], rn(V), 1e-5)), None, N * H * V * 8.0)
    o2 = rn(N * H, V)
    _report("  like: gated rmsnorm", it(lambda: K.gated_rmsnorm_fwd(o2, o2, one, 1e-5)), None, N * H * V * 6.0)
    del o, o2, pr, z, alpha
    # decode
    Bd, ctx, page = a.decode_batch, a.ctx, 64
    seen = torch.full((Bd,), ctx, dtype=torch.int32, device=dev)
    pd, zd = rn(Bd, 2 * H * (Kd + V)), torch.randn(Bd, H * Kd, device=dev)
    _report("gla step", it(lambda: S.gla_step(pd, zd, bias, rn(V), st, seen, H, Kd, V, 0.09, 16.0, 1e-5)), None, 8.0 * Bd * H * Kd * V, batch=Bd)
    blocks = -(-(ctx + 1) // page)
    table = torch.randperm(Bd * blocks, device=dev).to(torch.int32).view(Bd, blocks)
    lat, ql, qd = rn(Bd * blocks * page, R + d2), rn(Bd, H, R), rn(Bd, H * (d1 + d2))
    _report("latent decode attention", it(lambda: S.latent_decode(ql, qd, d1 + d2, d1, d2, lat, seen, table, page, 0.07)),
            2.0 * Bd * ctx * H * (2 * R + d2), 2.0 * Bd * ctx * (R + d2), batch=Bd, ctx=ctx, heads=H)
    kp, vp, qq = rn(Bd * blocks, page, a.kv_heads, 128), rn(Bd * blocks, page, a.kv_heads, 128), rn(Bd, H, 128)
    _report("  like: paged decode attention", it(lambda: K.decode_attn(qq, kp, vp, table, seen, page, 0.09)), None,
            4.0 * Bd * ctx * a.kv_heads * 128)
    uk, ol = rn(H * d1, R), torch.randn(Bd, H, R, device=dev)
    _report("latent absorb", it(lambda: S.latent_absorb(qd, d1 + d2, uk, H, d1, R, bf16)), None, 2.0 * H * R * (d1 + Bd))
    _report("latent expand", it(lambda: S.latent_expand(ol, uk, d1)), None, 2.0 * H * R * (d1 + 2 * Bd))
    xw, ww = rn(Bd, R), rn(H * d1, R)
    _report("  like: decode projection of as many weights", it(lambda: K.gemm(xw, ww)), None, 2.0 * H * d1 * R)


def bench_window(a, dev, flush):
    """Windowed attention and routed experts of the serving decoders, each next to the kernel of the Qwen3
    mixture it resembles (32 heads of 128 over --kv-heads, 8 of 128 experts of 768)."""
    from . import moe
    from . import serving as S

    it = lambda fn: timeit(fn, a.iters, a.warmup, flush)  # noqa: E731
    rn = lambda *s: torch.randn(*s, device=dev).to(bf16)  # noqa: E731
    B, T, D, H, G, hd = a.batch, a.seq, a.cols, a.heads, a.kv_heads, 128
    N, FF = B * T, 3 * D
    x, w, xb = torch.randn(N, D, device=dev), rn(D), rn(N, D)
    _report("rms norm rows fp32 -> bf16", it(lambda: S.rms_rows(x, w, 1e-5)), None, N * D * 6.0, rows=N, cols=D)
    _report("  like: rmsnorm bf16", it(lambda: K.rmsnorm_fwd(xb, w, 1e-5, want_rstd=False)), None, N * D * 4.0)
    gu = rn(N, 2 * FF)
    _report("gated gelu", it(lambda: S.gated_act(gu, "gelu_tanh")), None, N * FF * 6.0, rows=N, cols=FF)
    _report("gated silu", it(lambda: S.gated_act(gu, "silu")), None, N * FF * 6.0)
    _report("  like: swiglu", it(lambda: K.swiglu_fwd(gu)), None, N * FF * 6.0)
    del gu
    # q, k, v preparation
    pitch = (H + 2 * G) * hd
    proj, first = rn(N, pitch), rn(N, G * hd)
    pos = (torch.arange(N, device=dev) % T).to(torch.int32)
    row = torch.arange(N, device=dev, dtype=torch.int32)
    cos = torch.rand(T, hd // 2, device=dev)
    nw, cache, mix = rn((H + G) * hd), rn(N, 2 * G * hd), torch.tensor(0.3, device=dev).to(bf16)
    _report("window prepare (norms, rotation, value mixing, store)",
            it(lambda: S.window_prepare(proj, pos, row, cos, cos, H, G, hd, hd, nw, cache, 1e-6, mix=mix, v_first=first)), None,
            2.0 * N * hd * (2 * (H + G) + 2 * G + G + 2 * G))
    one, c3 = rn(128), torch.randn(N, 64, device=dev)
    _report("  like: qk-norm + rope", it(lambda: K.qknorm_rope_fwd(proj, one, one, c3, c3, H, G, hd, hd, 1e-6)), None,
            4.0 * N * (H + G) * hd)
    # prompt attention
    cu = torch.arange(B + 1, device=dev, dtype=torch.int32) * T
    q, k, v = proj[:, :H * hd], proj[:, H * hd:(H + G) * hd], proj[:, (H + G) * hd:]
    sink = rn(H)
    for window in (0, 4096, 1024, 128):
        w_ = min(window or T, T)
        pairs = B * (w_ * (w_ + 1) / 2 + (T - w_) * w_)          # (query, visible key)
        _report(f"window attention, prompt, window {window or 'all'}",
                it(lambda: S.attn_window(q, k, v, cu, T, H, G, hd, hd, 0.09, window, sink)), 4.0 * pairs * H * hd, None, batch=B, seq=T)
    q3, k3, v3 = q.unflatten(1, (H, hd)), k.unflatten(1, (G, hd)), v.unflatten(1, (G, hd))
    _report("  like: attention fwd", it(lambda: K.attn_fwd(q3, k3, v3, cu, T, 0.09, True, want_lse=False)), 2.0 * B * T * T * H * hd, None)
    if N % 256 == 0:        # as few tiles per query block as a window of 128 leaves
        cu_s = torch.arange(N // 256 + 1, device=dev, dtype=torch.int32) * 256
        _report("  like: attention fwd, sequences of 256", it(lambda: K.attn_fwd(q3, k3, v3, cu_s, 256, 0.09, True, want_lse=False)),
                2.0 * N * 256 * H * hd, None)
    del proj, first, cache, q, k, v, q3, k3, v3, c3
    # experts, prompts
    E, top, F = 128, 8, 768
    guw, dw, rw = rn(E, 2 * F, D) * 0.02, rn(E, D, F) * 0.02, rn(E, D)
    z = torch.randn(N, E, device=dev)
    zb = z.to(bf16)
    _report("sigmoid router", it(lambda: S.route_sigmoid(z, top)), None, N * (E * 4.0 + top * 8))
    _report("  like: softmax router", it(lambda: K.router_topk(zb, top, True)), None, N * (E * 6.0 + top * 8))
    wt, idx = S.route_sigmoid(z, top)
    fl = 6.0 * N * top * D * F
    _report("experts, prompt (plan, gather, products, gate, sum)", it(lambda: S.experts_into(xb, wt, idx, guw, dw, "silu", x)), fl, None, rows=N)
    i64 = idx.long()
    with torch.no_grad():
        _report("  like: expert mixture", it(lambda: moe.moe_mlp(xb, wt, i64, guw, dw)), fl, None)
    # decode
    Bd, ctx, page = a.decode_batch, a.ctx, 64
    seen = torch.full((Bd,), ctx, dtype=torch.int32, device=dev)
    blocks = -(-(ctx + 1) // page)
    table = torch.randperm(Bd * blocks, device=dev).to(torch.int32).view(Bd, blocks)
    rows_, qd = rn(Bd * blocks * page, 2 * G * hd), rn(Bd, H * hd)
    for window in (0, 1024, 128):
        _report(f"window decode attention, window {window or 'all'}",
                it(lambda: S.window_decode(qd, rows_, seen, table, page, H, G, hd, hd, 0.09, window, sink)), None,
                4.0 * Bd * min(window or ctx, ctx) * G * hd, batch=Bd, ctx=ctx)
    kp, vp, qq = rn(Bd * blocks, page, G, hd), rn(Bd * blocks, page, G, hd), rn(Bd, H, hd)
    _report("  like: paged decode attention", it(lambda: K.decode_attn(qq, kp, vp, table, seen, page, 0.09)), None, 4.0 * Bd * ctx * G * hd)
    hb, xd = rn(Bd, D), torch.randn(Bd, D, device=dev)
    wt, idx = S.route_sigmoid(torch.randn(Bd, E, device=dev), top)
    by = 6.0 * idx.unique().numel() * D * F                      # weights of the experts that are used
    _report("experts, decode", it(lambda: S.experts_into(hb, wt, idx, guw, dw, "silu", xd)), None, by, batch=Bd)
    i64 = idx.long()
    with torch.no_grad():
        _report("  like: expert mixture", it(lambda: moe.moe_mlp(hb, wt, i64, guw, dw)), None, by)
    _report("  (grouped products instead)", it(lambda: S.experts_into(hb, wt, idx, guw, dw, "silu", xd, few=False)), None, by)
    _report("router product", it(lambda: S.project(hb, rw, out_dtype=torch.float32)), None, 2.0 * E * D)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("what", choices=["gemm", "attn", "gdn", "decode", "elementwise", "ce", "serving", "window"])
    ap.add_argument("--m", type=int, default=16384)
    ap.add_argument("--n", type=int, default=6144)
    ap.add_argument("--k", type=int, default=4096)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--seq", type=int, default=4096)
    ap.add_argument("--ctx", type=int, default=4096)
    ap.add_argument("--decode-batch", type=int, default=32)
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--kv-heads", type=int, default=8)
    ap.add_argument("--k-heads", type=int, default=16)
    ap.add_argument("--head-dim", type=int, default=128)
    ap.add_argument("--rows", type=int, default=32768)
    ap.add_argument("--cols", type=int, default=4096)
    ap.add_argument("--vocab", type=int, default=151936)
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--baseline", action="store_true")
    a = ap.parse_args()
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    flush = torch.zeros(64 * 1024 * 1024, device=dev) if a.iters > 0 else None
    {"gemm": bench_gemm, "attn": bench_attn, "gdn": bench_gdn, "decode": bench_decode,
     "elementwise": bench_elementwise, "ce": bench_ce, "serving": bench_serving, "window": bench_window}[a.what](a, dev, flush)
    torch.cuda.synchronize()
    lib.check_status()


if __name__ == "__main__":
    main()
