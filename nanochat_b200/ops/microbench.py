"""
Micro-benchmarks of the hand-written kernels, one operation per invocation:

    python -m nanochat_b200.ops.microbench gemm --m 32768 --n 4992 --k 1664 --layout fwd
    python -m nanochat_b200.ops.microbench attn_fwd --batch 16 --seq 2048 --heads 13 --window -1
    python -m nanochat_b200.ops.microbench attn_bwd --batch 2 --iters 1 --warmup 1      # small: profiler runs
    python -m nanochat_b200.ops.microbench sweep --m 32768     # the memory-bound kernels against their algorithmic bytes
    python -m nanochat_b200.ops.microbench serve               # serving kernels beside the like kernels of GPT

Timing follows the usual hygiene: warm-up launches, a write larger than L2 between timed launches,
CUDA events on the launching stream, median of the timed launches. Prints one JSON line with the
time, the achieved TFLOP/s (useful FLOPs only: masked attention blocks are not counted) and, when a
`MEASURED_PEAKS.json` with this machine's measured cuBLAS bf16 rate lies in the working directory,
the fraction of that rate.
"""
import argparse
import json
import os

import torch


def _time(fn, iters, warmup, flush=True):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    scratch = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device="cuda") if flush else None
    times = []
    for _ in range(iters):
        if scratch is not None:
            scratch.zero_()                      # evict the previous launch's working set from L2
        e0 = torch.cuda.Event(enable_timing=True)
        e1 = torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1))
    times.sort()
    return times[len(times) // 2]


def _attn_pairs(T, window):
    if window < 0 or window >= T:
        return T * (T + 1) // 2
    return sum(min(i, window) + 1 for i in range(T))


def _operand(shape, dtype):
    """Random operand; 8-bit floats come with the de-quantisation scale of a per-tensor scaling."""
    x = torch.randn(shape, device="cuda")
    if dtype == "bf16":
        return x.to(torch.bfloat16), None
    t = torch.float8_e4m3fn
    scale = x.abs().max() / torch.finfo(t).max
    return (x / scale).to(t), scale.reshape(1).float()


def bench_gemm(args, nat):
    m, n, k = args.m, args.n, args.k
    bf16 = torch.bfloat16
    dev = "cuda"
    if args.dtype == "mxfp8":        # block-scaled fp8, y[m,n] = x[m,k] W[n,k]^T with both operands scaled along k
        assert args.layout == "fwd", "the block-scaled GEMM takes K-major operands: quantise along the reduction dim"
        A = torch.randn(m, k, device=dev).to(bf16)
        B = torch.randn(n, k, device=dev).to(bf16)
        (aq, asf), (bq, bsf) = nat.mx_quantize(A), nat.mx_quantize(B)
        C = torch.empty(m, n, device=dev, dtype=bf16)
        ms = _time(lambda: nat.gemm_mx(aq, asf, bq, bsf, C, bn=args.bn), args.iters, args.warmup)
        ms_q = _time(lambda: nat.mx_quantize(A), args.iters, args.warmup)
        return dict(op="gemm_mx/fwd", dtype="mxfp8", m=m, n=n, k=k, bn=args.bn, ms=ms, tflops=2.0 * m * n * k / ms / 1e9,
                    quantize_a_ms=ms_q, quantize_a_gbs=(m * k * 3 + m * k / 32) / ms_q / 1e6)
    if args.dtype == "fp8" or args.pair >= 0:
        shapes = {"fwd": ((m, k), (n, k)), "dgrad": ((m, k), (k, n)), "wgrad": ((k, m), (k, n))}[args.layout]
        (A, sa), (B, sb) = _operand(shapes[0], args.dtype), _operand(shapes[1], args.dtype)
        wg = args.layout == "wgrad"
        C = torch.zeros(m, n, device=dev, dtype=torch.float32 if wg else bf16)
        kw = dict(a_mn=wg, b_mn=args.layout != "fwd", bn=args.bn, pair=args.pair, scale_a=sa, scale_b=sb)
        if wg:
            kw.update(aux=C, beta=1.0)
        elif args.epi != "linear":     # the MLP's fused epilogues: relu^2 on the way out, or its derivative from the saved output
            kw.update(epi={"relu2": nat.EPI_RELU2, "mul2sqrt": nat.EPI_MUL2SQRT, "relu": nat.EPI_RELU,
                           "mulaux": nat.EPI_MULAUX, "residual": nat.EPI_LINEAR}[args.epi])
            if args.epi in ("mul2sqrt", "mulaux", "residual"):
                kw.update(aux=torch.rand(m, n, device=dev).to(bf16), beta=1.0)
        if args.amax:
            kw.update(amax_out=torch.zeros(1, device=dev))
        ms = _time(lambda: nat.gemm(A, B, C, **kw), args.iters, args.warmup)
        return dict(op=f"gemm/{args.layout}", dtype=args.dtype, pair=args.pair, epi=args.epi, m=m, n=n, k=k, bn=args.bn,
                    ms=ms, tflops=2.0 * m * n * k / ms / 1e9)
    if args.layout == "fwd":        # y[m,n] = x[m,k] W[n,k]^T
        A = torch.randn(m, k, device=dev).to(bf16)
        B = torch.randn(n, k, device=dev).to(bf16)
        C = torch.empty(m, n, device=dev, dtype=bf16)
        fn = lambda: nat.gemm(A, B, C, bn=args.bn)
    elif args.layout == "dgrad":    # dx[m,n] = dy[m,k] W[k,n]   (B is MN-major)
        A = torch.randn(m, k, device=dev).to(bf16)
        B = torch.randn(k, n, device=dev).to(bf16)
        C = torch.empty(m, n, device=dev, dtype=bf16)
        fn = lambda: nat.gemm(A, B, C, b_mn=True, bn=args.bn)
    elif args.layout == "wgrad":    # dW[m,n] (fp32) += dy[k,m]^T x[k,n]   (both MN-major)
        A = torch.randn(k, m, device=dev).to(bf16)
        B = torch.randn(k, n, device=dev).to(bf16)
        C = torch.zeros(m, n, device=dev, dtype=torch.float32)
        fn = lambda: nat.gemm(A, B, C, a_mn=True, b_mn=True, aux=C, beta=1.0, bn=args.bn)
    else:
        raise SystemExit(f"unknown layout {args.layout}")
    ms = _time(fn, args.iters, args.warmup)
    return dict(op=f"gemm/{args.layout}", m=m, n=n, k=k, bn=args.bn, ms=ms, tflops=2.0 * m * n * k / ms / 1e9)


def _attn_inputs(args):
    B, T, H, D = args.batch, args.seq, args.heads, 128
    qkv = torch.randn(B, T, 3 * H * D, device="cuda").to(torch.bfloat16)
    q = qkv[..., :H * D].view(B, T, H, D)
    k = qkv[..., H * D:2 * H * D].view(B, T, H, D)
    v = qkv[..., 2 * H * D:].view(B, T, H, D)
    return qkv, q, k, v


def bench_attn_fwd(args, nat):
    _, q, k, v = _attn_inputs(args)
    ms = _time(lambda: nat.attention_forward(q, k, v, args.window), args.iters, args.warmup)
    flops = 4.0 * args.batch * args.heads * _attn_pairs(args.seq, args.window) * 128
    return dict(op="attn_fwd", batch=args.batch, seq=args.seq, heads=args.heads, window=args.window, ms=ms,
                tflops=flops / ms / 1e9)


def bench_attn_bwd(args, nat):
    qkv, q, k, v = _attn_inputs(args)
    B, T, H, D = q.shape
    y, lse = nat.attention_forward(q, k, v, args.window)
    dy = torch.randn(B, T, H, D, device="cuda").to(torch.bfloat16)
    dqkv = torch.empty_like(qkv)
    views = (dqkv[..., :H * D].view(B, T, H, D), dqkv[..., H * D:2 * H * D].view(B, T, H, D),
             dqkv[..., 2 * H * D:].view(B, T, H, D))
    ms = _time(lambda: nat.attention_backward(dy, q, k, v, y, lse, args.window, views), args.iters, args.warmup)
    flops = 10.0 * B * H * _attn_pairs(T, args.window) * D
    return dict(op="attn_bwd", batch=B, seq=T, heads=H, window=args.window, ms=ms, tflops=flops / ms / 1e9)


def bench_sweep(args, nat):
    """The memory-bound kernels of a training / decode step on d26-shaped operands (inputs larger than L2, about 2 GB
    held in total): device time per launch (CUDA events), algorithmic bytes per launch and the fraction of the measured
    copy bandwidth. Run the same command under `ncu -k regex:... --section SpeedOfLight` for the DRAM counters."""
    C_ = nat._C
    bf16 = torch.bfloat16
    dev = "cuda"
    M, C, H = args.m, 1664, 13
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *shape: torch.randn(*shape, device=dev, generator=g).to(bf16)
    rows = []

    def add(name, fn, nbytes):
        ms = _time(fn, args.iters, args.warmup)
        rows.append(dict(kernel=name, ms=round(ms, 4), algorithmic_mb=round(nbytes / 1e6, 1), gbs=round(nbytes / ms / 1e6, 1)))

    x, x0 = rnd(M, C), rnd(M, C)
    xm, xn = torch.empty_like(x), torch.empty_like(x)
    lam_r, lam_0 = torch.ones(26, device=dev), torch.full((26,), 0.1, device=dev)
    amax = torch.zeros(1, device=dev)
    add("mixnorm_fwd_kernel", lambda: C_.mixnorm_fwd(x, x0, lam_r, lam_0, 3, xm, xn, amax), 4 * M * C * 2)
    add("norm_fwd_kernel", lambda: C_.norm_fwd(x, xn, amax), 2 * M * C * 2)
    dxn, dres = rnd(M, C), rnd(M, C)
    dx, dx0 = torch.empty_like(x), torch.empty_like(x)
    dlr, dl0 = torch.zeros(26, device=dev), torch.zeros(26, device=dev)
    add("mixnorm_bwd_kernel", lambda: C_.mixnorm_bwd(dxn, dres, None, xm, x, x0, lam_r, lam_0, 3, dx, dx0, False, dlr, dl0, amax),
        7 * M * C * 2)
    add("normadd_bwd_kernel", lambda: C_.normadd_bwd(dxn, x, dres, dx, amax), 4 * M * C * 2)
    q8 = torch.empty(M, C, dtype=torch.float8_e4m3fn, device=dev)
    inv = torch.empty(1, device=dev)
    am = x.float().abs().max().reshape(1)
    add("quantize_bf16_kernel", lambda: C_.quantize_bf16(x, am, q8, inv), M * C * 3)
    add("amax_bf16_kernel", lambda: C_.amax_bf16(x, amax), M * C * 2)
    sfb = torch.full((nat.mx_scale_bytes(M, C),), 127, dtype=torch.uint8, device=dev)
    add("mx_quantize_bf16_kernel", lambda: C_.mx_quantize(x, q8, sfb), M * C * 3 + M * C // 32)
    # rotary + QK-norm on the fused QKV buffer
    T = 2048
    qkv = rnd(M, 3 * H * 128)
    cos, sin = rnd(T, 64), rnd(T, 64)
    rstd = torch.empty(M, 2 * H, device=dev)
    add("qkv_post_fwd_kernel", lambda: C_.qkv_post_fwd(qkv, H, H, cos, sin, T, rstd, None, None, None, None),
        2 * M * 2 * H * 128 * 2)
    dqkv = rnd(M, 3 * H * 128)
    add("qkv_post_bwd_kernel", lambda: C_.qkv_post_bwd(dqkv, qkv, H, H, cos, sin, T, rstd, None, None, None, None, None, None,
                                                      None, amax), 3 * M * 2 * H * 128 * 2)
    # loss head on a slice of the logits matrix (rows x 32768 bf16)
    R, V = max(2048, M // 8), 32768
    logits = (rnd(R, V) * 4)
    tgt = torch.randint(0, V, (R,), device=dev, generator=g)
    loss, lse = torch.empty(R, device=dev), torch.empty(R, device=dev)
    add("softcap_ce_fwd_kernel", lambda: C_.softcap_ce_fwd(logits, tgt, loss, lse, V, 15.0), R * V * 2)
    gs = torch.full((1,), 1.0 / R, device=dev)
    g8 = torch.empty(R, V, dtype=torch.float8_e5m2, device=dev)
    add("softcap_ce_bwd_fp8_kernel", lambda: C_.softcap_ce_bwd_fp8(logits, tgt, lse, gs, gs, g8, inv, V, 15.0), R * V * 3)
    # optimizer elementwise passes
    n = 32 * 1024 * 1024
    p32, g32 = torch.randn(n, device=dev), torch.randn(n, device=dev)
    m32, v32 = torch.zeros(n, device=dev), torch.zeros(n, device=dev)
    sh = torch.empty(n, dtype=bf16, device=dev)
    add("adamw_kernel<float,float>", lambda: C_.adamw_step(p32, g32, m32, v32, sh, 1e-3, 0.8, 0.95, 1e-10, 0.0, 3, 1.0),
        n * (4 * 4 + 3 * 4 + 2))
    k, r, c = 8, 1664, 1664
    P, X = torch.randn(k, r, c, device=dev), rnd(k, r, c)
    sec = torch.zeros(k, r, device=dev)
    ss, sc = torch.empty(k * r, device=dev), torch.empty(k * r, device=dev)
    shadow = torch.empty(k, r, c, dtype=bf16, device=dev)
    add("muon_finish (sumsq + stats + muon_apply_kernel)", lambda: C_.muon_finish(P, X, sec, ss, sc, shadow, 0.02, 0.1, 0.9),
        k * r * c * (2 + 2 + 4 + 4 + 2))
    # decode: weight-streaming GEMV and split-key attention
    W = rnd(4 * C, C)
    for B in (1, 8):
        xv, out = rnd(B, C), torch.empty(B, 4 * C, dtype=bf16, device=dev)
        add(f"gemv_rows_kernel<{B}>", lambda: C_.gemv_rows(xv, W, out, None, 0, False), W.numel() * 2)
    Bd, Tc = 8, 2048
    kc, vc = rnd(Bd, Tc, H, 128), rnd(Bd, Tc, H, 128)
    qd, yd = rnd(Bd, H * 128), torch.empty(Bd, H * 128, dtype=bf16, device=dev)
    seq = torch.full((Bd,), Tc - 1, dtype=torch.int32, device=dev)
    scratch = torch.zeros(C_.decode_attn_scratch(Bd, H), device=dev)
    add("decode_attn_kernel", lambda: C_.decode_attn(qd, kc, vc, seq, H, H, -1, 0.088, scratch, yd), 2 * kc.numel() * 2)
    peak = None
    if os.path.exists("MEASURED_PEAKS.json"):
        with open("MEASURED_PEAKS.json") as f:
            peak = json.load(f).get("hbm_gbs")
    for row in rows:
        if peak:
            row["frac_of_measured_hbm"] = round(row["gbs"] / peak, 3)
    return dict(op="sweep", rows_m=M, kernels=rows, measured_hbm_gbs=peak)


def _time_chain(calls, iters=10):
    """Microseconds per call of a captured chain of calls (their launch cost is the graph's, as in a decode step)."""
    for c in calls:
        c()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for c in calls:
            c()
    return 1e3 * _time(g.replay, iters, 3) / len(calls)


def bench_serve(T=2048, C=1664, window=512, ctx=1024):
    """Every kernel of the latent-attention model at the d26 width beside the like kernel of GPT: time, roofline (the
    slower of its FLOPs at the measured GEMM rate and its bytes at the measured copy rate) and the ratio of the two
    distances. Prompt kernels: T tokens. Decode kernels: chains over several layers' weights (more than L2)."""
    from nanochat_b200.ops import native as nat
    from nanochat_b200.ops import serving as sv
    K, N = sv._S, nat._C
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    if os.path.exists("MEASURED_PEAKS.json"):
        with open("MEASURED_PEAKS.json") as f:
            peaks.update({k: v for k, v in json.load(f).items() if k in peaks})
    dev, bf16, f32 = "cuda", torch.bfloat16, torch.float32
    r = lambda *s, dtype=bf16: torch.randn(*s, device=dev).to(dtype)
    e = lambda *s, dtype=bf16: torch.empty(*s, device=dev, dtype=dtype)
    H, D, D2, DV, KV = C // 128, 128, 64, 128, 512
    E, TOP, FF = 16, 4, C
    rows, base = [], {}

    def add(name, us, flops=0.0, nbytes=0.0, like=None, key=None):
        roof = max(flops / peaks["bf16_tflops"] / 1e6, nbytes / peaks["hbm_gbs"] / 1e3)
        row = {"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "distance": round(us / roof, 2)}
        if like is not None:
            row["like"] = like
            row["relative_distance"] = round(us / roof / base[like], 2)
        if key is not None:
            base[key] = us / roof
        rows.append(row)

    us = lambda fn: 1e3 * _time(fn, 10, 3)
    # ------------------------------------------------------------------ prompts
    x, w, y = r(T, C), r(4 * C, C), e(T, 4 * C)
    add("gpt gemm (MLP up)", us(lambda: nat.gemm(x, w, y)), 2.0 * T * C * 4 * C, key="gemm")
    n_in = 1280 + 576 + 2 * C + 4 * C
    w_in, z = r(n_in, C), e(T, n_in)
    add("gemm (fused input projection)", us(lambda: K.gemm(x, w_in, z)), 2.0 * T * C * n_in, like="gemm")
    idx, wt = torch.empty(T, TOP, dtype=torch.int32, device=dev), e(T, TOP, dtype=f32)
    rank, slot, off = torch.empty_like(idx), torch.empty_like(idx), torch.empty(E, dtype=torch.int32, device=dev)
    counts, logits = torch.zeros(E, dtype=torch.int32, device=dev), r(T, E, dtype=f32)
    tiles = -(-(T * TOP + E * 127) // 128)
    tg = torch.empty(tiles, dtype=torch.int32, device=dev)
    xg, wgu, gu, act, wd, yg = e(tiles * 128, C), r(E, 2 * FF, C), e(tiles * 128, 2 * FF), e(tiles * 128, FF), r(E, C, FF), e(tiles * 128, C)

    def regroup():
        counts.zero_()
        K.route_topk(logits, E, idx, wt, counts, rank)
        K.group_rows(x, idx, rank, counts, off, tg, slot, xg)
    regroup()
    add("grouped gemm (experts' gate and up)", us(lambda: K.gemm(xg, wgu, gu, tg)), 2.0 * T * TOP * C * 2 * FF, like="gemm")
    add("grouped gemm (experts' down)", us(lambda: K.gemm(act, wd, yg, tg)), 2.0 * T * TOP * C * FF, like="gemm")
    for win, tag in ((-1, "all keys"), (window, f"window {window}")):
        q, k, v, o = (r(1, T, H, 128) for _ in range(4))
        lse = e(1, H, T, dtype=f32)
        pairs = _attn_pairs(T, win)
        add(f"gpt attention, {tag}", us(lambda: N.attn_fwd(q, k, v, o, lse, win, 0.088)), 4.0 * H * 128 * pairs, key=f"attn{win}")
        q4, k3, k2, v3, o3 = r(T, H, D + D2), r(T, H, D), r(T, D2), r(T, H, DV), e(T, H, DV)
        add(f"split attention, {tag}", us(lambda: K.attention_split(q4[..., :D], q4[..., D:], k3, k2, v3, o3, win, 0.07)),
            2.0 * H * (D + D2 + DV) * pairs, like=f"attn{win}")
    xr, lam = r(T, C), torch.ones(1, device=dev)
    xm, xn = e(T, C), e(T, C)
    add("gpt mix + norm", us(lambda: N.mixnorm_fwd(xr, x, lam, lam, 0, xm, xn, None)), nbytes=2.0 * T * C * 4, key="rows")
    xf, bias, wn = r(T, C, dtype=f32), r(C, dtype=f32), r(C, dtype=f32)
    g1, g2, y1, h = z[:, :C], z[:, C:2 * C], r(T, C), e(T, C)
    add("gated residual + norm, dense", us(lambda: K.gated_residual_norm(xf, [[g1, bias, y1], [g2, bias, y1]], 0.7, None, wn, 1e-6, C, h)),
        nbytes=T * C * (8 + 2 * 4 + 2.0), like="rows")
    add("gated residual + norm, experts", us(lambda: K.gated_residual_norm(xf, [[g1, bias, y1], [g2, bias, yg, slot, wt]], 0.7, None, wn, 1e-6, C, h)),
        nbytes=T * C * (8 + 2 * 3 + 2.0 * TOP + 2.0), like="rows")
    coef, zu, au = torch.tensor([0.7, 0.3, 0.1, 0.0], device=dev), z[:, :4 * C], e(T, 4 * C)
    add("normed-powers activation", us(lambda: K.poly_norm(zu, coef, 1e-6, 4 * C, au)), nbytes=2.0 * T * 4 * C * 2, like="rows")
    add("gather rows by expert", us(lambda: K.group_rows(x, idx, rank, counts, off, tg, slot, xg)), nbytes=2.0 * (1 + TOP) * T * C, like="rows")
    add("silu * up", us(lambda: K.silu_mul(gu, tg, act)), nbytes=2.0 * T * TOP * FF * 3, like="rows")
    P = 64
    pages = -(-(T + 1) // P)
    pool = torch.zeros(pages, P, KV + D2, dtype=bf16, device=dev)
    table = torch.arange(pages, dtype=torch.int32, device=dev)[None].contiguous()
    lens, freq = torch.zeros(1, dtype=torch.int32, device=dev), 10000.0 ** (-torch.arange(D2 // 2, device=dev, dtype=f32) * 2 / D2)
    qkv, cs = r(1, T, 3 * H * 128), e(1, T, 64)
    qw, kw, cq, kv = r(1280, dtype=f32), r(KV, dtype=f32), e(T, 1280), e(T, KV + D2)
    cs.fill_(0.7)
    rstd = e(T, 2 * H, dtype=f32)
    add("gpt rotary + QK norm", us(lambda: N.qkv_post_fwd(qkv, H, H, cs.view(T, 64), cs.view(T, 64), T, rstd, None, None, None, None)),
        nbytes=2.0 * T * 2 * H * 128 * 2, key="post")
    add("latent norms + store", us(lambda: K.latent_post(z, 1280, qw, cq, 1280, KV, KV, kw, 1e-6, 1280 + KV, D2, freq, pool, table, lens, T, kv)),
        nbytes=2.0 * T * (2 * 1280 + 3 * (KV + D2)), like="post")
    q5 = r(T, H * (D + D2))
    add("rotate query heads", us(lambda: K.rotate_heads(q5, H, D, freq, table, lens, T)), nbytes=4.0 * T * H * D2, like="post")
    # ------------------------------------------------------------------- decode
    L = 12                                          # chain length: weights of several layers, more than L2 holds
    for B in (1, 8):
        lens = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        xb, wq, ob = r(B, C), [r(3 * C, C) for _ in range(L)], e(B, 3 * C)
        add(f"gpt gemv (QKV), {B} rows", _time_chain([lambda a=a: N.gemv_rows(xb, a, ob, None, 0, True, None) for a in wq]), nbytes=2.0 * 3 * C * C, key=f"gemv{B}")
        wp, op, aux = [r(C, C) for _ in range(L)], e(B, C), r(B, C)
        add(f"gpt gemv (attention out), {B} rows", _time_chain([lambda a=a: N.gemv_rows(xb, a, op, aux, 0, False, None) for a in wp]), nbytes=2.0 * C * C, key=f"gemvo{B}")
        n_all = n_in
        wa, zb, xf = [r(n_all, C) for _ in range(L)], e(B, n_all, dtype=f32), r(B, C, dtype=f32)
        add(f"norm + input projection, {B} rows", _time_chain([lambda a=a: K.gemv_norm(xf, wn, 1e-6, C, a, zb) for a in wa]), nbytes=2.0 * n_all * C, like=f"gemv{B}")
        zb.normal_()
        pg = -(-ctx // P)
        pools = [torch.randn(B * pg, P, KV + D2, device=dev).to(bf16) for _ in range(L)]
        table = torch.arange(B * pg, dtype=torch.int32, device=dev).view(B, pg).contiguous()
        wqs, qb = [r(H * (D + D2), 1280) for _ in range(L)], e(B, H * (D + D2))
        add(f"query projection + store, {B} rows", _time_chain([lambda a=a, p=p: K.gemv_query_store(zb, 1280, qw, 1e-6, a, qb, 1280, KV, KV, kw, 1280 + KV, D2, freq, p, table, lens)
                                                                 for a, p in zip(wqs, pools)]), nbytes=2.0 * 1280 * H * (D + D2), like=f"gemvo{B}")
        wkv, qa, yb = [r(H * (D + DV), KV) for _ in range(L)], e(B, H, KV), e(B, H * DV)
        add(f"absorb queries, {B} rows", _time_chain([lambda a=a: K.absorb_query(qb, H, a[:H * D], qa, True) for a in wkv]), nbytes=2.0 * H * D * KV, like=f"gemvo{B}")
        k4 = [torch.randn(B * pg, P, H, 128, device=dev).to(bf16) for _ in range(L)]
        scratch, yg4, qg = torch.zeros(N.decode_attn_scratch(B, H), device=dev), e(B, H * 128), r(B, H * 128)
        add(f"gpt decode attention, {window} keys, {B} rows", _time_chain([lambda a=a: N.decode_attn(qg, a, a, lens, H, H, window - 1, 0.088, scratch, yg4, table) for a in k4]),
            nbytes=2.0 * B * window * H * 256, flops=4.0 * B * window * H * 128, key=f"dattn{B}")

        class P_:                                   # what attention_splits asks for
            heads, window = H, None
        splits = sv.attention_splits(P_, B, window, True)
        ml, acc = e(B, H, splits, 2, dtype=f32), e(B, H, splits, KV, dtype=f32)
        add(f"latent attention, {window} keys, {B} rows", _time_chain([lambda p=p: K.latent_attention(qa, qb, H, D, D2, freq, KV, p, table, lens, 1, window, 0.07, splits, ml, acc, True) for p in pools]),
            nbytes=2.0 * B * window * (KV + D2), flops=2.0 * B * window * H * (2 * KV + D2), like=f"dattn{B}")
        add(f"merge splits + values, {B} rows", _time_chain([lambda a=a: K.latent_values(ml, acc, B, H, splits, a[H * D:], yb, True) for a in wkv]), nbytes=2.0 * H * DV * KV, like=f"gemvo{B}")
        wo, gb = [r(C, H * DV) for _ in range(L)], zb[:, :C]
        add(f"output projection + gated residual, {B} rows", _time_chain([lambda a=a: K.gemv_residual(yb, a, xf, gb, bias, 0.7) for a in wo]), nbytes=2.0 * C * H * DV, like=f"gemvo{B}")
        wdn, zz, az = [r(C, 4 * C) for _ in range(L)], zb[:, :4 * C], e(B, 4 * C)
        hb, ff = r(B, 4 * C), e(B, C, dtype=f32)
        add(f"gpt gemv (MLP down), {B} rows", _time_chain([lambda a=a: N.gemv_rows(hb, a, op, aux, 0, False, None) for a in wdn]), nbytes=2.0 * 4 * C * C, key=f"gemvd{B}")
        add(f"activation, then down + gate, {B} rows", _time_chain([lambda a=a: (K.poly_norm(zz, coef, 1e-6, 4 * C, az), K.gemv_residual(az, a, ff, gb, bias, 0.7, accumulate=False)) for a in wdn]),
            nbytes=2.0 * 4 * C * C, like=f"gemvd{B}")
        lbs, hb, ab = [r(B, E, dtype=f32) for _ in range(L)], r(B, C), e(B * TOP, FF)       # other experts in every call
        ids, wts = torch.empty(B, TOP, dtype=torch.int32, device=dev), e(B, TOP, dtype=f32)
        used = min(B * TOP, E * (1 - (1 - TOP / E) ** B))      # experts a step reads, on average
        add(f"routing + experts, {B} rows", _time_chain([lambda l=l: (K.route_topk(l, E, ids, wts), K.expert_rows(hb, wgu, wd, ids, wts, ab, ff, gb, bias, 0.7)) for l in lbs]),
            nbytes=2.0 * used * 3 * FF * C, like=f"gemvd{B}")
    sv.check_status()
    nat.check_status()
    return rows


def bench_recurrent(T=2048, C=1664, window=512, ctx=1024):
    """Every kernel of the model with recurrent layers (Safepel) at the d26 width beside the like kernel of GPT, as
    `bench_serve` does: heads of 128 dimensions, as many as GPT's in every mixer, one key head per value head in the delta
    rule and one for all in the window attention. A recurrence's roofline counts its inputs, outputs and state once and
    6 (delta) or 4 (fixed decay) operations per state entry and token, whatever the kernels do internally."""
    from nanochat_b200.ops import native as nat
    from nanochat_b200.ops import serving as sv
    K, N = sv._S, nat._C
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    if os.path.exists("MEASURED_PEAKS.json"):
        with open("MEASURED_PEAKS.json") as f:
            peaks.update({k: v for k, v in json.load(f).items() if k in peaks})
    dev, bf16, f32 = "cuda", torch.bfloat16, torch.float32
    r = lambda *s, dtype=bf16: torch.randn(*s, device=dev).to(dtype)
    e = lambda *s, dtype=bf16: torch.empty(*s, device=dev, dtype=dtype)
    H, D, ff, taps, P = C // 128, 128, -(-C * 8 // 3 // 64) * 64, 4, 64
    rows, base = [], {}

    def add(name, us, flops=0.0, nbytes=0.0, like=None, key=None):
        roof = max(flops / peaks["bf16_tflops"] / 1e6, nbytes / peaks["hbm_gbs"] / 1e3)
        row = {"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "distance": round(us / roof, 2)}
        if like is not None:
            row["like"] = like
            row["relative_distance"] = round(us / roof / base[like], 2)
        if key is not None:
            base[key] = us / roof
        rows.append(row)

    us = lambda fn: 1e3 * _time(fn, 10, 3)
    # ------------------------------------------------------------------ prompts
    x, w, y = r(T, C), r(4 * C, C), e(T, 4 * C)
    add("gpt gemm (MLP up)", us(lambda: nat.gemm(x, w, y)), 2.0 * T * C * 4 * C, key="gemm")
    w_in, z = r(4 * H * D, C), e(T, 4 * H * D)
    add("gemm (delta input projection)", us(lambda: K.gemm(x, w_in, z)), 2.0 * T * C * 4 * H * D, like="gemm")
    gu, act = r(2 * ff, C), e(T, ff)
    add("gemm pair (gate with relu, up times gate)", us(lambda: (K.gemm(x, gu[:ff], act, epi=1), K.gemm(x, gu[ff:], act, epi=2, aux=act))),
        2.0 * T * C * 2 * ff, like="gemm")
    xr, lam = r(T, C), torch.ones(1, device=dev)
    xm, xn = e(T, C), e(T, C)
    add("gpt mix + norm", us(lambda: N.mixnorm_fwd(xr, x, lam, lam, 0, xm, xn, None)), nbytes=2.0 * T * C * 4, key="rows")
    xf, wn, h = r(T, C, dtype=f32), r(C, dtype=f32), e(T, C)
    add("norm + residual + norm", us(lambda: K.layer_norm_residual(None, x, 0, wn, xf, wn, 1e-6, C, h)), nbytes=T * C * (8 + 2 + 2.0), like="rows")
    hp = -(-H // 8) * 8
    wba, ba = r(2 * hp, C), e(T, 2 * hp, dtype=f32)
    add("beta and decay inputs (product of few outputs)", _time_chain([lambda: K.gemv_plain(x, wba, ba)] * 8), nbytes=2.0 * (T + 2 * hp) * C, like="rows")
    for win, tag in ((window, f"window {window}"),):
        q, k, v, o = (r(1, T, H, 128) for _ in range(4))
        lse = e(1, H, T, dtype=f32)
        pairs = _attn_pairs(T, win)
        add(f"gpt attention, {tag}", us(lambda: N.attn_fwd(q, k, v, o, lse, win, 0.088)), 4.0 * H * 128 * pairs, key="attn")
        q3, kv, o3 = r(T, H, D), r(T, 2, 1, D), e(T, H, D)
        for cap, what in ((0.0, "no cap"), (20.0, "soft cap")):
            add(f"grouped attention, {tag}, {what}", us(lambda: K.attention_capped(q3, kv[:, 0], kv[:, 1], o3, win - 1, 0.088, cap, 0.7)), 4.0 * H * 128 * pairs, like="attn")
    qkv, cs, rstd = r(1, T, 3 * H * 128), torch.full((1, T, 64), 0.7, device=dev, dtype=bf16), e(T, 2 * H, dtype=f32)
    add("gpt rotary + QK norm", us(lambda: N.qkv_post_fwd(qkv, H, H, cs.view(T, 64), cs.view(T, 64), T, rstd, None, None, None, None)),
        nbytes=2.0 * T * 2 * H * 128 * 2, key="post")
    size, ch = [H, H, D, D, D, D, taps, hp], 3 * H * D
    conv, one, lens = r(taps * ch, dtype=f32), torch.ones(hp, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    ring, state = torch.zeros(1, taps, ch, device=dev), torch.zeros(1, H, D, D, device=dev)
    norms, bg = e(T, 2 * H, dtype=f32), e(T, 2 * H, dtype=f32)
    tiles = torch.empty(K.recurrence_tiles(1, T, H, H, D, D), dtype=torch.uint8, device=dev)
    add("convolutions, unit norms, step sizes", us(lambda: K.delta_prepare(z, size, conv, ba, -one, one, ring, lens, T, tiles, norms, bg)), nbytes=2.0 * T * 2 * ch, like="post")
    o2, y2, scratch = e(T, H * D), e(T, H * D), torch.empty(K.recurrence_scratch(1, T, H, True), dtype=torch.uint8, device=dev)
    add("delta rule in chunks (two kernels)", us(lambda: K.recurrence(tiles, [H, H, D, D], norms, bg, None, state, lens, T, o2, scratch)),
        6.0 * T * H * D * D, nbytes=2.0 * T * 4 * H * D + 8.0 * H * D * D, like="attn")
    gate, wd = z[:, ch:], r(D, dtype=f32)
    add("head norm + gate", us(lambda: K.delta_finish(o2, gate, wd, 1e-6, y2, z, size, conv, -one, one, ring, lens, T)), nbytes=2.0 * T * 3 * H * D, like="post")
    add("silu of the fixed-decay inputs", us(lambda: K.decay_prepare(z[:, :ch], H, D, D, T, tiles)), nbytes=2.0 * T * 2 * ch, like="post")
    ld, wr = torch.full((hp,), -0.01, device=dev), r(H * D, dtype=f32)
    add("fixed decay in chunks (two kernels)", us(lambda: K.recurrence(tiles, [H, H, D, D], None, None, ld, state, lens, T, o2, scratch)),
        4.0 * T * H * D * D, nbytes=2.0 * T * 4 * H * D + 8.0 * H * D * D, like="attn")
    add("row norm + gate", us(lambda: K.norm_gate(o2, gate, wr, 1e-6, 1, H * D, True, 0.7, y2)), nbytes=2.0 * T * 3 * H * D, like="post")
    pages = -(-(T + 1) // P)
    pool, table = torch.zeros(pages, P, 2 * D, dtype=bf16, device=dev), torch.arange(pages, dtype=torch.int32, device=dev)[None].contiguous()
    freq, dense = torch.stack([10000.0 ** (-torch.arange(D // 2, device=dev, dtype=f32) * 2 / D), torch.zeros(D // 2, device=dev)]), e(T, 2 * D)
    wsize, wreal = [H, 1, D, 0, H * D, window], [0.088, 20.0, 0.7]
    add("rotate queries, keys into the store", us(lambda: K.window_post(z, wsize, wreal, freq, pool, table, lens, T, dense)), nbytes=2.0 * T * (2 * H * D + D + 4 * D), like="post")
    # ------------------------------------------------------------------- decode
    L = 12                                          # chain length: weights of several layers, more than L2 holds
    for B in (1, 8):
        lens = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        xb, wq, ob = r(B, C), [r(3 * C, C) for _ in range(L)], e(B, 3 * C)
        add(f"gpt gemv (QKV), {B} rows", _time_chain([lambda a=a: N.gemv_rows(xb, a, ob, None, 0, True, None) for a in wq]), nbytes=2.0 * 3 * C * C, key=f"gemv{B}")
        wp, op, aux = [r(C, C) for _ in range(L)], e(B, C), r(B, C)
        add(f"gpt gemv (attention out), {B} rows", _time_chain([lambda a=a: N.gemv_rows(xb, a, op, aux, 0, False, None) for a in wp]), nbytes=2.0 * C * C, key=f"gemvo{B}")
        lam, xs = torch.ones(1, device=dev), [r(B, C) for _ in range(L)]
        add(f"gpt mix + norm, {B} rows", _time_chain([lambda a=a: N.mixnorm_fwd(a, xb, lam, lam, 0, e1, e2, None) for e1, e2 in ((e(B, C), e(B, C)),) for a in xs]),
            nbytes=2.0 * B * C * 4, key=f"row{B}")
        n_in = 4 * H * D + 2 * hp
        wa, zb = [r(n_in, C) for _ in range(L)], e(B, n_in, dtype=f32)
        add(f"delta input projection, {B} rows", _time_chain([lambda a=a: K.gemv_plain(xb, a, zb) for a in wa]), nbytes=2.0 * n_in * C, like=f"gemv{B}")
        zb.normal_()
        pg = -(-ctx // P)
        table = torch.arange(B * pg, dtype=torch.int32, device=dev).view(B, pg).contiguous()
        k4 = [torch.randn(B * pg, P, H, 128, device=dev).to(bf16) for _ in range(L)]
        scr, yg, qg = torch.zeros(N.decode_attn_scratch(B, H), device=dev), e(B, H * 128), r(B, H * 128)
        add(f"gpt decode attention, {window} keys, {B} rows", _time_chain([lambda a=a: N.decode_attn(qg, a, a, lens, H, H, window - 1, 0.088, scr, yg, table) for a in k4]),
            nbytes=2.0 * B * window * H * 256, flops=4.0 * B * window * H * 128, key=f"dattn{B}")
        del k4
        states, rings, yb = [torch.zeros(B, H, D, D, device=dev) for _ in range(L)], torch.zeros(B, taps, ch, device=dev), e(B, H * D)
        add(f"delta step, {B} rows", _time_chain([lambda s=s: K.delta_step(zb, size, conv, zb[:, 4 * H * D:], -one, one, rings, s, lens, wd, 1e-6, ch, yb) for s in states]),
            nbytes=8.0 * B * H * D * D, flops=6.0 * B * H * D * D, like=f"dattn{B}")
        pools = [torch.randn(B * pg, P, 2 * D, device=dev).to(bf16) for _ in range(L)]
        zp, wsz = r(B, H * D + D + 4 * H * D, dtype=f32), [H, 1, D, 0, H * D, window]
        dsz = [H, D, D, D, H * D + D, 2 * H * D + D, 3 * H * D + D, 4 * H * D + D]
        o4, done, y4 = e(B, H * D, dtype=f32), torch.zeros(B, dtype=torch.int32, device=dev), e(B, 2 * H * D)
        add(f"window attention beside fixed decay, {B} rows",
            _time_chain([lambda p=p, s=s: K.parallel_step(zp, wsz, wreal, freq, p, table, lens, y4[:, :H * D], dsz, [1e-6, 0.7], ld, s, wr, o4, done, y4[:, H * D:])
                         for p, s in zip(pools, states)]),
            nbytes=8.0 * B * H * D * D + 2.0 * B * window * 2 * D, flops=4.0 * B * H * D * (D + window), like=f"dattn{B}")
        wo, out = [r(C, H * D) for _ in range(L)], e(B, C, dtype=f32)
        add(f"output projection, {B} rows", _time_chain([lambda a=a: K.gemv_plain(yb, a, out) for a in wo]), nbytes=2.0 * C * H * D, like=f"gemvo{B}")
        xf, hb = r(B, C, dtype=f32), e(B, C)
        add(f"norm + residual + norm, {B} rows", _time_chain([lambda: K.layer_norm_residual(None, out, 0, wn, xf, wn, 1e-6, C, hb) for _ in range(L)]),
            nbytes=B * C * (8 + 4 + 2.0), like=f"row{B}")
        wg, ab = [r(2 * ff, C) for _ in range(L)], e(B, ff)
        add(f"gate and up with activation, {B} rows", _time_chain([lambda a=a: K.gemv_relu_glu(xb, a, ab) for a in wg]), nbytes=2.0 * 2 * ff * C, like=f"gemv{B}")
        wdn = [r(C, ff) for _ in range(L)]
        add(f"down projection, {B} rows", _time_chain([lambda a=a: K.gemv_plain(ab, a, out) for a in wdn]), nbytes=2.0 * ff * C, like=f"gemv{B}")
    sv.check_status()
    nat.check_status()
    return rows


SERVE = {"Lupodra": bench_serve, "Safepel": bench_recurrent}


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("op", choices=["gemm", "attn_fwd", "attn_bwd", "sweep", "serve"])
    ap.add_argument("--model", default="Lupodra", choices=sorted(SERVE), help="serve: whose kernels")
    ap.add_argument("--m", type=int, default=32768)
    ap.add_argument("--n", type=int, default=4992)
    ap.add_argument("--k", type=int, default=1664)
    ap.add_argument("--bn", type=int, default=0, help="N tile (0 = heuristic)")
    ap.add_argument("--layout", default="fwd", choices=["fwd", "dgrad", "wgrad"])
    ap.add_argument("--dtype", default="bf16", choices=["bf16", "fp8", "mxfp8"], help="GEMM operand type")
    ap.add_argument("--pair", type=int, default=-1, help="GEMM: 1 = CTA-pair kernel, 0 = single-CTA kernel, -1 = library choice")
    ap.add_argument("--epi", default="linear", choices=["linear", "relu2", "mul2sqrt", "relu", "mulaux", "residual"], help="GEMM (fp8 / --pair): fused epilogue")
    ap.add_argument("--amax", type=int, default=0, help="GEMM (fp8 / --pair): 1 = the epilogue also reports max|output|")
    ap.add_argument("--batch", type=int, default=16)
    ap.add_argument("--seq", type=int, default=2048)
    ap.add_argument("--heads", type=int, default=13)
    ap.add_argument("--window", type=int, default=-1)
    ap.add_argument("--iters", type=int, default=10)
    ap.add_argument("--warmup", type=int, default=3)
    args = ap.parse_args()
    from nanochat_b200.ops import native as nat
    torch.manual_seed(0)
    if args.op == "serve":
        for row in SERVE[args.model]():
            print(json.dumps(row))
        return
    res = {"gemm": bench_gemm, "attn_fwd": bench_attn_fwd, "attn_bwd": bench_attn_bwd, "sweep": bench_sweep}[args.op](args, nat)
    nat.check_status()
    if os.path.exists("MEASURED_PEAKS.json"):
        with open("MEASURED_PEAKS.json") as f:
            peak = json.load(f).get("bf16_tflops")
        if peak and "tflops" in res:
            res["frac_of_measured_bf16_peak"] = res["tflops"] / peak
    print(json.dumps(res))


if __name__ == "__main__":
    main()
