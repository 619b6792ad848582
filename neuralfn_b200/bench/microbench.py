"""Isolated kernel timing harness (CUDA events, L2 flushed between iterations).

    python -m neuralfn_b200.bench.microbench gemm --m 16384 --n 2304 --k 768
    python -m neuralfn_b200.bench.microbench attention_fwd --batch 16 --heads 12 --seq 1024 --head-dim 64
    python -m neuralfn_b200.bench.microbench all            # the shapes of the GPT-2 124M step

Each case prints one JSON line: median milliseconds over ``--iters`` timed launches (after
``--warmup``), achieved TFLOP/s or GB/s from the algorithmic work, and - when ``--peak-tflops``
/ ``--peak-gbs`` are given - the fraction of that peak. Counterpart of the reference's
``linear_backward_bench.cpp`` / ``lm_head_backward_bench.cpp`` harnesses.
"""
from __future__ import annotations

import argparse
import json
import statistics
import sys

import torch


def _flush_buffer(dev):
    return torch.empty(192 * 1024 * 1024, dtype=torch.uint8, device=dev)  # larger than the 126 MB L2


def time_kernel(fn, iters: int, warmup: int, flush) -> float:
    for _ in range(max(3, warmup)):
        fn()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        flush.zero_()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        fn()
        stop.record()
        torch.cuda.synchronize()
        times.append(start.elapsed_time(stop))
    return statistics.median(times)


def _report(name, ms, *, flops=0.0, bytes_=0.0, args=None, extra=None):
    out = {"kernel": name, "ms": round(ms, 5)}
    if flops:
        out["tflops"] = round(flops / ms / 1e9, 2)
        if args.peak_tflops:
            out["frac_of_peak_tflops"] = round(out["tflops"] / args.peak_tflops, 3)
    if bytes_:
        out["gbs"] = round(bytes_ / ms / 1e6, 1)
        if args.peak_gbs:
            out["frac_of_peak_gbs"] = round(out["gbs"] / args.peak_gbs, 3)
    out.update(extra or {})
    print(json.dumps(out), flush=True)
    return out


def case_gemm(args, m=None, n=None, k=None, a_mn=False, b_mn=False, tag="gemm"):
    from neuralfn_b200.ops.gemm import gemm
    dev = torch.device("cuda")
    m, n, k = m or args.m, n or args.n, k or args.k
    a = torch.randn((k, m) if a_mn else (m, k), device=dev).bfloat16()
    b = torch.randn((k, n) if b_mn else (n, k), device=dev).bfloat16()
    out = torch.empty(m, n, device=dev, dtype=torch.bfloat16)
    ws = torch.empty(32 * 1024 * 1024, device=dev, dtype=torch.float32) if (a_mn or m <= 256) else None  # split-K: weight gradients, skinny decode products
    if getattr(args, "skinny_impl", -1) >= 0:
        from neuralfn_b200.ops import _lib
        _lib.load().nfn_gemm_skinny_set_impl(int(args.skinny_impl))
    ms = time_kernel(lambda: gemm(a, b, a_mn=a_mn, b_mn=b_mn, out=out, workspace=ws), args.iters, args.warmup, args.flush)
    return _report(tag, ms, flops=2.0 * m * n * k, bytes_=2.0 * (m * k + n * k + m * n), args=args,
                   extra={"m": m, "n": n, "k": k, "a_mn": a_mn, "b_mn": b_mn})


def case_skinny(args):
    """Decode-sized products of a Glimmer 29B layer at TP 4 (32 rows): the mma.sync weight-streaming kernel against the tcgen05
    split-K path, as fractions of the copy bandwidth."""
    from neuralfn_b200.ops import _lib
    from neuralfn_b200.ops.gemm import gemm
    dev = torch.device("cuda")
    L = _lib.load()
    ws = torch.empty(32 * 1024 * 1024, device=dev, dtype=torch.float32)
    out = []
    for m, n, k in ((32, 2304, 6656), (32, 6656, 1024), (32, 12288, 6656), (32, 6656, 6144), (8, 12288, 6656), (64, 12288, 6656), (32, 4096, 4096)):
        a = torch.randn(m, k, device=dev).bfloat16()
        w = torch.randn(n, k, device=dev).bfloat16()
        c = torch.empty(m, n, device=dev, dtype=torch.bfloat16)
        for impl in ((3, 2, 0) if m <= 32 else (2, 0)):
            old = L.nfn_gemm_skinny_set_impl(impl)
            ms = time_kernel(lambda: gemm(a, w, out=c, workspace=ws), args.iters, args.warmup, args.flush)  # L2 flushed between calls
            L.nfn_gemm_skinny_set_impl(old)
            out.append(_report({3: "skinny_mma_resident_cluster", 2: "skinny_mma", 0: "skinny_tcgen05_splitk"}[impl], ms, flops=2.0 * m * n * k, bytes_=2.0 * (n * k + m * k + m * n), args=args,
                               extra={"m": m, "n": n, "k": k}))
    return out


def case_grouped_k(args):
    """Weight gradients of all experts of an MoE layer (d = --k columns of the token buffer, hidden --n, --experts experts, --m rows
    in the expert-sorted buffer, split unevenly): one grouped launch against one TN GEMM per expert."""
    from neuralfn_b200.ops.gemm import gemm, gemm_grouped_k
    dev = torch.device("cuda")
    E, rows_total, d, h = args.experts, args.m, args.k, args.n
    g = torch.Generator(device=dev).manual_seed(0)
    w = torch.rand(E, device=dev, generator=g) + 0.2
    counts = (w / w.sum() * rows_total * 0.97).int().tolist()
    offs = [0]
    for c in counts:
        offs.append(offs[-1] + (c + 127) // 128 * 128)
    xs = torch.zeros(offs[-1], d, device=dev, dtype=torch.bfloat16)
    dh = (torch.randn(offs[-1], h, device=dev, generator=g) * 0.1).bfloat16()
    for e, c in enumerate(counts):
        xs[offs[e]:offs[e] + c] = (torch.randn(c, d, device=dev, generator=g) * 0.1).bfloat16()
    group_rows = torch.tensor(offs, device=dev, dtype=torch.int32)
    dw = torch.empty(E, d, h, device=dev, dtype=torch.bfloat16)
    flops = 2.0 * sum(counts) * d * h

    def loop():
        for e, c in enumerate(counts):
            gemm(xs[offs[e]:offs[e] + c], dh[offs[e]:offs[e] + c], a_mn=True, b_mn=True, out=dw[e])
    extra = {"experts": E, "rows": offs[-1], "d": d, "h": h}
    out = [_report("grouped_k", time_kernel(lambda: gemm_grouped_k(xs, dh, group_rows, dw), args.iters, args.warmup, args.flush), flops=flops, args=args, extra=extra)]
    if not args.no_baseline:
        out.append(_report("per_expert_loop", time_kernel(loop, args.iters, args.warmup, args.flush), flops=flops, args=args, extra=extra))
    return out


def case_attention(args, backward=False):
    from neuralfn_b200.ops import kernels as K
    dev = torch.device("cuda")
    B, H, T, D = args.batch, args.heads, args.seq, args.head_dim
    Hkv = args.kv_heads or H
    q = torch.randn(B * T, H * D, device=dev).bfloat16()
    k = torch.randn(B * T, Hkv * D, device=dev).bfloat16()
    v = torch.randn(B * T, Hkv * D, device=dev).bfloat16()
    o, lse = K.attention_forward(q, k, v, B=B, T=T, n_q_heads=H, n_kv_heads=Hkv, head_dim=D, causal=True)
    flops = 4.0 * B * H * T * T * D / 2  # causal
    if not backward:
        ms = time_kernel(lambda: K.attention_forward(q, k, v, B=B, T=T, n_q_heads=H, n_kv_heads=Hkv, head_dim=D, causal=True, out=o, lse=lse),
                         args.iters, args.warmup, args.flush)
        return _report("attention_fwd", ms, flops=flops, args=args, extra={"B": B, "H": H, "Hkv": Hkv, "T": T, "D": D})
    do = torch.randn_like(o)
    dq, dk, dv = torch.empty_like(q), torch.empty_like(k), torch.empty_like(v)
    delta = torch.empty(B, H, T, device=dev)
    acc = torch.empty(B * T, H * D, device=dev)
    ms = time_kernel(lambda: K.attention_backward(do, q, k, v, o, lse, B=B, T=T, n_q_heads=H, n_kv_heads=Hkv, head_dim=D, causal=True,
                                                  dq=dq, dk=dk, dv=dv, delta=delta, dq_accum=acc), args.iters, args.warmup, args.flush)
    return _report("attention_bwd", ms, flops=2.5 * flops, args=args, extra={"B": B, "H": H, "Hkv": Hkv, "T": T, "D": D})


def case_cross_entropy(args):
    from neuralfn_b200.ops import kernels as K
    dev = torch.device("cuda")
    rows, V = args.batch * args.seq, args.vocab
    Vp = (V + 127) // 128 * 128
    src = torch.randn(rows, Vp, device=dev).bfloat16()
    logits = torch.empty_like(src)
    tgt = torch.randint(0, V, (rows,), device=dev, dtype=torch.int32)
    row_loss, mean = torch.empty(rows, device=dev), torch.zeros(1, device=dev)

    def run():
        logits.copy_(src)  # the kernel overwrites logits with gradients
        K.cross_entropy(logits, tgt, vocab=V, cap=30.0, z_coef=1e-4, grad_scale=1.0 / rows, loss_scale=1.0 / rows, write_grad=True,
                        row_loss=row_loss, mean_loss=mean)

    copy_ms = time_kernel(lambda: logits.copy_(src), args.iters, args.warmup, args.flush)
    ms = time_kernel(run, args.iters, args.warmup, args.flush) - copy_ms
    return _report("cross_entropy_fwd_bwd", ms, bytes_=2.0 * rows * Vp * 2, args=args, extra={"rows": rows, "vocab": V})


def case_norm(args):
    from neuralfn_b200.ops import kernels as K
    dev = torch.device("cuda")
    rows, C = args.batch * args.seq, args.k
    x = torch.randn(rows, C, device=dev).bfloat16()
    w, b = torch.ones(C, device=dev).bfloat16(), torch.zeros(C, device=dev).bfloat16()
    y, mean, rstd = torch.empty_like(x), torch.empty(rows, device=dev), torch.empty(rows, device=dev)
    ms = time_kernel(lambda: K.norm_forward(x, w, b, eps=1e-5, mode=K.NORM_LAYER, out=y, mean=mean, rstd=rstd), args.iters, args.warmup, args.flush)
    return _report("layernorm_fwd", ms, bytes_=2.0 * rows * C * 2, args=args, extra={"rows": rows, "C": C})


def case_adamw(args):
    from neuralfn_b200.ops import kernels as K
    dev = torch.device("cuda")
    n = args.params
    master, m, v = (torch.zeros(n, device=dev) for _ in range(3))
    grads = torch.randn(n, device=dev).bfloat16()
    params = torch.empty(n, device=dev, dtype=torch.bfloat16)
    hyper = torch.zeros(K.HYPER_SIZE, device=dev)
    hyper[K.HP_LR], hyper[K.HP_BETA1], hyper[K.HP_BETA2], hyper[K.HP_EPS] = 1e-3, 0.9, 0.95, 1e-8
    hyper[K.HP_BC1], hyper[K.HP_BC2], hyper[K.HP_GRAD_SCALE], hyper[K.HP_MAX_NORM] = 0.1, 0.05, 1.0, 0.0
    clip = torch.ones(2, device=dev)
    ms = time_kernel(lambda: K.adamw_flat(master, m, v, grads, params, n, hyper, clip), args.iters, args.warmup, args.flush)
    return _report("adamw_flat", ms, bytes_=n * (3 * 4 * 2 + 2 + 2.0), args=args, extra={"params": n})


def case_decode_attention(args):
    from neuralfn_b200.ops import infer as I
    dev = torch.device("cuda")
    B, Hq, Hkv, D, ctx = args.batch, args.heads, args.kv_heads or 1, args.head_dim, args.seq
    kc = torch.randn(B, Hkv, ctx, D, device=dev).bfloat16()
    vc = torch.randn(B, Hkv, ctx, D, device=dev).bfloat16()
    qkv = torch.randn(B, (Hq + 2 * Hkv) * D, device=dev).bfloat16()
    lengths = torch.full((B,), ctx, dtype=torch.int32, device=dev)
    ws = I.DecodeAttentionWorkspace(B, Hq, Hkv, D, dev)
    cos, sin = I.rope_tables(ctx, D, device=dev)
    out = torch.empty(B, Hq * D, device=dev, dtype=torch.bfloat16)
    ms = time_kernel(lambda: I.decode_attention(qkv, kc, vc, lengths, n_q_heads=Hq, n_kv_heads=Hkv, head_dim=D, workspace=ws, cos=cos,
                                                sin=sin, qk_norm=True, out=out), args.iters, args.warmup, args.flush)
    return _report("decode_attention", ms, bytes_=2.0 * B * Hkv * ctx * D * 2, args=args, extra={"B": B, "Hq": Hq, "Hkv": Hkv, "ctx": ctx, "D": D})


def case_kquant_gemv(args):
    from neuralfn_b200.ops import infer as I
    from neuralfn_b200.quant import kquant
    dev = torch.device("cuda")
    N, Kd, B = args.n, args.k, min(args.batch, 8)
    raw = torch.from_numpy(kquant.random_blocks(12, N * Kd // 256, seed=0)).to(dev).reshape(-1)
    x = torch.randn(B, Kd, device=dev).bfloat16()
    out = torch.empty(B, N, device=dev, dtype=torch.bfloat16)
    ms = time_kernel(lambda: I.kquant_gemv(12, raw, x, N, out=out), args.iters, args.warmup, args.flush)
    return _report("q4_k_gemv", ms, bytes_=float(raw.numel()), flops=2.0 * B * N * Kd, args=args, extra={"B": B, "N": N, "K": Kd})



def case_gemm_kquant(args):
    """Prefill product over Q4_K weights, dequantisation fused into the GEMM pipeline, against the
    two-step path (dequantise to bf16, then the bf16 GEMM)."""
    from neuralfn_b200.ops import infer as I
    from neuralfn_b200.ops.gemm import gemm
    from neuralfn_b200.quant import kquant
    dev = torch.device("cuda")
    M, N, Kd = args.m, args.n, args.k
    raw = torch.from_numpy(kquant.random_blocks(12, N * Kd // 256, seed=0)).to(dev).reshape(-1)
    x = torch.randn(M, Kd, device=dev).bfloat16()
    out = torch.empty(M, N, device=dev, dtype=torch.bfloat16)
    wbuf = torch.empty(N * Kd, device=dev, dtype=torch.bfloat16)
    ms = time_kernel(lambda: I.gemm_kquant(12, x, raw, N, out=out), args.iters, args.warmup, args.flush)
    two = time_kernel(lambda: gemm(x, I.dequant_kquant(12, raw, out=wbuf).view(N, Kd), out=out), args.iters, args.warmup, args.flush)
    return _report("q4_k_gemm_fused_dequant", ms, bytes_=float(raw.numel()) + 2.0 * M * (Kd + N), flops=2.0 * M * N * Kd, args=args,
                   extra={"m": M, "n": N, "k": Kd, "two_step_ms": round(two, 5)})


def case_block_attention(args):
    """Speculative verification block (16 rows per sequence) against a bf16 KV cache."""
    from neuralfn_b200.ops import infer as I
    dev = torch.device("cuda")
    B, Hq, Hkv, D, ctx, R = args.batch, args.heads, args.kv_heads or 1, args.head_dim, args.seq, 16
    kc = torch.randn(B, Hkv, ctx + 128, D, device=dev).bfloat16()
    vc = torch.randn(B, Hkv, ctx + 128, D, device=dev).bfloat16()
    qkv = torch.randn(B * R, (Hq + 2 * Hkv) * D, device=dev).bfloat16()
    lengths = torch.full((B,), ctx, dtype=torch.int32, device=dev)
    ws = I.BlockAttentionWorkspace(B, R, Hq, Hkv, D, dev)
    out = torch.empty(B * R, Hq * D, device=dev, dtype=torch.bfloat16)
    ms = time_kernel(lambda: I.block_attention(qkv, kc, vc, lengths, rows=R, n_q_heads=Hq, n_kv_heads=Hkv, head_dim=D, workspace=ws, out=out),
                     args.iters, args.warmup, args.flush)
    return _report("block_attention_16_rows", ms, bytes_=2.0 * B * Hkv * ctx * D * 2, flops=4.0 * B * Hq * R * ctx * D, args=args,
                   extra={"B": B, "Hq": Hq, "Hkv": Hkv, "ctx": ctx, "D": D, "rows": R})


def case_turboquant_attention(args):
    """Decode attention over TurboQuant records (3.5 bits per coordinate)."""
    from neuralfn_b200.quant.turboquant import TurboQuantCodec, TurboQuantKVCache, default_outlier_indices
    dev = torch.device("cuda")
    B, Hq, Hkv, D, ctx = args.batch, args.heads, args.kv_heads or 1, args.head_dim, args.seq
    codec = TurboQuantCodec(D, profile="mse-3.5", seed=0, outlier_indices=default_outlier_indices(D))
    cache = TurboQuantKVCache(codec, B, Hkv, ctx, dev)
    cache.k.copy_(torch.randint(0, 255, cache.k.shape, dtype=torch.uint8, device=dev))
    cache.v.copy_(torch.randint(0, 255, cache.v.shape, dtype=torch.uint8, device=dev))
    cache.k.view(torch.float32)[..., 0] = 1.0  # finite norms
    cache.v.view(torch.float32)[..., 0] = 1.0
    cache._len_host = [ctx] * B
    cache.lengths.fill_(ctx)
    q = torch.randn(B, Hq * D, device=dev).bfloat16()
    ms = time_kernel(lambda: cache.attention(q, Hq), args.iters, args.warmup, args.flush)
    return _report("turboquant_decode_attention", ms, bytes_=float(B * ctx * cache.bytes_per_token), args=args,
                   extra={"B": B, "Hq": Hq, "Hkv": Hkv, "ctx": ctx, "D": D, "bytes_per_token": cache.bytes_per_token})



def case_engine_decode(args):
    """Resident-engine decode throughput on Llama-3-8B layer shapes (8 of the 32 layers, so that the
    weights stay a few GB): tokens/s for the whole batch and the weight bytes streamed per second."""
    import time

    from neuralfn_b200.serving import EngineConfig, ResidentEngine
    L, d, Hq, Hkv, hd, F, V = 8, 4096, 32, 8, 128, 14336, 32000
    B, ctx = max(1, args.batch), args.seq
    cfg = EngineConfig(family=1, n_layer=L, d_model=d, n_head=Hq, n_kv_head=Hkv, head_dim=hd, d_ff=F, vocab=V, padded_vocab=V,
                       max_seq=ctx + 80, max_batch=B, qk_norm=0, rope_hf=1, rope_theta=500000.0, norm_eps=1e-5, tie_embeddings=0)
    eng = ResidentEngine(cfg)
    g = torch.Generator().manual_seed(0)
    w = {n: (torch.ones(k) if n.endswith("norm") else torch.randn(k, generator=g) * 0.02).bfloat16() for n, k in eng.expected_tensors().items()}
    eng.load_named_tensors(w)
    weight_bytes = 2 * sum(k for n, k in eng.expected_tensors().items() if n != "tok_embeddings")
    prompt = torch.randint(0, V, (ctx,), generator=g).tolist()
    last = {b: eng.prefill(b, prompt) for b in range(B)}
    for _ in range(8):
        last = eng.decode(last)
    torch.cuda.synchronize()
    steps = 48
    t0 = time.perf_counter()
    for _ in range(steps):
        last = eng.decode(last)
    torch.cuda.synchronize()
    dt = (time.perf_counter() - t0) / steps
    return _report("engine_decode_llama8b_shape_8_layers", dt * 1e3, bytes_=float(weight_bytes), args=args,
                   extra={"batch": B, "context": ctx, "tokens_per_second": round(B / dt, 1), "ms_per_step": round(dt * 1e3, 3),
                          "kernel_launches_per_step": eng.launches // (steps + 8 + B) if hasattr(eng, "launches") else None})


def case_paged(args):
    """Kernels of the layer-list engine beside their closest counterparts, at one layer of ``--heads`` / ``--kv-heads`` x ``--head-dim`` with
    ``--window``: prompt attention over pages (``--seq`` rows) against flash attention, decode attention (``--batch`` rows) against the ring
    cache kernel, the row mix against SwiGLU, the residual row pass against RMS norm + residual."""
    from neuralfn_b200.ops import infer as I, kernels as K, paged as P
    dev = torch.device("cuda")
    H, G, D, T, B, W = args.heads, args.kv_heads or args.heads, args.head_dim, args.seq, args.batch, args.window
    slopes = torch.tensor([2.0 ** (-8 * (h + 1) / H) for h in range(H)], device=dev)
    kw = dict(heads=H, window=W, scale=D ** -0.5, slopes=slopes)
    rand = lambda *s: torch.randn(*s, device=dev).bfloat16()  # noqa: E731
    extra = {"H": H, "G": G, "D": D, "window": W}
    t = lambda fn: time_kernel(fn, args.iters, args.warmup, args.flush)  # noqa: E731
    w = min(W or T, T)
    flops = 4.0 * H * D * (w * (w + 1) / 2 + (T - w) * w)
    c = P.PagedCache(1, T, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q, gate, out = rand(T, H * D), rand(T, H * D), torch.empty(T, H * D, device=dev, dtype=torch.bfloat16)
    step = P.tile_rows(c, H)
    tiles = torch.tensor([[r, min(step, T - r), 0, r] for r in range(0, T, step)], dtype=torch.int32, device=dev)
    _report("paged_attention_tiles", t(lambda: P.attention_tiles(c, q, tiles, out, gate=gate, **kw)), flops=flops, args=args, extra={**extra, "T": T})
    k, v = rand(T, G * D), rand(T, G * D)
    fa = dict(B=1, T=T, n_q_heads=H, n_kv_heads=G, head_dim=D, causal=True, window=W)
    o, lse = K.attention_forward(q, k, v, **fa)
    _report("attention_fwd", t(lambda: K.attention_forward(q, k, v, out=o, lse=lse, **fa)), flops=flops, args=args, extra={**extra, "T": T})
    F = args.n
    x = rand(T, 2 * H * D + 2 * G * D + 2 * F)
    ch = H * D + 2 * G * D
    conv, state = rand(4, ch), torch.zeros(2, 1, 3, ch, device=dev, dtype=torch.bfloat16)
    cat, rt = torch.empty(T, H * D + F, device=dev, dtype=torch.bfloat16), P.row_tiles([(0, 0, T, 0)], dev)
    _report("mix_rows", t(lambda: P.mix_rows(c, x, rt, q, cat[:, H * D:], heads=H, off_gate=ch + H * D, off_up=ch + H * D + F, ff=F, conv=conv, state=state, temp=(0.1, 1024))),
            bytes_=4.0 * T * ch + 6.0 * T * F, args=args, extra={**extra, "T": T, "ff": F, "taps": 4})
    gu = rand(T, 2 * F)
    ffo = torch.empty(T, F, device=dev, dtype=torch.bfloat16)
    _report("swiglu", t(lambda: I.swiglu_forward(gu, F, out=ffo)), bytes_=6.0 * T * F, args=args, extra={"T": T, "ff": F})
    C = args.k
    xs, y, h, wt = torch.randn(T, C, device=dev), rand(T, C), torch.empty(T, C, device=dev, dtype=torch.bfloat16), rand(C)
    _report("row_norm (fp32 residual)", t(lambda: P.row_norm(xs, wt, h, eps=1e-5, y=y, y_weight=wt, x_out=xs)), bytes_=12.0 * T * C, args=args, extra={"T": T, "width": C})
    del c, q, gate, out, k, v, x, gu
    ctx = args.context
    c = P.PagedCache(B, ctx, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q1, g1, o1 = rand(B, H * D), rand(B, H * D), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
    slot, pos = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
    seen = min(W or ctx, ctx)
    _report("paged_attention_rows", t(lambda: P.attention_rows(c, q1, slot, pos, o1, gate=g1, **kw)), bytes_=4.0 * B * G * seen * D, args=args,
            extra={**extra, "B": B, "context": ctx})
    kc, vc, ws = rand(B, G, seen, D), rand(B, G, seen, D), I.DecodeAttentionWorkspace(B, H, G, D, dev)
    qkv, lens, (cos, sin) = rand(B, (H + 2 * G) * D), torch.full((B,), seen, dtype=torch.int32, device=dev), I.rope_tables(seen, D, device=dev)
    _report("decode_attention", t(lambda: I.decode_attention(qkv, kc, vc, lens, n_q_heads=H, n_kv_heads=G, head_dim=D, workspace=ws, cos=cos, sin=sin, qk_norm=True, out=o1)),
            bytes_=4.0 * B * G * seen * D, args=args, extra={**extra, "B": B, "context": ctx})


def case_layered(args):
    """Kernels of delta-rule layers, streams and routed experts beside their closest counterparts, at one layer of ``--heads`` / ``--kv-heads`` x
    ``--head-dim``, width ``--k``, ``--experts`` experts of which four of ``--n`` / 4 are used, four streams, ``--window`` with four kept tokens."""
    from neuralfn_b200.ops import infer as I, kernels as K, layered as Y, paged as P
    from neuralfn_b200.ops.gemm import gemm
    from neuralfn_b200.ops.moe import MoEWorkspace, _grouped_gemm, moe_forward
    dev = torch.device("cuda")
    H, G, D, T, B, W, C, E = args.heads, args.kv_heads or args.heads, args.head_dim, args.seq, args.batch, args.window, args.k, args.experts
    F, S = args.n // 4, 4
    rand = lambda *s: torch.randn(*s, device=dev).bfloat16()  # noqa: E731
    t = lambda fn: time_kernel(fn, args.iters, args.warmup, args.flush)  # noqa: E731
    i32 = dict(dtype=torch.int32, device=dev)
    # attention with kept tokens, soft cap, sink
    w = min(W or T, T)
    flops = 4.0 * H * D * (w * (w + 1) / 2 + (T - w) * w)
    c = P.PagedCache(1, T, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q, out = rand(T, H * D), torch.empty(T, H * D, device=dev, dtype=torch.bfloat16)
    step = P.tile_rows(c, H)
    tiles = torch.tensor([[r, min(step, T - r), 0, r] for r in range(0, T, step)], **i32)
    kw = dict(heads=H, window=W, scale=D ** -0.5, keep_first=4 if W else 0, softcap=30.0, sink=True)
    _report("paged_attention_tiles (cap, kept, sink)", t(lambda: P.attention_tiles(c, q, tiles, out, **kw)), flops=flops, args=args, extra={"T": T, "window": W})
    k, v = rand(T, G * D), rand(T, G * D)
    fa = dict(B=1, T=T, n_q_heads=H, n_kv_heads=G, head_dim=D, causal=True, window=W)
    o, lse = K.attention_forward(q, k, v, **fa)
    _report("attention_fwd", t(lambda: K.attention_forward(q, k, v, out=o, lse=lse, **fa)), flops=flops, args=args, extra={"T": T, "window": W})
    ctx = args.context
    seen = min(W or ctx, ctx)
    c = P.PagedCache(B, ctx, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q1, o1 = rand(B, H * D), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
    slot, pos = torch.arange(B, **i32), torch.full((B,), ctx - 1, **i32)
    _report("paged_attention_rows (cap, kept, sink)", t(lambda: P.attention_rows(c, q1, slot, pos, o1, **kw)), bytes_=4.0 * B * G * seen * D, args=args, extra={"B": B, "context": ctx})
    kc, vc, ws = rand(B, G, seen, D), rand(B, G, seen, D), I.DecodeAttentionWorkspace(B, H, G, D, dev)
    qkv, lens, (cos, sin) = rand(B, (H + 2 * G) * D), torch.full((B,), seen, **i32), I.rope_tables(seen, D, device=dev)
    _report("decode_attention", t(lambda: I.decode_attention(qkv, kc, vc, lens, n_q_heads=H, n_kv_heads=G, head_dim=D, workspace=ws, cos=cos, sin=sin, qk_norm=True, out=o1)),
            bytes_=4.0 * B * G * seen * D, args=args, extra={"B": B, "context": ctx})
    del c, k, v, kc, vc, q, out, o
    # delta rule: prompt in chunks, decode rows
    a_log, dt = torch.full((H,), -1.0, device=dev).bfloat16(), torch.full((H * D,), -1.0, device=dev).bfloat16()

    def rule(rows, seqs, slots):
        x, beta, decay, st = rand(rows, 3 * H * D), rand(rows, H), torch.randn(rows, H * D, device=dev), torch.zeros(slots, H, D, D, device=dev)
        return dict(qkv=x, beta=beta, decay=decay, a_log=a_log, dt_bias=dt, state=st, seqs=torch.tensor(seqs, **i32), kv_heads=H, dim=D)

    r = rule(T, [[0, T, 0, 0]], 1)
    wsp = torch.empty(96 << 20, device=dev, dtype=torch.uint8)
    _report("delta_chunks", t(lambda: Y.delta_rule(**r, form="chunks", workspace=wsp)), flops=7.0 * T * H * D * D, bytes_=14.0 * T * H * D, args=args, extra={"T": T, "heads": H, "dim": D})
    orow, gate, nw = torch.randn(T, H * D, device=dev), rand(T, H * D), rand(D)
    _report("delta_out", t(lambda: Y.delta_out(orow, gate, nw, heads=H, vdim=D, eps=1e-5)), bytes_=8.0 * T * H * D, args=args, extra={"T": T})
    cc, cx, conv, hist = P.PagedCache(1, 64, 1, 16, 16, dev), rand(T, 3 * H * D), rand(4, 3 * H * D), torch.zeros(2, 1, 3, 3 * H * D, device=dev, dtype=torch.bfloat16)
    cc.dim, qo, rt = 3 * D, torch.empty(T, 3 * H * D, device=dev, dtype=torch.bfloat16), P.row_tiles([(0, 0, T, 0)], dev)
    _report("mix_rows (SiLU)", t(lambda: P.mix_rows(cc, cx, rt, qo, None, heads=H, own_kv=False, conv=conv, state=hist, conv_act=3)), bytes_=4.0 * T * 3 * H * D, args=args,
            extra={"T": T, "taps": 4})
    r1 = rule(B, [[b, 1, b, 7] for b in range(B)], B)
    _report("delta_rows", t(lambda: Y.delta_rule(**r1)), bytes_=8.0 * B * H * D * D, args=args, extra={"B": B})
    del r, r1, orow, gate, cx, qo
    # streams
    xs, y, h, wt = torch.randn(T, S, C, device=dev), rand(T, C), torch.empty(T, C, device=dev, dtype=torch.bfloat16), rand(C)
    mix, one = torch.eye(S, device=dev).bfloat16(), torch.ones(S, device=dev).bfloat16()
    sp = dict(width=C, streams=S, ld=C, f32=False, weight=wt, mix=mix, out=one, into=one)
    _report("stream_pass", t(lambda: Y.stream_pass(xs, h, rows=T, x_out=xs, y=y, **sp)), bytes_=T * C * (8.0 * S + 4), args=args, extra={"T": T, "width": C, "streams": S})
    x1 = torch.randn(T, C, device=dev)
    _report("row_norm (fp32 residual)", t(lambda: P.row_norm(x1, wt, h, eps=1e-5, y=y, y_weight=wt, x_out=x1)), bytes_=12.0 * T * C, args=args, extra={"T": T, "width": C})
    del xs, x1
    # experts: prompt (grouped products), decode rows
    wg, wd, wr = rand(E, 2 * F, C) * C ** -0.5, rand(E, C, F) * F ** -0.5, rand(E, C) * C ** -0.5
    mw = MoEWorkspace(T, E, 4, C, F, dev)
    moe_forward(y, wr, wg, wd, 4, mw, score_fn="sigmoid", norm_topk=False)
    _report("grouped gemm (gate and up)", t(lambda: _grouped_gemm(mw.xs, wg, mw.h, mw)), flops=2.0 * 4 * T * 2 * F * C, args=args, extra={"T": T, "experts": E, "ff": F})
    wide, dense = rand(8 * F, C), torch.empty(T, 8 * F, device=dev, dtype=torch.bfloat16)
    _report("gemm (dense, same flops)", t(lambda: gemm(y, wide, out=dense)), flops=2.0 * T * 8 * F * C, args=args, extra={"T": T})
    y1 = rand(B, C)
    z = torch.randn(B, E, device=dev)
    idx, _, _ = Y.expert_rows(y1, z, wg, wd, experts=E, top=4)
    live = int(idx.unique().numel())
    _report("expert_rows (routing and products)", t(lambda: Y.expert_rows(y1, z, wg, wd, experts=E, top=4)), bytes_=2.0 * live * 3 * F * C, args=args, extra={"B": B, "experts_used": live})
    _report("gemm (dense, batch rows)", t(lambda: gemm(y1, wide, out=dense[:B])), bytes_=2.0 * 8 * F * C, args=args, extra={"B": B})


def case_mixers(args):
    """Kernels of rotated chunk attention, latent attention, time mixing, output norms and plain experts beside their closest counterparts, at one layer of
    ``--heads`` / ``--kv-heads`` x ``--head-dim``, width ``--k``: chunks of 1.5 x ``--window`` (queries in the middle of one), latents of 512 + 64 channels with
    ``--window``, ``--experts`` experts of which four of ``--n`` / 4 are used beside a shared one of ``--n`` / 2."""
    from neuralfn_b200.ops import infer as I, kernels as K, layered as Y, paged as P
    from neuralfn_b200.ops.gemm import gemm
    from neuralfn_b200.ops.moe import MoEWorkspace, _grouped_gemm, moe_forward
    dev = torch.device("cuda")
    H, G, D, T, B, W, C, E = args.heads, args.kv_heads or args.heads, args.head_dim, args.seq, args.batch, args.window, args.k, args.experts
    F, R, RANK, HD, chunk = args.n // 4, 64, 512, args.heads * args.head_dim, W + W // 2
    rand = lambda *s: torch.randn(*s, device=dev).bfloat16()  # noqa: E731
    t = lambda fn: time_kernel(fn, args.iters, args.warmup, args.flush)  # noqa: E731
    i32 = dict(dtype=torch.int32, device=dev)
    rep = lambda name, fn, **kw: _report(name, t(fn), args=args, **kw)  # noqa: E731
    w = min(W, T)
    win_keys = w * (w + 1) / 2 + (T - w) * w
    chunk_keys = sum(min(chunk, T - a) * (min(chunk, T - a) + 1) / 2 for a in range(0, T, chunk))

    def tile_list(step):
        return torch.tensor([[r, min(step, T - r), 0, r] for r in range(0, T, step)], **i32)

    # ---- prompt attention ----
    c = P.PagedCache(1, T, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q, out, tiles, kw = rand(T, HD), torch.empty(T, HD, device=dev, dtype=torch.bfloat16), tile_list(P.tile_rows(c, H)), dict(heads=H, scale=D ** -0.5)
    rep("paged_attention_tiles (chunk)", lambda: P.attention_tiles(c, q, tiles, out, chunk=chunk, **kw), flops=4.0 * HD * chunk_keys, extra={"T": T, "chunk": chunk})
    k, v = rand(T, G * D), rand(T, G * D)
    fa = dict(B=1, T=T, n_q_heads=H, n_kv_heads=G, head_dim=D, causal=True, window=W)
    o, lse = K.attention_forward(q, k, v, **fa)
    rep("attention_fwd", lambda: K.attention_forward(q, k, v, out=o, lse=lse, **fa), flops=4.0 * HD * win_keys, extra={"T": T, "window": W})
    lc = Y.LatentCache(1, T, RANK, R, dev)
    lc.k.normal_()
    ql, x, ltiles, base = rand(T, H * (D + R)), rand(T, 2 * HD), tile_list(128), torch.zeros(1, **i32)
    rep("latent_attention_tiles", lambda: Y.latent_attention_tiles(lc, ql, x, base, ltiles, out, heads=H, dim=D, vdim=D, window=W, scale=(D + R) ** -0.5),
        flops=2.0 * H * (2 * D + R) * win_keys, extra={"T": T, "window": W})
    spans, lat, wkvx = torch.tensor([[0, 0, T // 64, 0]], **i32), torch.empty(T, RANK, device=dev, dtype=torch.bfloat16), rand(2 * HD, RANK)
    rep("latent_gather", lambda: Y.latent_gather(lc, spans, lat, T // 64), bytes_=4.0 * T * RANK, extra={"T": T})
    rep("gemm (expansion)", lambda: gemm(lat, wkvx, out=x), flops=4.0 * T * HD * RANK, extra={"T": T})
    # ---- rows between products and attention ----
    rt, freq, wn = P.row_tiles([(0, 0, T, 0)], dev), Y.frequencies(R, 1e4, dev), rand(D)
    hx = rand(T, (H + G) * D)
    rep("head_rows", lambda: Y.head_rows(c, hx, rt, hx, heads=H, dim=D, freq=freq, rot_dims=R, eps=1e-5, q_norm=wn, k_norm=wn, key_values=True), bytes_=2.0 * T * D * (2 * H + 3 * G), extra={"T": T})
    lx = rand(T, H * (D + R) + RANK + R)
    cn = rand(RANK)
    rep("latent_rows", lambda: Y.latent_rows(lc, lx, rt, heads=H, dim=D, rot_dim=R, rank=RANK, c_norm=cn, eps=1e-5, freq=freq), bytes_=4.0 * T * (H * R + RANK + R), extra={"T": T})
    mx, mq = rand(T, (H + 2 * G) * D + 2 * 4 * F), torch.empty(T, HD, device=dev, dtype=torch.bfloat16)
    cat = torch.empty(T, 4 * F, device=dev, dtype=torch.bfloat16)
    rep("mix_rows (no convolution)", lambda: P.mix_rows(c, mx, rt, mq, None, heads=H), bytes_=4.0 * T * (H + 2 * G) * D, extra={"T": T})
    rep("ff_rows", lambda: Y.ff_rows(mx, cat, off_gate=0, off_up=4 * F, act=3), bytes_=6.0 * T * 4 * F, extra={"T": T, "ff": 4 * F})
    del c, k, v, q, o, mx, mq, cat, hx, lx, ql, x, lc
    # ---- decode attention ----
    seen, pos1 = W, chunk + W - 1
    c = P.PagedCache(B, pos1 + 1, G, D, D, dev)
    c.k.normal_(), c.v.normal_()
    q1, o1, slot, pos = rand(B, HD), torch.empty(B, HD, device=dev, dtype=torch.bfloat16), torch.arange(B, **i32), torch.full((B,), pos1, **i32)
    rep("paged_attention_rows (chunk)", lambda: P.attention_rows(c, q1, slot, pos, o1, chunk=chunk, **kw), bytes_=4.0 * B * G * seen * D, extra={"B": B, "keys": seen})
    kc, vc, ws = rand(B, G, seen, D), rand(B, G, seen, D), I.DecodeAttentionWorkspace(B, H, G, D, dev)
    qkv, lens, (cos, sin) = rand(B, (H + 2 * G) * D), torch.full((B,), seen, **i32), I.rope_tables(seen, D, device=dev)
    rep("decode_attention", lambda: I.decode_attention(qkv, kc, vc, lens, n_q_heads=H, n_kv_heads=G, head_dim=D, workspace=ws, cos=cos, sin=sin, qk_norm=True, out=o1),
        bytes_=4.0 * B * G * seen * D, extra={"B": B, "keys": seen})
    lc = Y.LatentCache(B, pos1 + 1, RANK, R, dev)
    lc.k.normal_()
    qa, oa = rand(B, H, RANK + R), torch.empty(B, H, RANK, device=dev, dtype=torch.bfloat16)
    rep("latent_attention_rows", lambda: Y.latent_attention_rows(lc, qa.view(B, -1), slot, pos, oa.view(B, -1), heads=H, window=W, scale=(D + R) ** -0.5),
        bytes_=2.0 * B * seen * (RANK + R), flops=2.0 * B * H * seen * (2 * RANK + R), extra={"B": B, "keys": seen})
    wut, wuv, ov = rand(H, RANK, D), rand(H, D, RANK), torch.empty(B, H, D, device=dev, dtype=torch.bfloat16)
    qn = rand(B, H, D + R)
    rep("group_products (keys)", lambda: Y.group_products(qn[..., :D], wut, qa), bytes_=2.0 * (H * RANK * D + B * H * (RANK + D)), extra={"B": B})
    rep("group_products (values)", lambda: Y.group_products(oa, wuv, ov), bytes_=2.0 * (H * RANK * D + B * H * (RANK + D)), extra={"B": B})
    w4, x4, y4 = rand(4, HD, C), rand(4, B, C), torch.empty(B, 4, HD, device=dev, dtype=torch.bfloat16)
    for b in sorted({1, min(8, B), min(16, B), B}):
        rep("group_products (r, k, v, gate)", lambda: Y.group_products(x4[:, :b].transpose(0, 1), w4, y4[:b]), bytes_=8.0 * HD * C, extra={"B": b})
        rep("gemm (one after another)", lambda: [gemm(x4[i, :b], w4[i], out=y4.view(4, B, HD)[i, :b]) for i in range(4)], bytes_=8.0 * HD * C, extra={"B": b})
        rep("gemm (same bytes)", lambda: gemm(x4[0, :b], w4.view(4 * HD, C), out=y4.view(B, 4 * HD)[:b]), bytes_=8.0 * HD * C, extra={"B": b})
    del c, kc, vc, lc, w4
    # ---- time mixing ----
    u, w0 = rand(HD), torch.full((HD,), -1.0, device=dev).bfloat16()

    def rule(rows, seqs, slots):
        return dict(rkv=rand(rows, 4 * HD), z=torch.randn(rows, HD, device=dev), w0=w0, u=u, state=torch.zeros(slots, H, D, D, device=dev), seqs=torch.tensor(seqs, **i32), dim=D)

    r, wsp = rule(T, [[0, T, 0, 0]], 1), torch.empty(96 << 20, device=dev, dtype=torch.uint8)
    rep("wkv_chunks", lambda: Y.wkv_rule(**r, form="chunks", workspace=wsp), bytes_=14.0 * T * HD, extra={"T": T, "heads": H, "dim": D})
    dt, a_log = w0, torch.full((H,), -1.0, device=dev).bfloat16()
    dr = dict(qkv=rand(T, 3 * HD), beta=rand(T, H), decay=torch.randn(T, HD, device=dev), a_log=a_log, dt_bias=dt, state=torch.zeros(1, H, D, D, device=dev), seqs=torch.tensor([[0, T, 0, 0]], **i32),
              kv_heads=H, dim=D)
    rep("delta_chunks", lambda: Y.delta_rule(**dr, form="chunks", workspace=wsp), bytes_=14.0 * T * HD, extra={"T": T, "heads": H, "dim": D})
    r1 = rule(B, [[b, 1, b, 7] for b in range(B)], B)
    rep("wkv_rows", lambda: Y.wkv_rule(**r1), bytes_=8.0 * B * HD * D, extra={"B": B})
    d1 = dict(qkv=rand(B, 3 * HD), beta=rand(B, H), decay=torch.randn(B, HD, device=dev), a_log=a_log, dt_bias=dt, state=torch.zeros(B, H, D, D, device=dev),
              seqs=torch.tensor([[b, 1, b, 7] for b in range(B)], **i32), kv_heads=H, dim=D)
    rep("delta_rows", lambda: Y.delta_rule(**d1), bytes_=8.0 * B * HD * D, extra={"B": B})
    low, w2, so, n1 = torch.randn(B, 64, device=dev), rand(HD, 128) * 0.1, torch.empty(B, HD, device=dev, dtype=torch.bfloat16), rand(HD)
    for b in sorted({1, min(8, B), B}):
        if b * H <= 4 * 148:
            st = P.row_tiles([(s, 7, 1, 0) for s in range(b)], dev)
            rep("wkv_step", lambda: Y.wkv_step(r1["rkv"][:b], low[:b], w2, w0, u, r1["state"], n1, so[:b], st, dim=D, eps=1e-5), bytes_=8.0 * b * HD * D, extra={"B": b})
    xs, mu, prev, sh = torch.randn(T, C, device=dev), rand(5, C), torch.zeros(2, 1, C, device=dev), torch.empty(5, T, C, device=dev, dtype=torch.bfloat16)
    rep("shift_rows", lambda: Y.shift_rows(xs, mu, prev, sh, rt), bytes_=14.0 * T * C, extra={"T": T, "width": C})
    del r, dr, d1, r1, sh
    # ---- residual, experts ----
    y, h, wt = rand(T, C), torch.empty(T, C, device=dev, dtype=torch.bfloat16), rand(C)
    rep("stream_pass (norm on the update)", lambda: Y.stream_pass(xs, h, width=C, streams=1, rows=T, ld=C, f32=False, x_out=xs, y=y, y_weight=wt, y_scale=0.5), bytes_=12.0 * T * C, extra={"T": T})
    rep("row_norm (fp32 residual)", lambda: P.row_norm(xs, wt, h, eps=1e-5, y=y, y_weight=wt, x_out=xs), bytes_=12.0 * T * C, extra={"T": T})
    ys, item, plus, order = rand(4 * T, C), torch.rand(4 * T, device=dev), rand(T, C), torch.randperm(4 * T, device=dev).int()
    rep("stream_pass (experts)", lambda: Y.stream_pass(xs, h, width=C, streams=1, rows=T, ld=C, f32=False, x_out=xs, y=ys, y_rows=4, y_index=order, y_item=item, y_plus=plus, y_weight=wt, y_scale=0.5),
        bytes_=20.0 * T * C, extra={"T": T})
    z, corr = torch.randn(T, E, device=dev), torch.zeros(E, device=dev).bfloat16()
    choice = dict(correction=corr, groups=8 if E % 8 == 0 else 0, keep=4, normalise=True, scale=1.5)
    rep("expert_choice", lambda: Y.expert_choice(z, 4, **choice), bytes_=4.0 * T * E + 32.0 * T, extra={"T": T})
    rep("expert_choice (no groups)", lambda: Y.expert_choice(z, 4), bytes_=4.0 * T * E + 32.0 * T, extra={"T": T})
    up, down, wr = rand(E, F, C) * C ** -0.5, rand(E, C, F) * F ** -0.5, rand(E, C) * C ** -0.5
    wg = rand(E, 2 * F, C) * C ** -0.5
    mw = MoEWorkspace(T, E, 4, C, F, dev)
    moe_forward(y, wr, wg, down, 4, mw, score_fn="sigmoid", norm_topk=False)
    rep("grouped gemm (gate and up)", lambda: _grouped_gemm(mw.xs, wg, mw.h, mw), flops=16.0 * T * F * C, extra={"T": T, "experts": E, "ff": F})
    mid = torch.empty(mw.xs.shape[0], F, device=dev, dtype=torch.bfloat16)
    rep("grouped gemm (up)", lambda: _grouped_gemm(mw.xs, up, mid, mw), flops=8.0 * T * F * C, extra={"T": T, "experts": E, "ff": F})
    y1, z1 = rand(B, C), torch.randn(B, E, device=dev)
    live = int(Y.expert_rows(y1, z1, up, down, experts=E, top=4, act=4, plain=True, **choice)[0].unique().numel())
    rep("expert_rows (plain)", lambda: Y.expert_rows(y1, z1, up, down, experts=E, top=4, act=4, plain=True, **choice), bytes_=4.0 * live * F * C, extra={"B": B, "experts_used": live})
    live = int(Y.expert_rows(y1, z1, wg, down, experts=E, top=4)[0].unique().numel())
    rep("expert_rows (gated)", lambda: Y.expert_rows(y1, z1, wg, down, experts=E, top=4), bytes_=6.0 * live * F * C, extra={"B": B, "experts_used": live})


def case_recurrences(args):
    """Linear attention with a decay per head, the gated recurrence, input convolutions, learned sinks, gates and clamped experts beside the like kernels of the other
    designs, at one layer of ``--heads`` x ``--head-dim`` (the gated recurrence as wide as all heads together), width ``--k``, ``--experts`` experts of which four of
    ``--n`` / 4 are used, latents of 512 + 64 channels over all earlier tokens."""
    from neuralfn_b200.ops import layered as Y, paged as P
    dev = torch.device("cuda")
    H, D, T, B, C, E = args.heads, args.head_dim, args.seq, args.batch, args.k, args.experts
    F, R, RANK, HD = args.n // 4, 64, 512, args.heads * args.head_dim
    rand = lambda *s: torch.randn(*s, device=dev).bfloat16()  # noqa: E731
    i32 = dict(dtype=torch.int32, device=dev)
    rep = lambda name, fn, **kw: _report(name, time_kernel(fn, args.iters, args.warmup, args.flush), args=args, **kw)  # noqa: E731
    one, pw = torch.tensor([[0, T, 0, 0]], **i32), Y.powers([1 - 2.0 ** (-1 - 9 * h / H) for h in range(H)], dev)
    rt, st = P.row_tiles([(0, 0, T, 0)], dev), P.row_tiles([(b, 7, 1, 0) for b in range(B)], dev)

    # ---- recurrences: prompts, then single tokens ----
    qkvg, state = rand(T, 4 * HD) * 0.1, torch.zeros(1, H, D, D, device=dev)
    lw = torch.empty(1, device=dev, dtype=torch.uint8)
    rep("linear_chunks", lambda: Y.linear_rule(qkvg, pw, state, one, form="chunks"), bytes_=10.0 * T * HD, extra={"T": T, "heads": H, "dim": D})
    rep("linear_chunks (no segments)", lambda: Y.linear_rule(qkvg, pw, state, one, form="chunks", workspace=lw), bytes_=10.0 * T * HD, extra={"T": T})
    u, w0, wn = rand(HD), torch.full((HD,), -1.0, device=dev).bfloat16(), rand(HD)
    z, wsp = torch.randn(T, HD, device=dev), torch.empty(96 << 20, device=dev, dtype=torch.uint8)
    rep("wkv_chunks", lambda: Y.wkv_rule(qkvg, z, w0, u, state, one, dim=D, form="chunks", workspace=wsp), bytes_=14.0 * T * HD, extra={"T": T})
    o, gate, out = torch.randn(T, HD, device=dev), rand(T, HD), torch.empty(T, HD, device=dev, dtype=torch.bfloat16)
    rep("row_out", lambda: Y.row_out(o, gate, wn, live=HD, eps=1e-5), bytes_=8.0 * T * HD, extra={"T": T})
    rep("delta_out (norm per head)", lambda: Y.delta_out(o, gate, wn[:D], heads=H, vdim=D, eps=1e-5), bytes_=8.0 * T * HD, extra={"T": T})
    gx, gs = rand(T, 3 * HD), torch.zeros(B, HD, device=dev)
    rep("gru_rows", lambda: Y.gru_rows(gx, gs, out, one, 0), bytes_=8.0 * T * HD, extra={"T": T, "width": HD})
    mb = min(8, B)
    parts = torch.tensor([[b * (T // mb), T // mb, b, 0] for b in range(mb)], **i32)
    rep("gru_rows (several prompts)", lambda: Y.gru_rows(gx, gs, out, parts, 0), bytes_=8.0 * T * HD, extra={"T": T // mb, "prompts": mb})
    for b in sorted({1, min(8, B), B}):
        states, so, cnt = torch.zeros(b, H, D, D, device=dev), torch.empty(b, HD, device=dev, dtype=torch.bfloat16), torch.zeros(b, **i32)
        low, w2 = torch.randn(b, 64, device=dev), rand(HD, 128) * 0.1
        rep("linear_step", lambda: Y.linear_step(qkvg[:b], pw, states, wn, so, st[:b], cnt, vdim=D, eps=1e-5), bytes_=8.0 * b * HD * D, extra={"B": b})
        rep("wkv_step", lambda: Y.wkv_step(qkvg[:b], low, w2, w0, u, states, wn, so, st[:b], dim=D, eps=1e-5), bytes_=8.0 * b * HD * D, extra={"B": b})
        seqs = torch.tensor([[i, 1, i, 7] for i in range(b)], **i32)
        rep("gru_rows (single tokens)", lambda: Y.gru_rows(gx[:b], gs, so, seqs, b), bytes_=16.0 * b * HD, extra={"B": b})
    # ---- residual and convolution on the way into a sublayer ----
    xs, y, h, hc, wt, g1 = torch.randn(T, C, device=dev), rand(T, C), torch.empty(T, C, device=dev, dtype=torch.bfloat16), torch.empty(T, C, device=dev, dtype=torch.bfloat16), rand(C), rand(1)
    conv, hist = rand(4, C), torch.zeros(2, B, 3, C, device=dev, dtype=torch.bfloat16)
    kw = dict(width=C, streams=1, ld=C, f32=False)
    rep("stream_pass (norms on both sides, one factor)", lambda: Y.stream_pass(xs, h, rows=T, x_out=xs, y=y, y_weight=g1, weight=g1, scalar_norms=True, **kw), bytes_=12.0 * T * C, extra={"T": T})
    rep("stream_pass (norm on the update)", lambda: Y.stream_pass(xs, h, rows=T, x_out=xs, y=y, y_weight=wt, **kw), bytes_=12.0 * T * C, extra={"T": T})
    rep("input_conv", lambda: Y.input_conv(h, conv, hist, hc, rt), bytes_=4.0 * T * C, extra={"T": T, "width": C})
    mu, prev, sh = rand(5, C), torch.zeros(2, 1, C, device=dev), torch.empty(5, T, C, device=dev, dtype=torch.bfloat16)
    rep("shift_rows", lambda: Y.shift_rows(xs, mu, prev, sh, rt), bytes_=14.0 * T * C, extra={"T": T, "width": C})
    del sh
    rep("stream_pass (with the convolution, single tokens)", lambda: Y.stream_pass(xs, h, rows=B, x_out=xs, y=y, y_weight=g1, weight=g1, scalar_norms=True, conv=conv, history=hist, tiles=st, **kw),
        bytes_=(12.0 + 12.0) * B * C, extra={"B": B})
    rep("stream_pass (single tokens)", lambda: Y.stream_pass(xs, h, rows=B, x_out=xs, y=y, y_weight=wt, **kw), bytes_=12.0 * B * C, extra={"B": B})
    # ---- latent attention: sinks, gate ----
    lc = Y.LatentCache(1, T, RANK, R, dev)
    lc.k.normal_()
    sinks, ql, x, base = rand(H), rand(T, H * (D + R)), rand(T, 2 * HD), torch.zeros(1, **i32)
    tiles = torch.tensor([[r, min(128, T - r), 0, r] for r in range(0, T, 128)], **i32)
    flops = 2.0 * H * (2 * D + R) * T * (T + 1) / 2
    la = dict(heads=H, dim=D, vdim=D, window=0, scale=(D + R) ** -0.5)
    rep("latent_attention_tiles (sinks, gate)", lambda: Y.latent_attention_tiles(lc, ql, x, base, tiles, out, sinks=sinks, gate=gate, **la), flops=flops, extra={"T": T})
    rep("latent_attention_tiles", lambda: Y.latent_attention_tiles(lc, ql, x, base, tiles, out, **la), flops=flops, extra={"T": T})
    del lc, x, ql
    keys = args.context
    lc = Y.LatentCache(B, keys, RANK, R, dev)
    lc.k.normal_()
    slot, pos = torch.arange(B, **i32), torch.full((B,), keys - 1, **i32)
    qa, oa = rand(B, H * (RANK + R)), torch.empty(B, H * RANK, device=dev, dtype=torch.bfloat16)
    for b in sorted({1, min(8, B), B}):
        lr = dict(heads=H, window=0, scale=(D + R) ** -0.5, max_keys=keys)
        rep("latent_attention_rows (sinks)", lambda: Y.latent_attention_rows(lc, qa[:b], slot[:b], pos[:b], oa[:b], sinks=sinks, **lr), bytes_=2.0 * b * keys * (RANK + R), extra={"B": b, "keys": keys})
        rep("latent_attention_rows", lambda: Y.latent_attention_rows(lc, qa[:b], slot[:b], pos[:b], oa[:b], **lr), bytes_=2.0 * b * keys * (RANK + R), extra={"B": b, "keys": keys})
    wuv, ov, gb = rand(H, D, RANK), torch.empty(B, H, D, device=dev, dtype=torch.bfloat16), rand(B, H, D)
    rep("group_products (values, gate)", lambda: Y.group_products(oa.view(B, H, RANK), wuv, ov, gate=gb), bytes_=2.0 * (HD * RANK + B * H * (RANK + 2 * D)), extra={"B": B})
    rep("group_products (values)", lambda: Y.group_products(oa.view(B, H, RANK), wuv, ov), bytes_=2.0 * (HD * RANK + B * H * (RANK + D)), extra={"B": B})
    # ---- feed-forward ----
    gu, mid, cl = rand(T, 8 * F), torch.empty(T, 4 * F, device=dev, dtype=torch.bfloat16), (7.0, 1.702, 1.0)
    rep("ff_rows (clamped)", lambda: Y.ff_rows(gu, mid, off_gate=0, off_up=4 * F, act=7, clamp=cl), bytes_=24.0 * T * F, extra={"T": T, "ff": 4 * F})
    rep("ff_rows", lambda: Y.ff_rows(gu, mid, off_gate=0, off_up=4 * F, act=3), bytes_=24.0 * T * F, extra={"T": T, "ff": 4 * F})
    del gu, mid
    zt = torch.randn(T, E, device=dev)
    rep("expert_choice (softmax)", lambda: Y.expert_choice(zt, 4, softmax=True), bytes_=4.0 * T * E + 32.0 * T, extra={"T": T})
    rep("expert_choice (no groups)", lambda: Y.expert_choice(zt, 4), bytes_=4.0 * T * E + 32.0 * T, extra={"T": T})
    wg, down = rand(E, 2 * F, C) * C ** -0.5, rand(E, C, F) * F ** -0.5
    y1, z1 = rand(B, C), torch.randn(B, E, device=dev)
    ex = dict(experts=E, top=4)
    live = int(Y.expert_rows(y1, z1, wg, down, **ex)[0].unique().numel())
    rep("expert_rows (clamped, softmax)", lambda: Y.expert_rows(y1, z1, wg, down, act=7, clamp=cl, weigh_output=True, softmax=True, **ex), bytes_=6.0 * live * F * C, extra={"B": B, "experts_used": live})
    rep("expert_rows (gated)", lambda: Y.expert_rows(y1, z1, wg, down, **ex), bytes_=6.0 * live * F * C, extra={"B": B, "experts_used": live})


CASES = {"gemm": case_gemm, "paged": case_paged, "layered": case_layered, "mixers": case_mixers, "recurrences": case_recurrences, "attention_fwd": case_attention, "attention_bwd": lambda a: case_attention(a, True),
         "cross_entropy": case_cross_entropy, "norm": case_norm, "adamw": case_adamw, "decode_attention": case_decode_attention,
         "skinny": case_skinny, "grouped_k": case_grouped_k, "kquant_gemv": case_kquant_gemv, "gemm_kquant": case_gemm_kquant, "block_attention": case_block_attention,
         "turboquant_attention": case_turboquant_attention, "engine_decode": case_engine_decode}


def run_all(args):
    M = 16 * 1024
    res = []
    for (n, k) in ((2304, 768), (768, 768), (3072, 768), (768, 3072), (50304, 768)):
        res.append(case_gemm(args, M, n, k, tag="gemm_fwd"))
    for (n, k) in ((768, 2304), (768, 3072), (3072, 768)):
        res.append(case_gemm(args, M, n, k, b_mn=True, tag="gemm_dx"))
    for (m, n) in ((2304, 768), (3072, 768), (768, 3072), (50304, 768)):
        res.append(case_gemm(args, m, n, M, a_mn=True, b_mn=True, tag="gemm_dw"))
    res.append(case_attention(args))
    res.append(case_attention(args, True))
    res.append(case_cross_entropy(args))
    res.append(case_norm(args))
    res.append(case_adamw(args))
    return res


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("case", choices=sorted(CASES) + ["all"])
    ap.add_argument("--m", type=int, default=16384)
    ap.add_argument("--n", type=int, default=2304)
    ap.add_argument("--k", type=int, default=768)
    ap.add_argument("--batch", type=int, default=16)
    ap.add_argument("--heads", type=int, default=12)
    ap.add_argument("--kv-heads", type=int, default=0)
    ap.add_argument("--seq", type=int, default=1024)
    ap.add_argument("--head-dim", type=int, default=64)
    ap.add_argument("--vocab", type=int, default=50257)
    ap.add_argument("--params", type=int, default=124 * 1000 * 1000)
    ap.add_argument("--window", type=int, default=0, help="paged case: sliding window")
    ap.add_argument("--context", type=int, default=4096, help="paged case: cached tokens per decode row")
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--experts", type=int, default=16, help="grouped_k and layered cases")
    ap.add_argument("--no-baseline", action="store_true", help="grouped_k case: skip the per-expert loop (profiler captures)")
    ap.add_argument("--skinny-impl", type=int, default=-1, help="gemm case: nfn_gemm_skinny_set_impl mode for products with 3 - 64 rows (-1: the default)")
    ap.add_argument("--warmup", type=int, default=5)
    ap.add_argument("--peak-tflops", type=float, default=0.0, help="measured bf16 GEMM peak to report fractions against")
    ap.add_argument("--peak-gbs", type=float, default=0.0, help="measured HBM copy bandwidth to report fractions against")
    args = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("microbench needs a CUDA device", file=sys.stderr)
        return 2
    args.flush = _flush_buffer(torch.device("cuda"))
    if args.case == "all":
        run_all(args)
    else:
        CASES[args.case](args)
    from neuralfn_b200.ops import _lib
    _lib.assert_status_ok("microbench")
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
