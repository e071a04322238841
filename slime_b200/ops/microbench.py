"""Kernel micro-benchmarks: ``python -m slime_b200.ops.microbench {gemm,decode,norm,...} [options]``.

Every number is a CUDA-event time on the launching stream after warm-up, median over ``--iters`` timed
repetitions with an L2 flush (a 256 MiB memset) between them. One JSON object per line on stdout.

    gemm    tcgen05 GEMM vs cuBLAS (torch.matmul) for forward / dgrad / wgrad layouts
    decode  each kernel of one rollout decode step at a given batch and context length
    norm    RMSNorm forward/backward bandwidth
    attn    flash attention forward / backward (own kernels; the flash-attn library on the same tensors for comparison)
    window  kernels of models with specified layers, each beside the like kernel of the existing models
    rules   kernels of Zetizen layers (capped, biased, chunked and latent attention, experts beside a mixer), likewise
    scan    kernels of Pebodra layers (linear recurrences, differential attention, grouped routing, norms in parts), likewise
    fused_emul  the peer-memory kernels (DP reduce / Adam, TP all-reduce + norm) with all ranks emulated on one GPU

``--small`` shrinks the working set to a case suitable for a profiler capture (a few launches, < 1 GB).
"""

from __future__ import annotations

import argparse
import json
import math
import os

import torch

from slime_b200 import ops
from slime_b200.ops import _lib

_FLUSH = None


def _flush_l2():
    global _FLUSH
    if _FLUSH is None:
        _FLUSH = torch.empty(256 * 1024 * 1024, dtype=torch.uint8, device="cuda")
    _FLUSH.zero_()


def time_ms(fn, iters: int = 20, warmup: int = 3, reps: int = 1, flush: bool = True) -> float:
    """Median device time of ``reps`` back-to-back calls of ``fn`` (divided by ``reps``)."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        if flush:
            _flush_l2()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record()
        for _ in range(reps):
            fn()
        e.record()
        torch.cuda.synchronize()
        times.append(s.elapsed_time(e) / reps)
    times.sort()
    return times[len(times) // 2]


def _emit(**kw):
    print(json.dumps(kw), flush=True)


# ------------------------------------------------------------------------------------ gemm
GEMM_SHAPES = [(16384, 1152, 896), (16384, 896, 896), (16384, 9728, 896), (16384, 896, 4864), (8192, 8192, 8192),
               (4096, 151936, 896), (256, 1152, 896), (256, 9728, 896), (256, 151936, 896)]  # fmt: skip
GRAD_SHAPES = [(16384, 9728, 896), (16384, 896, 4864), (16384, 1152, 896)]  # (tokens, out features, in features)


def bench_gemm(a):
    shapes, grads = (GEMM_SHAPES, GRAD_SHAPES) if not a.small else ([(4096, 4096, 4096)], [])
    if a.shape:
        shapes, grads = [tuple(a.shape)], []
    bf = torch.bfloat16
    for M, N, K in shapes:
        x = torch.randn(M, K, device="cuda", dtype=bf)
        w = torch.randn(N, K, device="cuda", dtype=bf)
        fl = 2.0 * M * N * K
        for bn in (128, 256):
            t = time_ms(lambda: ops.gemm(x, w, bn=bn), a.iters)
            _emit(kind="nt", M=M, N=N, K=K, bn=bn, ms=t, tflops=fl / t / 1e9)
        if not a.no_cublas:
            t = time_ms(lambda: x @ w.t(), a.iters)
            _emit(kind="cublas_nt", M=M, N=N, K=K, ms=t, tflops=fl / t / 1e9)
    for T, O, I in grads:
        dy = torch.randn(T, O, device="cuda", dtype=bf)
        w = torch.randn(O, I, device="cuda", dtype=bf)
        x = torch.randn(T, I, device="cuda", dtype=bf)
        acc = torch.zeros(O, I, device="cuda", dtype=torch.float32)
        fl = 2.0 * T * O * I
        for name, fn, ref in (
            ("dgrad", lambda: ops.gemm(dy, w, b_mn=True), lambda: dy @ w),
            ("wgrad", lambda: ops.gemm(dy, x, a_mn=True, b_mn=True, out_dtype=torch.float32), lambda: dy.t() @ x),
            ("wgrad_accumulate", lambda: ops.gemm(dy, x, a_mn=True, b_mn=True, out=acc, accumulate=True), None),
        ):
            t = time_ms(fn, a.iters)
            _emit(kind=name, T=T, O=O, I=I, ms=t, tflops=fl / t / 1e9)
            if ref is not None and not a.no_cublas:
                t = time_ms(ref, a.iters)
                _emit(kind="cublas_" + name, T=T, O=O, I=I, ms=t, tflops=fl / t / 1e9)
    _lib.check_status("cuda")


# ---------------------------------------------------------------------------------- decode
def bench_decode(a):
    """Times each kernel of a decode step in isolation (back-to-back launches, no L2 flush: in a real step the
    weights of a 0.5B model stay L2-resident), then one full layer loop, so shares and launch gaps are visible."""
    from slime_b200.models.config import get_preset

    cfg = get_preset(a.model)
    B, ctx, ps = a.batch, a.context, 16
    d, hq, hkv, H, F, V = cfg.head_dim, cfg.num_attention_heads, cfg.num_query_groups, cfg.hidden_size, cfg.ffn_hidden_size, cfg.vocab_size
    bf, dev = torch.bfloat16, "cuda"
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: (0.02 * torch.randn(*s, device=dev, generator=g)).to(bf)  # noqa: E731
    x, res = rnd(B, H), rnd(B, H)
    x32 = x.float()
    ln = torch.ones(H, device=dev, dtype=bf)
    wqkv, bqkv = rnd((hq + 2 * hkv) * d, H), (rnd((hq + 2 * hkv) * d) if cfg.add_qkv_bias else None)
    wo, wgu, wdn, wlm = rnd(H, hq * d), rnd(2 * F, H), rnd(H, F), rnd(V, H)
    pages = B * math.ceil((ctx + 1) / ps) + 1
    kc, vc = rnd(pages * ps, hkv, d), rnd(pages * ps, hkv, d)
    per = math.ceil((ctx + 1) / ps)
    bt = (1 + torch.arange(B * per, device=dev, dtype=torch.int32)).view(B, per).contiguous()
    seq = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    pos = seq - 1
    slots = (bt[:, -1] * ps).to(torch.int32)
    rope = ops.rope_cos_sin(ctx + 8, d, cfg.rotary_base, device=dev)
    qn = torch.ones(d, device=dev, dtype=bf) if cfg.qk_layernorm else None
    temp = torch.ones(B, device=dev)
    seeds = torch.arange(B, device=dev, dtype=torch.int64)
    outp = torch.zeros(B, device=dev, dtype=torch.int32)

    qkv = ops.gemm(x, wqkv, bias=bqkv)
    q3 = qkv.view(B, hq + 2 * hkv, d)
    attn = ops.paged_decode_attention(q3[:, :hq], kc, vc, bt, seq, ps)
    gu = ops.gemm(x, wgu)
    act = ops.swiglu(gu)
    logits = ops.gemm(x, wlm, out_dtype=torch.float32)
    steps = {
        "rmsnorm_add": lambda: ops.rmsnorm(x32, ln, 1e-6, res),  # reads the fp32 projection output
        "gemm_qkv": lambda: ops.gemm(x, wqkv, bias=bqkv),
        "rope_qk": lambda: ops.rope_qk(qkv, pos, rope, hq, hkv, d, qn, qn, 1e-6),
        "kv_write": lambda: ops.kv_write(q3[:, hq : hq + hkv].reshape(B, -1), q3[:, hq + hkv :].reshape(B, -1), slots, kc, vc),
        "rope_kv_write": lambda: ops.rope_kv_write(qkv, pos, rope, slots, kc, vc, hq, hkv, d, qn, qn, 1e-6),
        "paged_attention": lambda: ops.paged_decode_attention(q3[:, :hq], kc, vc, bt, seq, ps),
        "gemm_o": lambda: ops.gemm(attn.reshape(B, -1), wo, out_dtype=torch.float32),
        "gemm_gate_up": lambda: ops.gemm(x, wgu),
        "swiglu": lambda: ops.swiglu(gu),
        "gemm_down": lambda: ops.gemm(act, wdn, out_dtype=torch.float32),  # split-K, summed in fp32
        "gemm_lm_head": lambda: ops.gemm(x, wlm, out_dtype=torch.float32),
        "sample": lambda: ops.sample(logits, temp, None, None, None, seeds, outp, 0),
    }
    # rope_qk and kv_write (training-style ops, four launches) are timed for comparison; the engine uses the fused one
    per_layer = ["rmsnorm_add", "gemm_qkv", "rope_kv_write", "paged_attention", "gemm_o", "rmsnorm_add", "gemm_gate_up",
                 "swiglu", "gemm_down"]  # fmt: skip
    def attn_forced(flag, **kw):  # SLIME_B200_DECODE_ATTN_WS = "1": warp-specialised kernel, "0": the two-chain kernel
        os.environ["SLIME_B200_DECODE_ATTN_WS"] = flag
        try:
            return ops.paged_decode_attention(q3[:, :hq], kc, vc, bt, seq, ps, **kw)
        finally:
            os.environ.pop("SLIME_B200_DECODE_ATTN_WS", None)

    def attn_ws():
        return attn_forced("1", splits=a.splits)

    def attn_ws_loads():  # the same kernel with every landed tile handed straight back: the cost of its copy path alone
        _lib.lib().sb_paged_decode_ws_load_path_only(1)
        try:
            return attn_ws()
        finally:
            _lib.lib().sb_paged_decode_ws_load_path_only(0)

    if d == 64:
        steps["paged_attention_warp_specialised"] = attn_ws
        steps["paged_attention_two_chain"] = lambda: attn_forced("0")
        steps["paged_attention_warp_specialised_load_path"] = attn_ws_loads
    steps["paged_attention_cuda_cores"] = lambda: ops.paged_decode_attention(q3[:, :hq], kc, vc, bt, seq, ps,
                                                                             use_tensor_cores=False)
    t_of = {}
    for name, fn in steps.items():
        # `reps` launches inside one CUDA graph: device time per launch without the host's launch cost
        fn()
        gk = torch.cuda.CUDAGraph()
        with torch.cuda.graph(gk):
            for _ in range(a.reps):
                fn()
        t_of[name] = time_ms(gk.replay, a.iters, flush=False) / a.reps
        _emit(kind="decode_kernel", name=name, batch=B, context=ctx, us=1e3 * t_of[name])
    try:  # a measurement build (-DSB_WS_CHAIN_TIMING) also reports where a softmax group's time per tile goes
        import ctypes

        ticks_fn = _lib.bind("sb_paged_decode_ws_chain_ticks", [ctypes.c_void_p, ctypes.c_int])
    except AttributeError:
        ticks_fn = None
    if ticks_fn is not None and d == 64:
        buf = (ctypes.c_ulonglong * 16)()
        torch.cuda.synchronize()
        ticks_fn(ctypes.addressof(buf), 1)
        attn_ws()
        torch.cuda.synchronize()
        ticks_fn(ctypes.addressof(buf), 0)
        tiles = max(1, buf[6])
        names = ["wait_s", "tmem_ld_max", "group_exchange", "merge_prev", "exp_p_fence", "end_of_item"]
        _emit(kind="decode_attn_ws_chain", batch=B, context=ctx, tiles=int(buf[6]),
              cycles_per_tile={k: buf[i] / tiles for i, k in enumerate(names)})
        inames = ["s_queue", "s_wait_k", "s_wait_group", "s_issue", "o_wait_p", "o_wait_v", "o_wait_group", "o_issue"]
        # the issuers handle the tiles of all four groups: per tile of the CTA (4 x the tiles the clocked group saw)
        _emit(kind="decode_attn_ws_issuers", batch=B, context=ctx,
              cycles_per_cta_tile={k: buf[8 + i] / (4 * tiles) for i, k in enumerate(inames)})
    est = cfg.num_layers * sum(t_of[k] for k in per_layer) + t_of["gemm_lm_head"] + t_of["sample"] + t_of["rmsnorm_add"]

    def layer_loop():
        for _ in range(cfg.num_layers):
            for k in per_layer:
                steps[k]()

    eager = time_ms(layer_loop, max(3, a.iters // 4), flush=False)
    gr = torch.cuda.CUDAGraph()
    with torch.cuda.graph(gr):
        layer_loop()
    graphed = time_ms(gr.replay, max(3, a.iters // 4), flush=False)
    kv_bytes = 2.0 * B * ctx * hkv * d * 2 * cfg.num_layers
    w_bytes = 2.0 * (cfg.num_params() - (0 if cfg.tie_word_embeddings else V * H))
    _emit(kind="decode_step", batch=B, context=ctx, model=a.model, sum_of_kernels_ms=est, layers_eager_ms=eager,
          layers_graph_ms=graphed, kv_bytes=kv_bytes, weight_bytes=w_bytes)
    _lib.check_status("cuda")


# ------------------------------------------------------------------------------------ norm
def bench_norm(a):
    for T, H in ((131072, 896), (1048576, 128), (16384, 4096), (65536, 2560)) if not a.small else ((4096, 4096),):
        x = torch.randn(T, H, device="cuda", dtype=torch.bfloat16, requires_grad=True)
        r = torch.randn(T, H, device="cuda", dtype=torch.bfloat16)
        w = torch.ones(H, device="cuda", dtype=torch.bfloat16, requires_grad=True)
        t = time_ms(lambda: ops.rmsnorm(x.detach(), w.detach(), 1e-6, r), a.iters)
        _emit(kind="rmsnorm_fwd", T=T, H=H, ms=t, gbs=4 * T * H * 2 / t / 1e6)  # read x, r; write y, h
        y, h = ops.rmsnorm(x, w, 1e-6, r)
        gy, gh = torch.randn_like(y), torch.randn_like(h)
        t = time_ms(lambda: torch.autograd.grad([y, h], [x], [gy, gh], retain_graph=True), a.iters)
        _emit(kind="rmsnorm_bwd", T=T, H=H, ms=t, gbs=4 * T * H * 2 / t / 1e6)  # read dy, dres, h; write dh


def bench_fp8(a):
    """Block-scaled fp8 GEMM against this library's bf16 GEMM and torch._scaled_mm (per-tensor scales: a different,
    cheaper scaling scheme, shown only as the library fp8 ceiling)."""
    shapes = [(4096, 4096, 7168), (16384, 2048, 7168), (8192, 1536, 2048), (256, 4096, 7168)] if not a.small else [(1024, 1024, 1024)]
    for M, N, K in shapes:
        x = torch.randn(M, K, device="cuda", dtype=torch.bfloat16)
        w = torch.randn(N, K, device="cuda", dtype=torch.bfloat16) * 0.1
        xq, xs = ops.block_fp8_quant(x, (1, 128))
        wq, ws = ops.block_fp8_quant(w, (128, 128))
        fl = 2.0 * M * N * K
        t = time_ms(lambda: ops.fp8_block_gemm(xq, xs, wq, ws), a.iters)
        _emit(kind="fp8_block", M=M, N=N, K=K, ms=t, tflops=fl / t / 1e9)
        t = time_ms(lambda: ops.gemm(x, w), a.iters)
        _emit(kind="bf16_ours", M=M, N=N, K=K, ms=t, tflops=fl / t / 1e9)
        t = time_ms(lambda: ops.fp8_act_quant(x), a.iters)
        _emit(kind="act_quant_1x128", M=M, K=K, ms=t, gbs=3.0 * M * K / t / 1e6)
        if not a.no_cublas:
            one = torch.ones((), device="cuda")
            try:
                t = time_ms(lambda: torch._scaled_mm(xq, wq.t(), scale_a=one, scale_b=one, out_dtype=torch.bfloat16), a.iters)
                _emit(kind="scaled_mm_per_tensor", M=M, N=N, K=K, ms=t, tflops=fl / t / 1e9)
            except Exception as e:  # noqa: BLE001
                _emit(kind="scaled_mm_per_tensor", error=repr(e)[:200])
    _lib.check_status("cuda")


def bench_moe(a):
    """Expert MLP of Qwen3-30B-A3B (hidden 2048, expert FFN 768, 16 local experts of 128 under EP8): grouped GEMMs
    against the per-expert loop over the same GEMM kernel, for a training-sized and a decode-sized token count."""
    from slime_b200.ops import grouped

    E, H, F = 16, 2048, 768
    w13 = torch.randn(E, 2 * F, H, device="cuda", dtype=torch.bfloat16) * 0.02
    w2 = torch.randn(E, H, F, device="cuda", dtype=torch.bfloat16) * 0.02
    for rows in ((16384, 2048) if not a.small else (2048,)):
        g = torch.Generator(device="cuda").manual_seed(rows)
        cuts = torch.sort(torch.randint(0, rows, (E - 1,), device="cuda", generator=g)).values.tolist()
        counts = [b - c for c, b in zip([0] + cuts, cuts + [rows])]
        x = torch.randn(rows, H, device="cuda", dtype=torch.bfloat16)
        lay = grouped.PaddedLayout(counts, "cuda")
        xp = lay.pad(x)

        def fused():
            return grouped.grouped_gemm(ops.swiglu(grouped.grouped_gemm(xp, w13, lay)), w2, lay)

        def loop():
            outs, s = [], 0
            for e, n in enumerate(counts):
                if n:
                    outs.append(ops.gemm(ops.swiglu(ops.gemm(x[s : s + n], w13[e])), w2[e]))
                    s += n
            return outs

        fl = 2.0 * rows * (2 * F * H + H * F)
        t = time_ms(fused, a.iters)
        _emit(kind="moe_grouped", rows=rows, experts=E, ms=t, tflops=fl / t / 1e9)
        t = time_ms(loop, a.iters)
        _emit(kind="moe_expert_loop", rows=rows, experts=E, ms=t, tflops=fl / t / 1e9)
    _lib.check_status("cuda")


def bench_attn(a):
    """Flash attention forward / backward (own tcgen05 kernels) on packed equal-length sequences, and the flash-attn
    library (an mma.sync-class kernel) on the same tensors when it is importable. FLOPs: causal, 4 * S^2 * H * D / 2 per
    sequence forward, 2.5 x that backward."""
    from slime_b200.ops import attention

    try:
        from flash_attn.flash_attn_interface import _flash_attn_varlen_backward, _flash_attn_varlen_forward
    except Exception:  # noqa: BLE001
        _flash_attn_varlen_forward = None
    cases = [(14, 2, 64, 1024, 16), (14, 2, 64, 4096, 4), (32, 8, 128, 2048, 4), (32, 8, 128, 8192, 1), (16, 4, 128, 8192, 1)]
    if a.small:
        cases = [(32, 8, 128, 2048, 2)]
    for Hq, Hkv, D, S_, nseq in cases:
        T = S_ * nseq
        qkv = (torch.randn(T, (Hq + 2 * Hkv) * D, device="cuda") * 0.5).to(torch.bfloat16)
        x3 = qkv.view(T, Hq + 2 * Hkv, D)
        q, k, v = x3[:, :Hq], x3[:, Hq : Hq + Hkv], x3[:, Hq + Hkv :]
        cu = torch.arange(0, T + 1, S_, dtype=torch.int32, device="cuda")
        seg = attention.segments_from_cu_seqlens(cu)
        scale = 1.0 / math.sqrt(D)
        fwd_flops = 4.0 * S_ * S_ * Hq * D / 2 * nseq
        out, lse = attention.flash_fwd(q, k, v, seg, scale)
        d_o = torch.randn_like(out)
        dqkv = torch.zeros_like(qkv)
        d3 = dqkv.view(T, Hq + 2 * Hkv, D)
        tf = time_ms(lambda: attention.flash_fwd(q, k, v, seg, scale, out=out), a.iters)
        tb = time_ms(lambda: attention.flash_bwd(q, k, v, out, d_o, lse, seg, scale, dq=d3[:, :Hq], dk=d3[:, Hq : Hq + Hkv],
                                                 dv=d3[:, Hq + Hkv :]), a.iters)  # fmt: skip
        rec = dict(kind="flash_attn", Hq=Hq, Hkv=Hkv, D=D, seqlen=S_, nseq=nseq, fwd_ms=tf, fwd_tflops=fwd_flops / tf / 1e9,
                   bwd_ms=tb, bwd_tflops=2.5 * fwd_flops / tb / 1e9)  # fmt: skip
        if _flash_attn_varlen_forward is not None and not a.no_cublas:
            res = _flash_attn_varlen_forward(q, k, v, cu, cu, S_, S_, 0.0, scale, causal=True)
            lo, llse, rng = res[0], res[1], res[3]
            lf = time_ms(lambda: _flash_attn_varlen_forward(q, k, v, cu, cu, S_, S_, 0.0, scale, causal=True), a.iters)
            lb = time_ms(lambda: _flash_attn_varlen_backward(d_o, q, k, v, lo, llse, d3[:, :Hq], d3[:, Hq : Hq + Hkv],
                                                             d3[:, Hq + Hkv :], cu, cu, S_, S_, 0.0, scale, True, -1, -1, 0.0,
                                                             None, False, rng), a.iters)  # fmt: skip
            rec.update(lib_fwd_ms=lf, lib_bwd_ms=lb, lib_fwd_tflops=fwd_flops / lf / 1e9, lib_bwd_tflops=2.5 * fwd_flops / lb / 1e9)
        _emit(**rec)
    _lib.check_status("cuda")


def _peaks() -> tuple[float, float]:
    """(copy GB/s, bf16 TFLOP/s burst) of this pool, measured or an earlier measurement."""
    try:
        with open(os.path.join(os.path.dirname(__file__), "..", "..", "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"], d["bf16_tflops"]
    except OSError:
        return 6650.0, 1590.0


def _window_keys(n: int, window: int, keep: int) -> int:
    """Visible (query, key) pairs of one fresh prompt of ``n`` tokens."""
    return sum(min(i + 1, window) + min(keep, max(0, i + 1 - window)) for i in range(n))


def bench_window(a):
    from slime_b200.ops import attention, stream
    from slime_b200.ops import window_attention as wa

    gbs, tf = _peaks()
    ps, keep, dev, bf16 = 64, 8, "cuda", torch.bfloat16
    rnd = lambda *sh: (torch.randn(*sh, device=dev) * 0.5).to(bf16)  # noqa: E731

    def pair(what, t_new, t_old, work_new, work_old, peak, **kw):
        f_new, f_old = work_new / t_new / peak, work_old / t_old / peak
        _emit(kind=what, us=round(t_new * 1e3, 2), like_us=round(t_old * 1e3, 2), of_peak=round(f_new, 3), like_of_peak=round(f_old, 3),
              times_further=round(f_old / f_new, 2), **kw)  # fmt: skip

    for hq, hkv, d in ((32, 8, 128), (32, 8, 64), (32, 4, 128)) if not a.small else ((32, 8, 128),):
        slopes = torch.tensor([2.0 ** (-8 * (h + 1) / hq) for h in range(hq)], device=dev)
        for n, nseq, window in ((1024, 8, 1024), (4096, 2, 1024), (4096, 2, 4096)) if not a.small else ((2048, 1, 1024),):
            T = n * nseq
            x = rnd(T, hq + 2 * hkv, d)
            q, k, v = x[:, :hq], x[:, hq : hq + hkv], x[:, hq + hkv :]
            pages = [list(range(i * n // ps, (i + 1) * n // ps)) for i in range(nseq)]
            batch = wa.ExtendBatch.build(pages, [0] * nseq, [n] * nseq, ps, dev)
            kc, vc = k.contiguous(), v.contiguous()
            seg = attention.segments_from_cu_seqlens(torch.arange(0, T + 1, n, dtype=torch.int32, device=dev))
            t = time_ms(lambda: wa.window_extend(q, kc, vc, batch, d**-0.5, window, keep, slopes), a.iters)
            t2 = time_ms(lambda: attention.flash_fwd(q, k, v, seg, d**-0.5), a.iters)
            per = 4.0 * d * hq * nseq / 1e9
            pair("attention_prefill", t, t2, per * _window_keys(n, window, keep), per * n * (n + 1) / 2, tf, heads=f"{hq}/{hkv}x{d}",
                 prompts=f"{nseq}x{n}", window=window)  # fmt: skip
        for B, ctx, window in ((64, 1024, 1024), (64, 4096, 1024), (64, 4096, 4096), (4, 1024, 1024)) if not a.small else ((64, 1024, 1024),):
            npg = ctx // ps
            kc, vc = rnd(B * npg * ps, hkv, d), rnd(B * npg * ps, hkv, d)
            bt = torch.randperm(B * npg, device=dev).to(torch.int32).view(B, npg)
            sl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
            q = rnd(B, hq, d)
            t = time_ms(lambda: wa.window_decode(q, kc, vc, bt, sl, sl - 1, ps, d**-0.5, window, keep, slopes), a.iters)
            t2 = time_ms(lambda: ops.paged_decode_attention(q, kc, vc, bt, sl, ps, d**-0.5), a.iters)
            per = B * hkv * d * 4 / 1e6
            seen = min(ctx, window) + (keep if ctx > window else 0)
            pair("attention_decode", t, t2, per * seen, per * ctx, gbs, heads=f"{hq}/{hkv}x{d}", batch=B, context=ctx, window=window)
    for T, H in ((8192, 2560), (64, 2560), (8192, 2048), (4, 2048)) if not a.small else ((8192, 2560),):
        y, res, w, r16 = torch.randn(T, H, device=dev), torch.randn(T, H, device=dev), rnd(H), rnd(T, H)
        t = time_ms(lambda: stream.stream_norm(y, res, w, 1e-5, kind="layer", post_w=w), a.iters)
        t2 = time_ms(lambda: ops.rmsnorm(y, w, 1e-6, r16), a.iters)
        pair("stream_norm", t, t2, T * H * 14 / 1e6, T * H * 10 / 1e6, gbs, rows=T, width=H)
        F = 8192
        gu = rnd(T, 2 * F)
        t = time_ms(lambda: stream.feed_forward_act(gu, "gelu_tanh", True), a.iters)
        t2 = time_ms(lambda: ops.swiglu(gu), a.iters)
        pair("activation", t, t2, T * F * 6 / 1e6, T * F * 6 / 1e6, gbs, rows=T, width=F)
        kv, slots = rnd(T, 48 * 128), torch.randperm(T, device=dev).to(torch.int32)
        kc, vc = rnd(T, 8, 128), rnd(T, 8, 128)
        table, pos = torch.randn(T, 128, device=dev), torch.arange(T, dtype=torch.int32, device=dev)
        t = time_ms(lambda: stream.kv_scatter(kv[:, 4096:5120], kv[:, 5120:], slots, kc, vc), a.iters)
        t2 = time_ms(lambda: ops.rope_kv_write(kv, pos, table, slots, kc, vc, 32, 8, 128), a.iters)
        pair("cache_write", t, t2, T * 8 * 128 * 8 / 1e6, T * (40 * 128 * 4 + 8 * 128 * 6) / 1e6, gbs, rows=T)
    from slime_b200.ops import grouped

    E, H, F, k = 128, 2048, 768, 8
    w1, w13, w2, router = rnd(E, F, H), rnd(E, 2 * F, H), rnd(E, H, F), rnd(136, H)
    for T in (8192, 64, 4) if not a.small else (64,):
        x, sh, res, w = rnd(T, H), rnd(T, H), torch.randn(T, H, device=dev), rnd(H)
        logits = ops.gemm(x, router, out_dtype=torch.float32)
        probs, idx = grouped.route_topk(logits[:, :E], k, renorm=False, raw_index=True)
        lay = grouped.DeviceLayout(idx, E)
        full = rnd(lay.rows_padded, H)
        hit = min(E, T * k) * H * 2 / 1e6

        def new():
            return grouped.grouped_gemm(stream.feed_forward_act(grouped.grouped_gemm(lay.pad(x), w1, lay), "relu2", False), w2, lay)

        def old():
            return grouped.grouped_gemm(ops.swiglu(grouped.grouped_gemm(lay.pad(x), w13, lay)), w2, lay)

        t, t2 = time_ms(new, a.iters), time_ms(old, a.iters)
        if T >= 1024:
            pair("experts", t, t2, 4.0 * T * k * H * F / 1e9, 6.0 * T * k * H * F / 1e9, tf, tokens=T)
        else:
            pair("experts", t, t2, 2 * F * hit, 3 * F * hit, gbs, tokens=T)
        t = time_ms(lambda: stream.stream_norm(stream.ExpertSum(full, lay.slot_dest, probs, sh, logits[:, E]), res, w, 1e-5, kind="layer", post_w=w), a.iters)
        t2 = time_ms(lambda: ops.rmsnorm(grouped.gather_sum(full, lay.slot_dest, probs, k), w, 1e-6, sh), a.iters)
        pair("experts_sum_norm", t, t2, T * H * (2 * k + 2 + 10) / 1e6, T * H * (2 * k + 10) / 1e6, gbs, tokens=T)
        t = time_ms(lambda: grouped.DeviceLayout(idx, E), a.iters)
        _emit(kind="layout", us=round(t * 1e3, 2), tokens=T)
    _lib.check_status("cuda")


def bench_delta(a):
    """Kernels of recurrent layers beside the torch ops of the trainer's delta-net layer (the form the engine used for it), and
    the other kernels of Ledazen layers beside their nearest relatives. Fractions of the copy bandwidth."""
    from slime_b200.models import mixers
    from slime_b200.ops import delta, stream
    from slime_b200.ops import window_attention as wa

    dev, bf = torch.device("cuda"), torch.bfloat16
    gbs, _ = _peaks()
    rnd = lambda *s, dt=bf: torch.randn(*s, device=dev).to(dt)  # noqa: E731

    def emit(what, t, t2, mb, **kw):
        _emit(kind=what, us=round(t * 1e3, 2), of_peak=round(mb / t / gbs, 4), like_us=None if t2 is None else round(t2 * 1e3, 2), **kw)

    for H, G, D, DV, pc in ((32, 16, 128, 128, False), (32, 16, 128, 128, True), (16, 16, 64, 64, True)):
        C = 2 * G * D + H * DV
        conv, rate, bias, w = rnd(C, 4), torch.randn(H, device=dev), torch.randn(H * D if pc else H, device=dev) - 3, rnd(DV)
        tag = dict(heads=H, qk_heads=G, dim=D, vdim=DV, per_channel=pc)

        def inputs(T):
            x, ab, z = rnd(T, C), rnd(T, bias.numel() + 64), rnd(T, H * DV)
            q, k, v = x.split([G * D, G * D, H * DV], 1)
            return x, z, delta.DeltaInputs(q, k, v, ab[:, : bias.numel()], ab[:, bias.numel() : bias.numel() + H], conv, rate, bias)

        for n, L in ((8, 1024), (2, 4096)) if not a.small else ((8, 1024),):
            T = n * L
            x, z, inp = inputs(T)
            state, ring = torch.zeros(n, H, D, DV, device=dev), rnd(n, 4, C)
            batch = wa.ExtendBatch.build([[0]] * n, [0] * n, [L] * n, 8192, dev, state_slots=list(range(n)))
            out = rnd(T, H * DV)
            prof = {}

            def new():
                o = delta.delta_extend(inp, state, ring, batch)
                delta.head_gate(o, z, w, "silu", 1e-5, 1.0, out)
                prof["o"] = o

            t = time_ms(new, a.iters)
            cu = torch.arange(0, T + 1, L, device=dev, dtype=torch.int32)
            pos = torch.arange(T, device=dev) % L

            def old():
                y = mixers.causal_short_conv(x, conv, pos)
                q, k, v = y.split([G * D, G * D, H * DV], -1)
                q, k = (s.view(T, G, D).repeat_interleave(H // G, 1) for s in (q, k))
                g = -rate.exp() * torch.nn.functional.softplus(inp.a.float() + bias)
                o = mixers.gated_delta_rule_chunked(q, k, v.view(T, H, DV), g, torch.sigmoid(inp.b.float()), cu)
                (mixers._rms(o, w, 1e-5).float() * torch.nn.functional.silu(z.view(T, H, DV).float())).to(bf)

            t2 = None if pc else time_ms(old, 3)  # the torch form has no decay per key channel
            mb = T * 2 * (C + 2 * H * DV + bias.numel() + H) / 1e6 + n * H * D * DV * 4 / 1e6
            emit("delta_extend", t, t2, mb, tokens=T, requests=n, **tag)
            o = prof["o"]
            t = time_ms(lambda: delta.head_gate(o, z, w, "silu", 1e-5, 1.0, out), a.iters)
            emit("head_gate", t, None, T * H * DV * 8 / 1e6, tokens=T, **tag)
        for B in (64, 4):
            x, z, inp = inputs(B)
            state, ring = torch.zeros(4 * 64, H, D, DV, device=dev), rnd(4 * 64, 4, C)  # rotating slots: states come from memory
            i32 = lambda v: torch.as_tensor(v, dtype=torch.int32, device=dev)  # noqa: E731
            sets = [i32(range(j * B, (j + 1) * B)) for j in range(4 * 64 // B)]
            one, at, turn, out = i32([1] * B), i32([77] * B), [0], rnd(B, H * DV)

            def new():
                turn[0] = (turn[0] + 1) % len(sets)
                delta.delta_step(inp, state, ring, sets[turn[0]], one, at, z, w, "silu", 1e-5, 1.0, out)

            S, hist = torch.zeros(B, H, D, DV, device=dev), rnd(B, 3, C)

            def old():
                y = mixers.short_conv_step(x, conv, hist)
                q, k, v = y.split([G * D, G * D, H * DV], -1)
                q, k = (s.view(B, G, D).repeat_interleave(H // G, 1) for s in (q, k))
                g = -rate.exp() * torch.nn.functional.softplus(inp.a.float() + bias)
                o = mixers.gated_delta_rule_step(q, k, v.view(B, H, DV), g, torch.sigmoid(inp.b.float()), S)
                (mixers._rms(o.to(bf), w, 1e-5).float() * torch.nn.functional.silu(z.view(B, H, DV).float())).to(bf)

            t, t2 = time_ms(new, a.iters), None if pc else time_ms(old, a.iters)
            emit("delta_step", t, t2, B * (H * D * DV * 8 + C * 10 + H * DV * 4) / 1e6, rows=B, **tag)
    for T in (8192, 64):
        kv, slots = rnd(T, 48 * 128), torch.randperm(T, device=dev).to(torch.int32)
        kc, vc = rnd(T, 8, 128), rnd(T, 8, 128)
        pos, qn = torch.arange(T, dtype=torch.int32, device=dev), rnd(128)
        table = stream.rotary_table(T, 128, 1e6, dev)
        t = time_ms(lambda: stream.place_heads(kv[:, :4096], kv[:, 4096:5120], kv[:, 5120:], slots, kc, vc, q_norm=qn, k_norm=qn, eps=1e-6,
                                               table=table, positions=pos), a.iters)  # fmt: skip
        t2 = time_ms(lambda: ops.rope_kv_write(kv, pos, table, slots, kc, vc, 32, 8, 128, qn, qn, 1e-6), a.iters)
        emit("heads_to_cache", t, t2, T * (40 * 128 * 4 + 8 * 128 * 4) / 1e6, rows=T)
        y, res, r16, w = torch.randn(T, 2560, device=dev), torch.randn(T, 2560, device=dev), rnd(T, 2560), rnd(2560)
        t = time_ms(lambda: stream.stream_norm(y, res, w, 1e-5, offset=1.0), a.iters)
        t2 = time_ms(lambda: ops.rmsnorm(y, w, 1e-6, r16), a.iters)
        emit("stream_norm", t, t2, T * 2560 * 14 / 1e6, rows=T, like_of_peak=round(T * 2560 * 10 / 1e6 / t2 / gbs, 4))
        up, out, gu = rnd(T, 10240 + 256), rnd(T, 10240 + 4096), rnd(T, 2 * 6912)
        t = time_ms(lambda: stream.feed_forward_act(up[:, 256:], "relu2", False, out[:, 4096:]), a.iters)
        t2 = time_ms(lambda: ops.swiglu(gu), a.iters)
        emit("activation", t, t2, T * 10240 * 4 / 1e6, rows=T, like_of_peak=round(T * 6912 * 6 / 1e6 / t2 / gbs, 4))
    _lib.check_status("cuda")


def bench_rules(a):
    """Kernels of Zetizen layers beside the like kernel of the existing models: capped scores with a learned distance bias, chunks,
    latent attention, norms over whole projections, experts beside a mixer."""
    from slime_b200.models.layer_spec import DistanceBiasSpec
    from slime_b200.ops import attention, latent, stream
    from slime_b200.ops import window_attention as wa

    gbs, tf = _peaks()
    ps, dev, bf16 = 64, "cuda", torch.bfloat16
    rnd = lambda *sh: (torch.randn(*sh, device=dev) * 0.5).to(bf16)  # noqa: E731
    i32 = lambda *sh: torch.arange(*sh, dtype=torch.int32, device=dev)  # noqa: E731

    def pair(what, t_new, t_old, work_new, work_old, peak, **kw):
        f_new, f_old = work_new / t_new / peak, work_old / t_old / peak
        _emit(kind=what, us=round(t_new * 1e3, 2), like_us=round(t_old * 1e3, 2), of_peak=round(f_new, 3), like_of_peak=round(f_old, 3),
              times_further=round(f_old / f_new, 2), **kw)  # fmt: skip

    hq, hkv, d, chunk = 32, 4, 128, 1024
    spec = DistanceBiasSpec(32, 128)
    table = torch.randn(spec.rows, hq, device=dev)[spec.by_distance()].contiguous()
    forms = {"bias_cap": dict(softcap=30.0, bias=table), "chunk_cap": dict(softcap=30.0, chunk=chunk), "bias": dict(bias=table), "chunk": dict(chunk=chunk)}
    L = latent.Latent(16, 128, 128, 512, 192**-0.5, rnd(16 * 192, 768), rnd(16 * 256, 512), torch.randn(8192, 64, device=dev))
    for n, nseq in ((1024, 8), (4096, 2)) if not a.small else ((2048, 1),):
        T = n * nseq
        x = rnd(T, hq + 2 * hkv, d)
        q, k, v = x[:, :hq], x[:, hq : hq + hkv], x[:, hq + hkv :]
        pages = [list(range(i * n // ps, (i + 1) * n // ps)) for i in range(nseq)]
        batch = wa.ExtendBatch.build(pages, [0] * nseq, [n] * nseq, ps, dev)
        kc, vc, gate = k.contiguous(), v.contiguous(), rnd(T, hq)
        seg = attention.segments_from_cu_seqlens(i32(0, T + 1, n))
        t2 = time_ms(lambda: attention.flash_fwd(q, k, v, seg, d**-0.5), a.iters)
        per = 4.0 * d * hq * nseq / 1e9
        for name, form in forms.items():
            t = time_ms(lambda: wa.window_extend(q, kc, vc, batch, d**-0.5, gate=gate, **form), a.iters)
            c = form.get("chunk", n)
            pair("attention_prefill", t, t2, per * (n // min(c, n)) * min(c, n) * (min(c, n) + 1) / 2, per * n * (n + 1) / 2, tf, form=name,
                 heads=f"{hq}/{hkv}x{d}", prompts=f"{nseq}x{n}")  # fmt: skip
        H = L.heads
        cache, qq, g, out = rnd(T, 1, 576), rnd(T, H, 192), rnd(T, H, 128), rnd(T, H, 128)
        kv = ops.gemm(cache[:, 0, :512], L.up_kv)
        rule = wa.Rule.of(qq, 128, L.scale, gate=g.flatten(1))
        _, tab, tiles = batch.expansion(tuple(range(nseq)))
        import ctypes

        def core():
            _lib.check(_lib.lib().sb_flash_latent(
                _lib.ptr(qq), _lib.ptr(kv), _lib.ptr(cache[:, 0, 512:]), _lib.ptr(kv[:, H * 128 :]), _lib.ptr(tab), _lib.ptr(tiles), _lib.ptr(out),
                tiles.shape[0], T, H, 128, 64, 128, ps, tab.stride(0), T, qq.stride(0), kv.stride(0), 576, kv.stride(0), out.stride(0),
                ctypes.byref(rule), _lib.ptr(_lib.status_word(qq.device)), _lib.stream()), "sb_flash_latent")  # fmt: skip

        t = time_ms(core, a.iters)
        work = 2.0 * (192 + 128) * H * nseq * n * (n + 1) / 2 / 1e9
        pair("latent_prefill_core", t, t2, work, per * n * (n + 1) / 2, tf, heads=f"{H}x(128+64)/128", prompts=f"{nseq}x{n}")
        t = time_ms(lambda: latent.latent_extend(L, qq, cache, batch, g, out), a.iters)
        _emit(kind="latent_prefill", us=round(t * 1e3, 2), of_peak=round((work + 2.0 * T * H * 256 * 512 / 1e9) / t / tf, 3), prompts=f"{nseq}x{n}")
    for B, ctx in ((64, 1024), (64, 4096), (4, 1024)) if not a.small else ((64, 1024),):
        npg = ctx // ps
        kc, vc = rnd(B * npg * ps, hkv, d), rnd(B * npg * ps, hkv, d)
        bt = torch.randperm(B * npg, device=dev).to(torch.int32).view(B, npg)
        sl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, gate = rnd(B, hq, d), rnd(B, hq)
        t2 = time_ms(lambda: ops.paged_decode_attention(q, kc, vc, bt, sl, ps, d**-0.5), a.iters)
        per = B * hkv * d * 4 / 1e6
        for name, form in forms.items():
            t = time_ms(lambda: wa.window_decode(q, kc, vc, bt, sl, sl - 1, ps, d**-0.5, gate=gate, **form), a.iters)
            pair("attention_decode", t, t2, per * min(ctx, form.get("chunk", ctx)), per * ctx, gbs, form=name, batch=B, context=ctx)
        for H in (16, 128):
            cache, ql = rnd(B * npg * ps, 1, 576), rnd(B, H, 576)
            t = time_ms(lambda: latent.latent_rows(ql, cache, 512, bt, None, sl - 1, ps, 0.07, ctx), a.iters)
            pair("latent_decode", t, t2, B * ctx * 576 * 2 / 1e6, per * ctx, gbs, heads=H, batch=B, context=ctx,
                 of_flops=round(2.0 * B * ctx * H * (576 + 512) / 1e9 / t / tf, 3))  # fmt: skip
    for T in (8192, 64, 4) if not a.small else (64,):
        x, slots, pos = rnd(T, 40 * 128 + 4 * 128), torch.randperm(T, device=dev).to(torch.int32), i32(T)
        kc, vc, table = rnd(T, 4, 128), rnd(T, 4, 128), torch.randn(T, 128, device=dev)
        wq, wk, qn = rnd(4096), rnd(512), rnd(128)
        t = time_ms(lambda: stream.place_heads(x[:, :4096], x[:, 4096:4608], x[:, 4096:4608], slots, kc, vc, q_norm=wq, k_norm=wk, eps=1e-6, table=table,
                                               positions=pos, interleaved=False), a.iters)  # fmt: skip
        y = rnd(T, 40 * 128)
        t2 = time_ms(lambda: ops.rope_kv_write(y, pos, table, slots, kc, vc, 32, 4, 128, qn, qn, 1e-6), a.iters)
        mb = T * (32 * 128 * 4 + 4 * 128 * 2 + 4 * 128 * 4) / 1e6
        pair("heads_over_all", t, t2, mb, mb, gbs, rows=T)
        x, cache, wq, wk, table = rnd(T, 768 + 576), rnd(T, 1, 576), rnd(768), rnd(512), torch.randn(T, 64, device=dev)
        t = time_ms(lambda: latent.latent_place(x[:, :768], x[:, 768:], wq, wk, 1e-6, table, pos, slots, cache), a.iters)
        pair("latent_place", t, t2, T * 1344 * 4 / 1e6, mb, gbs, rows=T)
        qq, lat, out, g = rnd(T, 16, 192), rnd(T, 16, 576), rnd(T, 16, 128), rnd(T, 16, 128)
        gemm_ms = time_ms(lambda: ops.gemm(x[:, :768], L.up_q), a.iters)
        work = (T * 16 * (128 + 512) + 16 * 128 * 512) * 2 / 1e6
        like = (T * (768 + 3072) + 768 * 3072) * 2 / 1e6
        t = time_ms(lambda: latent.head_gemm(qq[..., :128], L.up_k, lat[..., :512], transposed=True), a.iters)
        pair("absorb_queries", t, gemm_ms, work, like, gbs, rows=T)
        t = time_ms(lambda: latent.head_gemm(lat[..., :512], L.up_v, out, gate=g), a.iters)
        pair("expand_values", t, gemm_ms, work + T * 16 * 128 * 2 / 1e6, like, gbs, rows=T)
        t = time_ms(lambda: latent.turn_into(qq, lat[..., 512:], table, pos), a.iters)
        pair("latent_turn", t, t2, T * 16 * 64 * 4 / 1e6, mb, gbs, rows=T)
    from slime_b200.ops import grouped

    E, H, k = 128, 2048, 8
    for T in (8192, 64) if not a.small else (64,):
        res, w, base, sh = torch.randn(T, H, device=dev), rnd(H), torch.randn(T, H, device=dev), rnd(T, H)
        logits, shift = torch.randn(T, 136, device=dev)[:, :E], torch.randn(E, device=dev)
        t = time_ms(lambda: grouped.route_topk(logits, k, renorm=True, raw_index=True, shift=shift), a.iters)
        t2 = time_ms(lambda: grouped.route_topk(logits, k, renorm=True, raw_index=True), a.iters)
        pair("route", t, t2, T * E * 4 / 1e6, T * E * 4 / 1e6, gbs, tokens=T)
        probs, idx = grouped.route_topk(logits, k, renorm=True, raw_index=True, shift=shift)
        lay = grouped.DeviceLayout(idx, E)
        full = rnd(lay.rows_padded, H)
        t = time_ms(lambda: stream.stream_norm(stream.ExpertSum(full, lay.slot_dest, probs, base=base), res, w, 1e-5, kind="layer"), a.iters)
        t2 = time_ms(lambda: ops.rmsnorm(grouped.gather_sum(full, lay.slot_dest, probs, k), w, 1e-6, sh), a.iters)
        pair("experts_beside_norm", t, t2, T * H * (2 * k + 4 + 10) / 1e6, T * H * (2 * k + 10) / 1e6, gbs, tokens=T)
    _lib.check_status("cuda")


def bench_fused_emul(a):
    """The peer-memory kernels with every "rank" a buffer of THIS GPU (profilers attach to one process on one GPU, and
    kernels that wait on one another must not run as separate launches on one device): the data path, instruction mix
    and DRAM behaviour are those of the multi-GPU run, the NVLink hop is not. Flags are preset so no wait occurs."""
    import ctypes

    lib, P = _lib.lib(), _lib.ptr
    dev = torch.device("cuda")
    status = _lib.status_word(dev)
    # ---- data-parallel reduce-scatter shard + squared norm, then Adam + all-gather stores (world = 4)
    world, n = 4, (8 if a.small else 64) * 1024 * 1024
    grads = [torch.randn(n, device=dev) for _ in range(world)]
    params = [torch.zeros(n, device=dev, dtype=torch.bfloat16) for _ in range(world)]
    gp = (ctypes.c_void_p * world)(*[g.data_ptr() for g in grads])
    pp = (ctypes.c_void_p * world)(*[p.data_ptr() for p in params])
    shard = n // world
    partials, ctl = torch.zeros(148 * 8, device=dev), torch.zeros(2, device=dev)
    master, m, v = (torch.zeros(shard, device=dev) for _ in range(3))

    def reduce():
        _lib.check(lib.sb_dp_reduce_shard(gp, world, 0, 0, 0, shard, P(grads[0][:shard]), P(partials), P(ctl), P(status),
                                          _lib.stream()), "sb_dp_reduce_shard")  # fmt: skip

    def adam():
        _lib.check(lib.sb_dp_adam_bcast(P(master), P(m), P(v), P(grads[0][:shard]), pp, world, 0, 0, 0, shard, 1e-6, 0.9, 0.98,
                                        1e-8, 0.1, 0.1, 0.02, 1.0, 1.0, P(ctl), 0, _lib.stream()), "sb_dp_adam_bcast")  # fmt: skip

    t = time_ms(reduce, a.iters)
    _emit(kind="dp_reduce_shard_emulated", world=world, shard_elems=shard, ms=t, read_gbs=world * shard * 4 / t / 1e6)
    t = time_ms(adam, a.iters)
    _emit(kind="dp_adam_bcast_emulated", world=world, shard_elems=shard, ms=t,
          bytes_gbs=(shard * (4 * 4 + 3 * 4) + world * shard * 2) / t / 1e6)  # fmt: skip
    # ---- tensor-parallel all-reduce + residual + RMSNorm (world = 2)
    T, H, world = 256, 2560, 2
    parts = [torch.randn(T, H, device=dev).to(torch.bfloat16) for _ in range(world)]
    flags = torch.full((148 * 8,), 1 << 30, dtype=torch.int32, device=dev)  # every peer "has arrived" already
    epochs = torch.zeros(148, dtype=torch.int32, device=dev)
    res, w = torch.randn(T, H, device=dev).to(torch.bfloat16), torch.ones(H, device=dev, dtype=torch.bfloat16)
    y, r = torch.empty_like(res), torch.empty_like(res)
    ptrs = (ctypes.c_void_p * world)(*[x.data_ptr() for x in parts])
    fl = (ctypes.c_void_p * world)(*[flags.data_ptr()] * world)

    def ar():
        _lib.check(lib.sb_tp_ar_add_rmsnorm(ptrs, fl, P(epochs), P(res), P(w), P(y), P(r), T, H, 1e-6, 0, world, 0, P(status),
                                            _lib.stream()), "sb_tp_ar_add_rmsnorm")  # fmt: skip

    t = time_ms(ar, a.iters)
    _emit(kind="tp_ar_add_rmsnorm_emulated", T=T, H=H, world=world, us=t * 1e3, gbs=(world + 3) * T * H * 2 / t / 1e6)
    want = (parts[0].float() + parts[1].float() + res.float())
    want = want * torch.rsqrt(want.pow(2).mean(-1, keepdim=True) + 1e-6)
    assert (y.float() - want).abs().max() < 0.05
    _lib.check_status(dev)


def bench_scan(a):
    """Kernels of Pebodra layers beside the like kernel of the existing models: Mamba-2 and mLSTM against the gated delta rule with as
    many state elements, differential attention against plain attention of the same projections, and what stands around them."""
    from slime_b200.ops import attention, delta, grouped, linear_scan, stream
    from slime_b200.ops import window_attention as wa

    gbs, tf = _peaks()
    dev, bf = torch.device("cuda"), torch.bfloat16
    rnd = lambda *s, dt=bf: torch.randn(*s, device=dev).to(dt)  # noqa: E731
    i32 = lambda v: torch.as_tensor(v, dtype=torch.int32, device=dev)  # noqa: E731

    def pair(what, t, t2, work, work2, peak=gbs, **kw):
        f, f2 = work / t / peak, None if t2 is None else work2 / t2 / peak
        like = {} if t2 is None else dict(like_us=round(t2 * 1e3, 2), like_of_peak=round(f2, 3), times_further=round(f2 / f, 2))
        _emit(kind=what, us=round(t * 1e3, 2), of_peak=round(f, 3), **like, **kw)

    def space(T, H, G, N, DV):
        ch, widths = H * DV + 2 * G * N, [H * DV, H * DV, G * N, G * N, H]
        return linear_scan.StateSpace(*rnd(T, sum(widths)).split(widths, 1), rnd(ch, 4), rnd(ch), rnd(H, dt=torch.float32), rnd(H, dt=torch.float32) - 3,
                                      rnd(H, dt=torch.float32), rnd(H * DV), G, 1e-5)  # fmt: skip

    def memory(T, H, D, DV):
        widths = [H * D, H * D, H * DV, H, H, H * DV]
        return linear_scan.MatrixMemory(*rnd(T, sum(widths)).split(widths, 1), rnd(H, dt=torch.float32), rnd(H, dt=torch.float32) + 3, rnd(H * DV), 15.0, 1e-5)

    def slots_of(n, H, D, DV, ch=0, normed=False):
        z = lambda *s: torch.zeros(n, *s, device=dev)  # noqa: E731
        return linear_scan.SlotState(z(H, D, DV), z(4, ch).to(bf) if ch else None, z(H, D) if normed else None, z(H, 2) if normed else None)

    def rule(T):
        H, G, D, DV = 32, 16, 128, 128
        x, ab = rnd(T, 2 * G * D + H * DV), rnd(T, 2 * H)
        q, k, v = x.split([G * D, G * D, H * DV], 1)
        inp = delta.DeltaInputs(q, k, v, ab[:, :H], ab[:, H:], rnd(x.shape[1], 4), rnd(H, dt=torch.float32), rnd(H, dt=torch.float32) - 3)
        return inp.gated(rnd(T, H * DV), rnd(DV), "silu", 1e-5)

    # algorithmic bytes: projections in, result out, states of the requests read (steps) and written
    ssm, mem = (64, 8, 128, 64), (8, 256, 512)
    ssm_row, mem_row, rule_row = 2 * (3 * 4096 + 2 * 1024 + 64), 2 * (3 * 4096 + 4096 + 16), 2 * (4096 + 3 * 4096 + 64)
    ssm_S, mem_S, rule_S = 64 * 128 * 64 * 4, 8 * 256 * 513 * 4, 32 * 128 * 128 * 4
    for n, L in ((8, 1024), (2, 4096)) if not a.small else ((4, 256),):
        T, kw = n * L, dict(prompts=f"{n}x{L}")
        batch = wa.ExtendBatch.build([[0]] * n, [0] * n, [L] * n, 8192, dev, state_slots=list(range(n)))
        d, ds = rule(T), slots_of(n, 32, 128, 128, 8192)
        t2 = time_ms(lambda: d.extend(ds, batch), a.iters)
        for what, m, s, row, S in (("mamba2_prompt", space(T, *ssm), slots_of(n, 64, 128, 64, 4096 + 2048), ssm_row, ssm_S),
                                   ("mlstm_prompt", memory(T, *mem), slots_of(n, *mem, normed=True), mem_row, mem_S)):
            out = rnd(T, 4096)
            t = time_ms(lambda: m.extend(s, batch, out), a.iters)
            pair(what, t, t2, (T * row + n * S) / 1e6, (T * rule_row + n * rule_S) / 1e6, **kw)
        m, s = space(T, *ssm), slots_of(n, 64, 128, 64, 4096 + 2048)
        H, G, N, DV = ssm
        x, B, C, gates = (torch.rand(T, *sh, device=dev) for sh in ((H, DV), (G, N), (G, N), (H, 4)))
        segs, runs = batch.segments(), batch.tiles(linear_scan.RUN)
        t = time_ms(lambda: linear_scan._scan(C, B, x, gates, segs, s, skip=m.skip, ring_in=(m.x, m.B, m.C)), a.iters)
        pair("mamba2_scan", t, None, (T * (H * DV * 8 + G * N * 8 + H * 16)) / 1e6, None, **kw)
        P = _lib.ptr
        t = time_ms(lambda: _lib.check(_lib.lib().sb_ssd_prep(P(m.x), P(m.B), P(m.C), P(m.dt), m.x.stride(0), P(m.conv), P(m.conv_b), P(m.A_log),
                    P(m.dt_bias), P(s.ring), P(runs), P(segs), runs.shape[0], P(x), P(B), P(C), P(gates), H, G, N, DV, 4, 0, _lib.stream()), "x"), a.iters)  # fmt: skip
        pair("mamba2_prep", t, None, T * (6 * (H * DV + 2 * G * N) + H * 18) / 1e6, None, **kw)
        o, z, w, out = torch.randn(T, 4096, device=dev), rnd(T, 4096), rnd(4096), rnd(T, 4096)
        t2 = time_ms(lambda: delta.head_gate(o.view(T, 32, 128), z, w[:128], "silu", 1e-5, 1.0, out), a.iters)
        for parts in (8, 1):
            t = time_ms(lambda: linear_scan.part_gate(o, z, w, parts, "silu", 1e-5, gate_first=True, out=out), a.iters)
            pair("part_gate", t, t2, T * 4096 * 8 / 1e6, T * 4096 * 8 / 1e6, parts=parts, **kw)
        H, D, DV = mem
        q, k, v = (torch.rand(T, H, w, device=dev) for w in (D, D, DV))
        s, gates, den = slots_of(n, *mem, normed=True), torch.rand(T, H, 4, device=dev), torch.rand(T, H, device=dev)
        t = time_ms(lambda: linear_scan._scan(q, k, v, gates, segs, s, den=den), a.iters)
        pair("mlstm_scan", t, None, T * H * (DV * 8 + D * 8 + 20) / 1e6, None, **kw)
    for B in (64, 4):
        turn, sets = [0], [i32(range(j * B, (j + 1) * B)) for j in range(256 // B)]  # rotating slots: states come from memory
        one, at = i32([1] * B), i32([77] * B)
        d, ds = rule(B), slots_of(256, 32, 128, 128, 8192)

        def step(m, s, out):
            turn[0] = (turn[0] + 1) % len(sets)
            m.step(s, sets[turn[0]], one, at, out)

        out = rnd(B, 4096)
        t2 = time_ms(lambda: step(d, ds, out), a.iters)
        for what, m, s, row, S in (("mamba2_step", space(B, *ssm), slots_of(256, 64, 128, 64, 6144), ssm_row, ssm_S),
                                   ("mlstm_step", memory(B, *mem), slots_of(256, *mem, normed=True), mem_row, mem_S)):
            t = time_ms(lambda: step(m, s, out), a.iters)
            pair(what, t, t2, B * (row + 2 * S) / 1e6, B * (rule_row + 2 * rule_S) / 1e6, rows=B)
    # differential attention: 32/8 heads of two 64-wide halves and 128-wide values, against 32/8 x 128
    H, G, D, ps, win = 32, 8, 128, 64, 1024
    lam = wa.Pair(torch.tensor([0.4], device=dev), 0.5, 1e-5)
    for n, nseq in ((1024, 8), (4096, 2)) if not a.small else ((1024, 1),):
        T = n * nseq
        x = rnd(T, H + 2 * G, D)
        kc, vc = x[:, H : H + G].contiguous(), x[:, H + G :].contiguous()
        pages = [list(range(i * n // ps, (i + 1) * n // ps)) for i in range(nseq)]
        batch = wa.ExtendBatch.build(pages, [0] * nseq, [n] * nseq, ps, dev)
        seg = attention.segments_from_cu_seqlens(torch.arange(0, T + 1, n, dtype=torch.int32, device=dev))
        t2 = time_ms(lambda: attention.flash_fwd(x[:, :H], kc, vc, seg, D**-0.5), a.iters)
        t3 = time_ms(lambda: wa.window_extend(x[:, :H], kc, vc, batch, D**-0.5, win), a.iters)
        q, wide = rnd(T, H * D), rnd(T, 2 * H, D)
        t = time_ms(lambda: wa.window_extend(wide, kc, vc, batch, 0.125, win, pair=lam), a.iters)
        seen = nseq * (n * (n + 1) / 2 - max(0, n - win) * (n - win + 1) / 2)
        work, causal = 2.0 * H * (2 * 64 + 2 * 128) / 1e9, 4.0 * H * D / 1e9
        pair("pair_attention", t, t2, work * seen, causal * nseq * n * (n + 1) / 2, tf, prompts=f"{nseq}x{n}", plain_windowed_us=round(t3 * 1e3, 2),
             plain_windowed_of_peak=round(causal * seen / t3 / tf, 3))  # fmt: skip
        kv, slots, pos, nw, nd = rnd(T, 2 * G * D), torch.randperm(T, device=dev).int(), torch.arange(T, device=dev).int() % n, rnd(64), rnd(D)
        table, tab2 = stream.rotary_table(n, 64, 1e5, dev), stream.rotary_table(n, 128, 1e5, dev)
        qkv = rnd(T, (H + 2 * G) * D)
        t2 = time_ms(lambda: ops.rope_kv_write(qkv, pos, tab2, slots, kc, vc, H, G, D, nd, nd, 1e-6), a.iters)
        for own in (True, False):
            k, v = (kv[:, : G * D], kv[:, G * D :]) if own else (None, None)
            t = time_ms(lambda: stream.place_heads(q, k, v, slots, kc, vc, q_norm=nw, k_norm=nw if own else None, eps=1e-6, table=table, positions=pos,
                                                   interleaved=False, maps=2), a.iters)  # fmt: skip
            pair("pairs_to_cache", t, t2, T * (H * D * 6 + (2 * G * D * 4 if own else 0)) / 1e6, T * (H * D * 4 + 2 * G * D * 4) / 1e6, rows=T, own_keys=own)
    for B, ctx in ((64, 1024), (64, 4096), (4, 1024)):
        pages = -(-ctx // ps)
        kc, vc = rnd(B * pages * ps, G, D), rnd(B * pages * ps, G, D)
        bt, lens = torch.randperm(B * pages, device=dev).int().view(B, pages), i32([ctx] * B)
        q, wide = rnd(B, H, D), rnd(B, 2 * H, D)
        t2 = time_ms(lambda: ops.paged_decode_attention(q, kc, vc, bt, lens, ps, D**-0.5), a.iters)
        t3 = time_ms(lambda: wa.window_decode(q, kc, vc, bt, lens, lens - 1, ps, D**-0.5, win, max_context=8192), a.iters)
        pos = lens - 1
        t = time_ms(lambda: wa.window_decode(wide, kc, vc, bt, lens, pos, ps, 0.125, win, max_context=8192, pair=lam), a.iters)
        mb = lambda n: B * n * G * D * 4 / 1e6  # noqa: E731
        pair("pair_decode", t, t2, mb(min(ctx, win)), mb(ctx), batch=B, context=ctx, plain_windowed_us=round(t3 * 1e3, 2))
    for T in (8192, 64):
        y, res, r16, w = torch.randn(T, 2560, device=dev), torch.randn(T, 2560, device=dev), rnd(T, 2560), rnd(2560)
        t2 = time_ms(lambda: ops.rmsnorm(y, w, 1e-6, r16), a.iters)
        t = time_ms(lambda: stream.stream_norm(y, res, None, 1e-5, post_w=w, groups=4, emit=bf), a.iters)
        pair("parts_norm", t, t2, T * 2560 * 14 / 1e6, T * 2560 * 10 / 1e6, rows=T)
        z, gu, coef = rnd(T, 9728), rnd(T, 2 * 6912), torch.rand(4, device=dev)
        t, t2 = time_ms(lambda: stream.poly_norm(z, coef, 1e-5), a.iters), time_ms(lambda: ops.swiglu(gu), a.iters)
        pair("poly_norm", t, t2, T * 9728 * 4 / 1e6, T * 6912 * 6 / 1e6, rows=T)
        logits = torch.randn(T, 128, device=dev)
        t = time_ms(lambda: grouped.route_topk(logits, 8, score="sigmoid", renorm=False, raw_index=True, groups=(8, 4)), a.iters)
        t2 = time_ms(lambda: grouped.route_topk(logits, 8, raw_index=True), a.iters)
        pair("grouped_routing", t, t2, T * (512 + 64) / 1e6, T * (512 + 64) / 1e6, rows=T)
    x = torch.randn(64, 151936, device=dev)
    t = time_ms(lambda: stream.softcap_(x, 30.0), a.iters)
    pair("softcap", t, None, x.numel() * 8 / 1e6, None, rows=64)
    _lib.check_status("cuda")


def main(argv=None):
    p = argparse.ArgumentParser(prog="python -m slime_b200.ops.microbench")
    p.add_argument("what", choices=["gemm", "decode", "norm", "fp8", "moe", "attn", "window", "delta", "rules", "scan", "fused_emul"])
    p.add_argument("--iters", type=int, default=20)
    p.add_argument("--reps", type=int, default=20, help="back-to-back launches per timed repetition (decode)")
    p.add_argument("--small", action="store_true")
    p.add_argument("--no-cublas", action="store_true")
    p.add_argument("--shape", type=int, nargs=3, metavar=("M", "N", "K"))
    p.add_argument("--model", default="qwen2.5-0.5b")
    p.add_argument("--batch", type=int, default=256)
    p.add_argument("--context", type=int, default=768)
    p.add_argument("--splits", type=int, default=None, help="sequence splits of the warp-specialised decode attention")
    a = p.parse_args(argv)
    from slime_b200.ops import build

    build.build()
    {"gemm": bench_gemm, "decode": bench_decode, "norm": bench_norm, "fp8": bench_fp8, "moe": bench_moe, "attn": bench_attn, "window": bench_window, "delta": bench_delta, "rules": bench_rules, "scan": bench_scan, "fused_emul": bench_fused_emul}[a.what](a)


if __name__ == "__main__":
    main()
