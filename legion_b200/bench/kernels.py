"""Kernel micro-benchmarks: device-timed (CUDA events, warm-up, L2 flush between iterations), reported
as achieved TFLOP/s or GB/s and as a fraction of the measured peaks in ``MEASURED_PEAKS.json``.

Usage: ``python -m legion_b200.bench.kernels [--only gemm,moe,decode_attn,prefill_attn] [--json out.json]``
The reference ships one hidden ``legion <kernel>-bench`` command per custom kernel (``src/cli/mod.rs:109-215``);
this module is their counterpart.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch


def peaks():
    here = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    p = os.path.join(here, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return d["hbm_gbs"], d["bf16_tflops"], "measured"
    return 6650.0, 1590.0, "fallback"


_flush = None
CASE = {"tokens": None, "attn": None, "gemm": None}


def flush_l2():
    """Evicts L2 by READING a buffer twice its size: the lines it leaves behind are clean, so the timed kernel
    does not pay for write-backs of the flush itself."""
    global _flush
    if _flush is None:
        _flush = torch.zeros(64 << 20, dtype=torch.int32, device="cuda")
    _flush.sum()


ITERS = {"iters": None, "warmup": None}


def timeit(fn, iters=10, warmup=3, flush=True):
    iters = ITERS["iters"] or iters
    warmup = ITERS["warmup"] if ITERS["warmup"] is not None else warmup
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(iters):
        if flush:
            flush_l2()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    ts.sort()
    return ts[len(ts) // 2]


_flush_graph_ms = {}


def timeit_graph(fn, iters=5, warmup=3, reps=20):
    """Device time of one call of ``fn`` replayed from a CUDA graph (no host launch cost in the number) with a cold
    L2. One graph holds ``reps`` x (L2 flush, fn) back to back so the GPU stays busy and at its working clocks (a
    lone kernel between two synchronisations runs at idle clocks and reads several times too slow); the time of a
    graph of ``reps`` flushes alone is subtracted."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()

    def capture(body):
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            for _ in range(reps):
                flush_l2()
                body()
        return g

    def run(g):
        ts = []
        for _ in range(ITERS["iters"] or iters):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            g.replay()                      # brings the clocks up
            a.record()
            g.replay()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        ts.sort()
        return ts[len(ts) // 2]
    flush_l2()
    if reps not in _flush_graph_ms:
        _flush_graph_ms[reps] = run(capture(lambda: None))
    total = run(capture(fn))
    return max(0.0, total - _flush_graph_ms[reps]) / reps


def bench_layer_parts(rows):
    """The pieces of one decode step of a 30B-A3B-shaped layer (16 users, 8K context), each replayed from a CUDA
    graph: which kernel the step time goes to."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    T, H, E, k, F, Hq, Hkv, D, page, ctx = 16, 2048, 128, 8, 768, 32, 4, 128, 64, 8256
    dev = "cuda"
    x = torch.randn(T, H, device=dev).bfloat16()
    res = torch.randn(T, H, device=dev).bfloat16()
    nw = torch.ones(H, device=dev)
    w_qkv = (torch.randn((Hq + 2 * Hkv) * D, H, device=dev) * 0.02).bfloat16()
    w_o = (torch.randn(H, Hq * D, device=dev) * 0.02).bfloat16()
    w_r = (torch.randn(E, H, device=dev) * 0.02).bfloat16()
    wgu = (torch.randn(E, 2 * F, H, device=dev) * 0.02).bfloat16()
    wd = (torch.randn(E, H, F, device=dev) * 0.02).bfloat16()
    attn_in = torch.randn(T, Hq * D, device=dev).bfloat16()
    nb = T * ((ctx + page - 1) // page)
    kc = torch.randn(nb, page, Hkv, D, device=dev).bfloat16()
    vc = torch.randn(nb, page, Hkv, D, device=dev).bfloat16()
    bt = torch.arange(nb, device=dev, dtype=torch.int32).view(T, -1)
    q = torch.randn(T, Hq, D, device=dev).bfloat16()
    cl = torch.full((T,), ctx, device=dev, dtype=torch.int32)
    routing = sm100.router(x, w_r, k)
    ids, wts = routing

    def add(name, fn, byts=0):
        ms = timeit_graph(fn)
        rows.append(dict(kernel="layer_part", part=name, us=ms * 1e3, gbs=byts / ms / 1e6 if byts else 0.0,
                         frac_hbm=byts / ms / 1e6 / hbm if byts else 0.0, peaks=src))
        print(rows[-1], flush=True)

    add("rmsnorm", lambda: sm100.rmsnorm(x, nw, 1e-6, residual=res))
    add("qkv_gemm", lambda: sm100.linear(x, w_qkv), w_qkv.numel() * 2)
    add("o_gemm", lambda: sm100.linear(attn_in, w_o, residual=res), w_o.numel() * 2)
    kv_bytes = T * ctx * Hkv * D * 2 * 2
    for s in (CASE["tokens"] or (4, 8, 9, 10, 12, 16, 22, 33)):
        add(f"decode_attn_splits{s}", lambda: sm100.paged_decode(q, kc, vc, bt, cl, D ** -0.5, n_splits=s,
                                                                   max_ctx=ctx), kv_bytes)
    add("router_route", lambda: sm100.router(x, w_r, k), w_r.numel() * 2)
    add("norm_router_route", lambda: sm100.router(x, w_r, k, norm=(nw, 1e-6, 0.0)), w_r.numel() * 2)
    n_act = int(torch.unique(ids).numel())
    add("moe_experts_dense", lambda: sm100.moe_experts(x, ids, wts, wgu, wd, F, residual=res, norm=(nw, 1e-6, 0.0),
                                                       routing=routing), n_act * 3 * H * F * 2)
    from legion_b200.ops.sm100 import QWeight
    qgu = QWeight(torch.randint(0, 256, (E, 2 * F, H // 2), device=dev, dtype=torch.uint8),
                  torch.randint(48, 64, (E, 2 * F, H // 16), device=dev, dtype=torch.uint8),
                  torch.ones(2 * E, device=dev))
    qd = QWeight(torch.randint(0, 256, (E, H, F // 2), device=dev, dtype=torch.uint8),
                 torch.randint(48, 64, (E, H, F // 16), device=dev, dtype=torch.uint8), torch.ones(E, device=dev))
    add("moe_experts_dense_nvfp4", lambda: sm100.moe_experts(x, ids, wts, qgu, qd, F, residual=res,
                                                            norm=(nw, 1e-6, 0.0), routing=routing),
        n_act * 3 * H * F * 9 // 16)
    add("moe_experts_gather", lambda: sm100.moe_experts(x, ids, wts, wgu, wd, F, residual=res, norm=(nw, 1e-6, 0.0)),
        n_act * 3 * H * F * 2)
    # the MoE pieces on their own
    C = sm100.ext()
    ws = sm100.Workspace.get(torch.device(dev))
    plan = sm100.MoePlan(T, k, E, 32, dev)
    P = T * k
    plan.x_sorted = torch.zeros(P + 32, H, dtype=torch.bfloat16, device=dev)
    plan.h_sorted = torch.zeros(P + 32, F, dtype=torch.bfloat16, device=dev)
    plan.y_pairs = torch.zeros(P, H, dtype=torch.bfloat16, device=dev)
    out = torch.empty(T, H, dtype=torch.bfloat16, device=dev)
    normed = torch.empty_like(out)
    f_plan = lambda: C.moe_plan_gather(ids, wts, 0, E, 32, plan.counts, plan.offsets, plan.sorted_token,
                                       plan.sorted_pair, plan.sorted_w, plan.tile_group, plan.tile_tok0,
                                       plan.tile_ntok, plan.meta, x, plan.x_sorted)
    f_gu = lambda: C.wgemm(wgu.view(E * 2 * F, H), plan.x_sorted, plan.h_sorted, None, None, None, F, True, F, 32, 1,
                           None, None, ws.status, plan.tile_group, plan.tile_tok0, plan.tile_ntok, plan.meta,
                           plan.max_tiles, 2 * F, 0, [])
    f_dn = lambda: C.wgemm(wd.view(E * H, F), plan.h_sorted, plan.y_pairs, None, plan.sorted_w, plan.sorted_pair, H,
                           False, 0, 32, 1, None, None, ws.status, plan.tile_group, plan.tile_tok0, plan.tile_ntok,
                           plan.meta, plan.max_tiles, H, 0, [])
    f_cb = lambda: C.moe_combine(plan.y_pairs, ids, 0, E, None, None, res, out, nw, 1e-6, 0.0, normed)
    f_plan()
    add("moe.plan_gather", f_plan)
    add("moe.gate_up", f_gu, n_act * 2 * H * F * 2)
    add("moe.down", f_dn, n_act * H * F * 2)
    add("moe.combine_norm", f_cb)


def bench_decode_pages(rows):
    """Decode attention at 16 x 8K context for several KV page sizes and head groupings (graph-replayed)."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    B, D, ctx = 16, 128, 8256
    for (Hq, Hkv, page, splits) in ((32, 4, 32, 2), (32, 4, 64, 2), (32, 4, 128, 2), (32, 8, 64, 1), (64, 4, 64, 2),
                                    (32, 4, 64, 1), (32, 4, 128, 1)):
        nb = B * ((ctx + page - 1) // page)
        kc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        vc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        bt = torch.arange(nb, device="cuda", dtype=torch.int32).view(B, -1)
        q = torch.randn(B, Hq, D, device="cuda").bfloat16()
        cl = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        ms = timeit_graph(lambda: sm100.paged_decode(q, kc, vc, bt, cl, D ** -0.5, n_splits=splits, max_ctx=ctx))
        byts = B * ctx * Hkv * D * 2 * 2
        rows.append(dict(kernel="paged_decode", Hq=Hq, Hkv=Hkv, page=page, splits=splits, us=ms * 1e3,
                         gbs=byts / ms / 1e6, frac_hbm=byts / ms / 1e6 / hbm, peaks=src))
        print(rows[-1], flush=True)


def bench_mla(rows):
    """Latent attention, absorbed form: decode at 16 and 64 users x 8K context with 128 heads (graph-replayed).
    FLOPs per key row = 2 * heads * (576 + 512); bytes per key row = 1152."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    nh, page = 128, 64
    cases = ((16, 8192, 1), (64, 8192, 1), (1, 8192, 512))
    if CASE.get("attn"):
        cases = tuple((c[0], c[1], c[2] if len(c) > 2 else 1) for c in CASE["attn"])
    for (B, ctx, q_len) in cases:
        nb = B * ((ctx + page - 1) // page)
        cache = (torch.randn(nb, page, 1, 576, device="cuda") * 0.5).bfloat16()
        bt = torch.arange(nb, device="cuda", dtype=torch.int32).view(B, -1)
        q = (torch.randn(B * q_len, nh, 576, device="cuda") * 0.5).bfloat16()
        cu = torch.arange(0, (B + 1) * q_len, q_len, device="cuda", dtype=torch.int32)
        cl = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        splits = sm100.mla_splits(B, q_len, nh, ctx)
        ms = timeit_graph(lambda: sm100.mla_attn(q, cache, cu, cl, bt, page, q_len, 192 ** -0.5, n_splits=splits))
        keys = B * (ctx * q_len - q_len * (q_len - 1) // 2)
        flops = 2.0 * nh * (576 + 512) * keys
        byts = B * ctx * 1152
        rows.append(dict(kernel="mla_attn", B=B, ctx=ctx, q_len=q_len, splits=splits, us=ms * 1e3,
                         tflops=flops / ms / 1e9, frac_tc=flops / ms / 1e9 / tf, gbs=byts / ms / 1e6, peaks=src))
        print(rows[-1], flush=True)


def bench_moe_fp8(rows):
    """Routed experts of a 30B-A3B-shaped layer at 16 tokens, bf16 against block-scaled FP8 weights (graph-replayed),
    plus the qkv-sized dense projection."""
    from legion_b200.ops import sm100
    from legion_b200.ops.sm100 import Fp8Weight
    hbm, tf, src = peaks()
    T, H, E, k, F = 16, 2048, 128, 8, 768
    dev = "cuda"
    x = torch.randn(T, H, device=dev).bfloat16()
    w_r = (torch.randn(E, H, device=dev) * 0.02).bfloat16()
    routing = sm100.router(x, w_r, k)
    n_act = int(torch.unique(routing.ids).numel())
    gu = (torch.randn(E, 2 * F, H, device=dev) * 0.02).bfloat16()
    dn = (torch.randn(E, H, F, device=dev) * 0.02).bfloat16()
    gq, dq = Fp8Weight.quantize(gu), Fp8Weight.quantize(dn)
    for name, a, b, bytes_per in (("bf16", gu, dn, 2), ("fp8", gq, dq, 1)):
        ms = timeit_graph(lambda: sm100.moe_experts(x, routing.ids, routing.wts, a, b, F, routing=routing))
        byts = n_act * 3 * H * F * bytes_per
        rows.append(dict(kernel="moe_experts_" + name, T=T, active_experts=n_act, us=ms * 1e3, gbs=byts / ms / 1e6,
                         frac_hbm=byts / ms / 1e6 / hbm, peaks=src))
        print(rows[-1], flush=True)
    wq = (torch.randn(5120, H, device=dev) * 0.02).bfloat16()
    wq8 = Fp8Weight.quantize(wq)
    for name, w, bytes_per in (("bf16", wq, 2), ("fp8", wq8, 1)):
        ms = timeit_graph(lambda: sm100.linear(x, w))
        byts = wq.numel() * bytes_per
        rows.append(dict(kernel="linear_5120x2048_" + name, T=T, us=ms * 1e3, gbs=byts / ms / 1e6, peaks=src))
        print(rows[-1], flush=True)


def bench_moe_nvfp4(rows):
    """Routed experts of a 30B-A3B-shaped layer at 16 tokens with the weights kept in NVFP4 (graph-replayed)."""
    from legion_b200.ops import sm100
    from legion_b200.ops.sm100 import QWeight
    hbm, tf, src = peaks()
    T, H, E, k, F = 16, 2048, 128, 8, 768
    dev = "cuda"
    x = torch.randn(T, H, device=dev).bfloat16()
    w_r = (torch.randn(E, H, device=dev) * 0.02).bfloat16()
    routing = sm100.router(x, w_r, k)
    n_act = int(torch.unique(routing.ids).numel())
    qgu = QWeight(torch.randint(0, 256, (E, 2 * F, H // 2), device=dev, dtype=torch.uint8),
                  torch.randint(48, 64, (E, 2 * F, H // 16), device=dev, dtype=torch.uint8),
                  torch.ones(2 * E, device=dev))
    qd = QWeight(torch.randint(0, 256, (E, H, F // 2), device=dev, dtype=torch.uint8),
                 torch.randint(48, 64, (E, H, F // 16), device=dev, dtype=torch.uint8), torch.ones(E, device=dev))
    ms = timeit_graph(lambda: sm100.moe_experts(x, routing.ids, routing.wts, qgu, qd, F, routing=routing))
    byts = n_act * 3 * H * F * 9 // 16
    rows.append(dict(kernel="moe_experts_nvfp4", T=T, active_experts=n_act, us=ms * 1e3, gbs=byts / ms / 1e6,
                     frac_hbm=byts / ms / 1e6 / hbm, peaks=src))
    print(rows[-1], flush=True)


def bench_moe_nv4(rows):
    """MoE block at decode size on the native NVFP4 (W4A4) path, graph-replayed, whole and by piece, for the
    30B-A3B expert shape (128 experts top-8, FFN 768) and the 80B-A3B one (512 experts top-10, FFN 512, shared
    expert stacked behind the routed ones). Bytes = the quantised bytes of the active experts (codes + scales)."""
    from legion_b200.ops import sm100
    from legion_b200.ops.sm100 import Nv4Weight
    hbm, tf, src = peaks()
    dev = "cuda"
    C = sm100.ext()
    for (name, T, H, E, k, F, shared) in (("30b-a3b", 16, 2048, 128, 8, 768, False),
                                          ("80b-a3b", 16, 2048, 512, 10, 512, True),
                                          ("80b-a3b", 64, 2048, 512, 10, 512, True),
                                          ("80b-a3b", 1, 2048, 512, 10, 512, True)):
        if CASE["tokens"] and T not in CASE["tokens"]:
            continue
        G = E + (1 if shared else 0)
        x = torch.randn(T, H, device=dev).bfloat16()
        res = torch.randn(T, H, device=dev).bfloat16()
        nw = torch.ones(H, device=dev)
        w_r = (torch.randn(E, H, device=dev) * 0.02).bfloat16()
        sh_gate = (torch.randn(1, H, device=dev) * 0.02).bfloat16() if shared else None

        def rand_w(rows_, K):
            codes = torch.randint(0, 256, (G, rows_, K // 2), device=dev, dtype=torch.uint8)
            lin = torch.randint(48, 64, (G * rows_, K // 16), device=dev, dtype=torch.uint8)
            atoms = torch.zeros(C.nv4_sf_bytes(G * rows_, K), dtype=torch.uint8, device=dev)
            C.nv4_pack_scales(lin, atoms)
            return codes, atoms
        gc, gs = rand_w(2 * F, H)
        dc, ds = rand_w(H, F)
        qgu = Nv4Weight(gc, gs, torch.full((2 * G,), 1e-3, device=dev))
        qdn = Nv4Weight(dc, ds, torch.full((G,), 1e-3, device=dev))
        kw = dict(shared_slot=shared, sh_gate=sh_gate, slot_stride=128)
        routing = sm100.router(x, w_r, k, **kw)
        n_act = int(torch.unique(routing.ids).numel()) + (1 if shared else 0)
        byts = n_act * 3 * H * F * 9 // 16

        def block():
            xq = sm100.nv4_quant_act(x, norm=(nw, 1e-6, 0.0), residual=res, want_normed=True, key="bench_x")
            r = sm100.router(xq.normed, w_r, k, **kw)
            return sm100._moe_experts_nv4(xq.normed, r.ids, r.wts, qgu, qdn, F, 0, None, None, xq.summed, None,
                                          (nw, 1e-6, 0.0), r, xq=xq)

        def add(part, fn, b=0):
            ms = timeit_graph(fn)
            rows.append(dict(kernel="moe_nv4", shape=name, T=T, part=part, active=n_act, us=ms * 1e3,
                             gbs=b / ms / 1e6 if b else 0.0, frac_hbm=b / ms / 1e6 / hbm if b else 0.0, peaks=src))
            print(rows[-1], flush=True)
        add("block(addnorm+quant, route, gate_up, down, combine+norm)", block, byts)
        xq = sm100.nv4_quant_act(x, key="bench_x2")
        ws = sm100.Workspace.get(torch.device(dev))
        dr = routing.dense
        hs = torch.tensor([32.0 / 2688.0], device=dev)
        rows_h = dr.n_slots * dr.stride
        hq = torch.zeros(rows_h, F // 2, dtype=torch.uint8, device=dev)
        hsf = torch.zeros(C.nv4_sf_bytes(rows_h, F), dtype=torch.uint8, device=dev)
        y = torch.zeros(T * k + 64, H, dtype=torch.bfloat16, device=dev)
        add("addnorm_quant", lambda: sm100.nv4_quant_act(x, norm=(nw, 1e-6, 0.0), residual=res, want_normed=True,
                                                         key="bench_x3"))
        add("route", lambda: sm100.router(x, w_r, k, **kw), w_r.numel() * 2)
        add("gate_up", lambda: C.wgemm_nv4(qgu.view2d(), qgu.sf, qgu.gscale, xq.codes, xq.sf, xq.gscale, 1, None, None,
                                           None, None, F, True, F, 0, dr.bn, ws.status, dr.tile_group, dr.zeros,
                                           dr.tile_ntok, dr.meta, dr.n_slots, 2 * F, 0, dr.slot_base, hq, hsf, hs),
            n_act * 2 * H * F * 9 // 16)
        add("down", lambda: C.wgemm_nv4(qdn.view2d(), qdn.sf, qdn.gscale, hq, hsf, hs, 0, y, None, dr.tok_scale,
                                        dr.out_rows, H, False, 0, 0, dr.bn, ws.status, dr.tile_group, dr.slot_base,
                                        dr.tile_ntok, dr.meta, dr.n_slots, H, 0, None, None, None, None),
            n_act * H * F * 9 // 16)


def bench_gdn(rows):
    """Gated DeltaNet recurrence over a prompt (80B-A3B hybrid shape: 16 key / 32 value heads of dim 128) and over a
    decode step of 16 sequences: tokens per second of the state update."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    nk, nv, dk, dv = 16, 32, 128, 128
    C = 2 * nk * dk + nv * dv
    for n_seq, L in (CASE["attn"] or ((1, 8192), (16, 1))):
        T = n_seq * L
        qkv = (torch.randn(T, C, device="cuda") * 0.3).bfloat16()
        g = -torch.rand(T, nv, device="cuda") * 0.1
        beta = torch.rand(T, nv, device="cuda")
        state = torch.zeros(n_seq, nv, dk, dv, device="cuda")
        cu = torch.arange(0, (n_seq + 1) * L, L, device="cuda", dtype=torch.int32)
        slots = torch.arange(n_seq, device="cuda", dtype=torch.int32)
        cu_host = list(range(0, (n_seq + 1) * L, L))
        ms = timeit(lambda: sm100.gdn_recurrent(qkv, g, beta, state, cu, slots, nk, nv, dk, dv, False, dk ** -0.5,
                                                cu_host=cu_host), iters=5, flush=False)
        # prompts of >= 64 tokens run the chunked tensor-core scan (prep + scan kernels), decode rows the
        # state-streaming kernel. Chunk-form FLOPs per 64-token chunk and head: K K^T, Q K^T, T V, T K (prep) and
        # W S, Q' S, M D, D^T K' (scan), each 2 * 64 * 64 * 128 or 2 * 64 * 128 * 128
        row = dict(kernel="gdn (chunked scan)" if L >= 64 else "gdn_recurrent", n_seq=n_seq, L=L, ms=ms,
                   tok_s=T / ms * 1e3, state_gbs=n_seq * nv * dk * dv * 4 * 2 / ms / 1e6, peaks=src)
        if L >= 64:
            chunks = n_seq * ((L + 63) // 64) * nv
            flops = chunks * (4 * 2 * 64 * 64 * 128 + 4 * 2 * 64 * 128 * 128)
            row["tflops"] = flops / ms / 1e9
        rows.append(row)
        print(rows[-1], flush=True)


def bench_linear(rows):
    """Linear-attention state with a scalar decay (constant per head; selective as in Mamba-2) beside the recurrent
    kernels of the other families, over a prompt and over decode steps. frac_hbm: bytes the operands and the state must
    move once, over the measured copy bandwidth."""
    from legion_b200.ops import sm100
    hbm, _, src = peaks()

    def row(kernel, n_seq, L, ms, byts, launches=None):
        rows.append(dict(kernel=kernel, n_seq=n_seq, L=L, us=round(ms * 1e3, 2), mbytes=round(byts / 1e6, 1),
                         frac_hbm=round(byts / ms / 1e6 / hbm, 3), peaks=src))
        print(rows[-1], flush=True)
    for n_seq, L in (CASE["attn"] or ((1, 8192), (16, 1), (64, 1))):
        T = n_seq * L
        cu = torch.arange(0, (n_seq + 1) * L, L, device="cuda", dtype=torch.int32)
        cu_host = list(range(0, (n_seq + 1) * L, L))
        slots = torch.arange(n_seq, device="cuda", dtype=torch.int32)
        rnd = lambda *s: (torch.randn(*s, device="cuda") * 0.3).bfloat16()          # noqa: E731
        tm = timeit if L > 1 else timeit_graph
        # Lightning attention, 16 heads of 128 x 128
        H, N, P = 16, 128, 128
        proj = rnd(T, 4 * H * N)
        st = torch.zeros(n_seq, H, P, N, device="cuda")
        dec = torch.full((H,), 0.99, device="cuda")
        q, k, v, g = (proj[:, i * H * N:(i + 1) * H * N] for i in range(4))
        scan = lambda: sm100.linear_scan(q, k, v, st, cu, slots, H, H, N, P, decay=dec, silu_in=True, max_len=L,   # noqa: E731
                                         cu_host=cu_host)
        row("linear_scan constant 16x128x128", n_seq, L, tm(scan), T * 4 * H * N * 2 + st.numel() * 8)
        o, w = scan(), torch.ones(H * P, device="cuda")
        row("group_norm_gate 2048", n_seq, L, tm(lambda: sm100.group_norm_gate(o, g, w, 1e-5)), T * H * P * 6)
        # Mamba-2, 64 heads of 64, state 128, 8 groups
        H, N, P, G = 64, 128, 64, 8
        C = H * P + 2 * G * N
        proj = rnd(T, H * P + C + H)
        z, xbc, dt = proj[:, :H * P], proj[:, H * P:H * P + C], proj[:, H * P + C:]
        st = torch.zeros(n_seq, H, P, N, device="cuda")
        conv = torch.zeros(n_seq, C, 3, device="cuda")
        cw, cb = torch.randn(C, 4, device="cuda"), torch.zeros(C, device="cuda")
        A, D, db = (-torch.ones(H, device="cuda") for _ in range(3))
        ssd_bytes = T * (2 * H * P + C + H) * 2 + st.numel() * 8
        c = sm100.causal_conv1d_silu(xbc, cw, cb, conv, cu, slots, max_len=L)
        if L == 1:
            row("ssd_decode 64x64x128 (with convolution)", n_seq, L,
                tm(lambda: sm100.ssd_decode(xbc, cw, cb, conv, dt, db, A, D, z, st, cu, slots, H, G, N, P)),
                ssd_bytes + conv.numel() * 8)
        else:
            row("linear_scan selective 64x64x128", n_seq, L,
                tm(lambda: sm100.linear_scan(c[:, H * P + G * N:], c[:, H * P:H * P + G * N], c[:, :H * P], st, cu, slots,
                                             H, G, N, P, dt=dt, dt_bias=db, A=A, D=D, z=z, max_len=L, cu_host=cu_host)),
                ssd_bytes)
            row("conv1d_silu", n_seq, L, tm(lambda: sm100.causal_conv1d_silu(xbc, cw, cb, conv, cu, slots, max_len=L)),
                T * C * 4)
        st2 = torch.zeros(n_seq, H, P, N, device="cuda")
        row("mamba2_scan 64x64x128 (Nemotron-H)", n_seq, L,
            tm(lambda: sm100.mamba2_scan(c, dt, z, A, D, db, st2, cu, slots, H, P, G, N)), ssd_bytes)
        # Gated DeltaNet, 16 heads of 128 x 128
        H = 16
        qkv = rnd(T, 3 * H * 128)
        gg, beta = -torch.rand(T, H, device="cuda") * 0.1, torch.rand(T, H, device="cuda")
        st = torch.zeros(n_seq, H, 128, 128, device="cuda")
        gdn_bytes = T * 4 * H * 128 * 2 + st.numel() * 8
        if L > 1:
            row("gdn chunked 16x128x128", n_seq, L,
                tm(lambda: sm100.gdn_recurrent(qkv, gg, beta, st, cu, slots, H, H, 128, 128, False, 128 ** -0.5,
                                               cu_host=cu_host)), gdn_bytes)
        else:
            pj = rnd(T, 4 * H * 128 + 2 * H)
            cw, hist = torch.randn(3 * H * 128, 4, device="cuda"), torch.zeros(n_seq, 3 * H * 128, 3, device="cuda")
            one = torch.ones(128, device="cuda")
            row("gdn_decode_fused 16x128x128 (convolution, norm and gate included)", n_seq, L,
                tm(lambda: sm100.gdn_decode_fused(pj, cw, hist, -one[:H], one[:H], one, 1e-6, "silu", st, slots, H, H, 128,
                                                  128, False, 128 ** -0.5)), T * 5 * H * 128 * 2 + st.numel() * 8 + hist.numel() * 8)


def bench_hyper(rows):
    """The stream update of hyper-connections (4 fp32 streams, next input and norm included) beside the residual + RMS
    norm launch of the other families."""
    from legion_b200.ops import sm100
    hbm, _, src = peaks()
    S, H = 4, 2048
    for T in CASE["tokens"] or (16, 64, 1024, 8192):
        X, y = torch.randn(T, S, H, device="cuda"), torch.randn(T, H, device="cuda").bfloat16()
        mix, v, w = torch.eye(S, device="cuda"), torch.ones(S, device="cuda"), torch.zeros(H, device="cuda")
        tm = timeit_graph if T <= 64 else timeit
        for name, fn, byts in (
                ("hyper_step 4x2048", lambda: sm100.hyper_step(X, [(y, 1.0)], mix, v, v, w, 1e-5, 1.0),
                 T * H * (S * 8 + 4)),
                ("residual + rmsnorm 2048", lambda: sm100.rmsnorm(y, w, 1e-5, 1.0, y), T * H * 8)):
            ms = tm(fn)
            rows.append(dict(kernel=name, T=T, us=round(ms * 1e3, 2), frac_hbm=round(byts / ms / 1e6 / hbm, 3), peaks=src))
            print(rows[-1], flush=True)


def bench_resid(rows):
    """The residual step between grouped norms (input convolution of four taps and history included) beside the residual +
    RMS norm launch and the hyper-connection step of the other families."""
    from legion_b200.ops import sm100
    hbm, _, src = peaks()
    for T, n_seq in ((1, 1), (16, 16), (64, 64), (1024, 1), (8192, 1), (8192, 8)):
        for H in (2048, 4096):
            x, y = torch.randn(T, H, device="cuda"), torch.randn(T, H, device="cuda").bfloat16()
            w, taps, hist = torch.ones(H, device="cuda"), torch.randn(4, H, device="cuda"), torch.zeros(n_seq, 3, H, device="cuda")
            L = T // n_seq
            cu = torch.arange(0, T + 1, L, device="cuda", dtype=torch.int32)
            slots = torch.arange(n_seq, device="cuda", dtype=torch.int32)
            tm = timeit_graph
            for name, fn, byts in (
                    (f"resid_step {H}", lambda: sm100.resid_step(x, y, w, w, 4, 1e-5, (taps, hist, cu, slots, True), max_len=L),
                     T * H * 12 + hist.numel() * 8),
                    (f"residual + rmsnorm {H}", lambda: sm100.rmsnorm(y, w, 1e-5, 0.0, y), T * H * 8)):
                ms = tm(fn)
                rows.append(dict(kernel=name, T=T, n_seq=n_seq, us=round(ms * 1e3, 2), frac_hbm=round(byts / ms / 1e6 / hbm, 3),
                                 peaks=src))
                print(rows[-1], flush=True)


def bench_diag(rows):
    """RG-LRU (2560 channels, 10 blocks): decode launch (convolution, gates, recurrence, GELU branch) and the launches of a
    prompt. frac_hbm: bytes that must move once."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    W, nb, KC = 2560, 10, 4
    d = W // nb
    f = lambda *s: torch.randn(*s, device="cuda")                                    # noqa: E731
    in_b, cw, cb, gb, ld, yb = f(W), f(W, KC), f(W), f(2 * W), -torch.rand(W, device="cuda"), f(W)
    gw = (f(2 * W, d) * d ** -0.5).bfloat16()
    for n, L in ((1, 1), (16, 1), (64, 1), (1, 8192), (8, 1024)):
        T = n * L
        cu, cu_host = torch.arange(0, T + 1, L, device="cuda", dtype=torch.int32), list(range(0, T + 1, L))
        slots = torch.arange(n, device="cuda", dtype=torch.int32)
        proj = f(T, 2 * W).bfloat16()
        y, x = proj[:, :W], proj[:, W:]
        conv, st = torch.zeros(n, W, KC - 1, device="cuda"), torch.zeros(n, W, device="cuda")
        if L == 1:
            parts = [("rglru_decode", lambda: sm100.rglru_decode(x, in_b, cw, cb, conv, gw, gb, ld, y, yb, st, cu, slots, nb),
                      T * W * 6 + st.numel() * 8 + conv.numel() * 8 + gw.numel() * 2)]
        else:
            cv = lambda: sm100.causal_conv1d_silu(x, cw, cb, conv, cu, slots, max_len=L, in_bias=in_b, silu=False)   # noqa: E731
            u = cv()
            gates = sm100.block_gates(u, gw, nb)
            scan = lambda: sm100.gated_recurrence(u, gates, gb, ld, y, yb, st, cu, slots, nb, max_len=L, cu_host=cu_host)  # noqa: E731

            def whole():
                v = cv()
                sm100.gated_recurrence(v, sm100.block_gates(v, gw, nb), gb, ld, y, yb, st, cu, slots, nb, max_len=L,
                                       cu_host=cu_host)
            parts = [("conv1d", cv, T * W * 4), ("block_gates", lambda: sm100.block_gates(u, gw, nb), T * W * 10 + gw.numel() * 2),
                     ("gated_recurrence", scan, T * W * 14), ("rglru all", whole, T * W * 6)]
        for name, fn, byts in parts:
            ms = (timeit_graph if L == 1 else timeit)(fn)
            rows.append(dict(kernel=name, n_seq=n, L=L, us=round(ms * 1e3, 2), frac_hbm=round(byts / ms / 1e6 / hbm, 3), peaks=src))
            print(rows[-1], flush=True)


def bench_delta(rows):
    """Gurozen: delta rule with a decay per key channel, what lies between the attention projections and the scores, soft-capped
    attention, squared-ReLU experts and the residual step, each beside the like kernel of the other families. frac_hbm: bytes
    that must move once; frac_tc: FLOPs over measured cuBLAS bf16 (attention, experts)."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    f = lambda *s: (torch.randn(*s, device="cuda") * 0.5).bfloat16()                 # noqa: E731

    def row(kernel, n, L, ms, byts=None, flops=None):
        r = dict(kernel=kernel, n_seq=n, L=L, us=round(ms * 1e3, 2), peaks=src)
        if byts:
            r["frac_hbm"] = round(byts / ms / 1e6 / hbm, 3)
        if flops:
            r["frac_tc"] = round(flops / ms / 1e9 / tf, 3)
        rows.append(r)
        print(r, flush=True)
    H, D, KC = 16, 128, 4
    C = 3 * H * D
    cw, A, db, one = torch.randn(KC, C, device="cuda"), -torch.ones(H, device="cuda"), torch.zeros(H * D, device="cuda"), torch.ones(D, device="cuda")
    for n, L in (CASE["attn"] or ((1, 1), (16, 1), (64, 1), (1, 8192), (4, 2048))):
        T = n * L
        cu, cu_host = torch.arange(0, T + 1, L, device="cuda", dtype=torch.int32), list(range(0, T + 1, L))
        slots = torch.arange(n, device="cuda", dtype=torch.int32)
        tm = timeit if L > 1 else timeit_graph
        qkv, araw, braw, gate = f(T, C), f(T, H * D), f(T, H), f(T, H * D)
        st, hist = torch.zeros(n, H, D, D, device="cuda"), torch.zeros(n, KC - 1, C, device="cuda")
        args = (qkv, cw, hist, araw, A, db, braw, st, cu, slots, H, H, D, D)
        byts = T * 5 * H * D * 2 + st.numel() * 8 + hist.numel() * 8
        cwg, histg = torch.randn(C, KC, device="cuda"), torch.zeros(n, C, KC - 1, device="cuda")      # Gated DeltaNet's layout
        gg, beta = -torch.rand(T, H, device="cuda") * 0.1, torch.rand(T, H, device="cuda")
        if L == 1:
            row("channel_delta_decode 16x128x128 (convolution, norm and gate included)", n, L,
                tm(lambda: sm100.channel_delta_decode(*args, gate, one, 1e-6)), byts + T * H * D * 2)
            pj = f(T, 4 * H * D + 2 * H)
            row("gdn_decode_fused, same size", n, L, tm(lambda: sm100.gdn_decode_fused(
                pj, cwg, histg, -one[:H], one[:H], one, 1e-6, "silu", st, slots, H, H, D, D, False, D ** -0.5)), byts)
        else:
            row("channel_delta 16x128x128 (convolution included)", n, L, tm(lambda: sm100.channel_delta(*args, max_len=L)), byts)
            c = sm100.causal_conv1d_silu(qkv, cwg, None, histg, cu, slots, max_len=L)
            row("gdn chunked, same size", n, L, tm(lambda: sm100.gdn_recurrent(c, gg, beta, st, cu, slots, H, H, D, D, False, D ** -0.5,
                                                                             cu_host=cu_host)), byts)
            row("conv1d_silu in front of it", n, L, tm(lambda: sm100.causal_conv1d_silu(qkv, cwg, None, histg, cu, slots, max_len=L)), T * C * 4)
            o = f(T, H * D)
            row("head_norm_gate 16x128", n, L, tm(lambda: sm100.head_norm_gate(o, gate, one, 1e-6, H)), T * H * D * 6)
            row("gated_rmsnorm (Gated DeltaNet)", n, L, tm(lambda: sm100.gated_rmsnorm(o.view(T, H, D), gate, one, 1e-6)), T * H * D * 6)
        # attention: 16 query heads over 4 kv heads of 128
        G, page = 4, 64
        nb, ctx = max(1, -(-L // page)), max(L, 2048)
        nb = ctx // page
        kc, vc = f(n * nb, page, G, D), f(n * nb, page, G, D)
        bt = torch.arange(n * nb, device="cuda", dtype=torch.int32).view(n, nb)
        pos = torch.arange(ctx - L, ctx, device="cuda", dtype=torch.int32).repeat(n)
        cells = (bt.long()[:, :, None] * page + torch.arange(page, device="cuda")).view(n, -1)[:, ctx - L:].reshape(-1).contiguous()
        proj, cs = f(T, (H + 2 * G) * D), torch.randn(ctx, 64, device="cuda")
        Cq = proj.shape[1]
        aw, ab, ah = torch.randn(KC, Cq, device="cuda"), torch.randn(Cq, device="cuda"), torch.zeros(n, KC - 1, Cq, device="cuda")
        qn, kn = torch.ones(H * D, device="cuda"), torch.ones(G * D, device="cuda")
        row("qkv_conv_append 16/4 heads of 128", n, L, tm(lambda: sm100.qkv_conv_append(
            proj, ab, aw, ah, cu, slots, qn, kn, "all", 1e-6, cs, "half", pos, cells, kc, vc, H, max_len=L)), T * Cq * 4)
        row("qk_norm_rope_append, same size", n, L, tm(lambda: sm100.qk_norm_rope_append(
            proj, H, G, D, one, one, 1e-6, 0.0, cs, 64, pos, cells, kc, vc)), T * Cq * 4)
        q, cl = f(T, H, D), torch.full((n,), ctx, device="cuda", dtype=torch.int32)
        for cap in (30.0, 0.0):
            name = "soft-capped attention" if cap else "attention"
            if L == 1:
                row(f"{name}, decode at {ctx}", n, L, tm(lambda: sm100.paged_decode(q, kc, vc, bt, cl, D ** -0.5, max_ctx=ctx, softcap=cap)),
                    n * ctx * G * D * 4)
            else:
                row(f"{name}, prompt", n, L, tm(lambda: sm100.prefill_attn(q, kc, vc, cu, cl, bt, L, D ** -0.5, softcap=cap)),
                    flops=n * L * L / 2 * H * D * 4)
        # residual step of 2048 columns
        W = 2048
        x, y, nw = torch.randn(T, W, device="cuda"), f(T, W), torch.zeros(W, device="cuda")
        row("prenorm_step 2048", n, L, tm(lambda: sm100.prenorm_step(x, [(y, 1.0)], 0.5, nw, 1e-6, 1.0, dtype=torch.bfloat16)), T * W * 12)
        xb = f(T, W)
        row("residual + RMS norm 2048", n, L, tm(lambda: sm100.rmsnorm(y, nw, 1e-6, 1.0, residual=xb)), T * W * 8)
        # experts: 32 of 1536 (squared ReLU), of 1024 (gated), top 4
        E, k = 32, 4
        rw = f(E + 1, W)
        for act, ff in (("relu2", 1536), ("silu", 1024)):
            up, dn = f(E + 1, ff if act == "relu2" else 2 * ff, W), f(E + 1, W, ff)
            sh = act == "relu2"

            def experts():
                r = sm100.router(y, rw if sh else rw[:E], k, "sigmoid", "sum", 2.0, None, 8, 4, n_local=E, gate_row=sh, shared_slots=int(sh))
                m = E + int(sh and r.dense is not None)
                return sm100.moe_experts(y, r.ids, r.wts, up[:m], dn[:m], ff, 0, routing=r, defer_combine="pairs", act=act)
            slots_used = k + (1 if sh and T <= 64 else 0)
            seen = min(E, E * (1 - (1 - k / E) ** T)) + (1 if sh and T <= 64 else 0)
            row(f"router + experts {act} {ff}", n, L, tm(experts), byts=seen * (up[0].numel() + dn[0].numel()) * 2 + T * W * 2 * (2 + slots_used),
                flops=2.0 * T * slots_used * (up[0].numel() + dn[0].numel()))
            del up, dn


def bench_forget(rows):
    """Mananex: HGRN2 state, rotation and append, windowed attention with sinks, kept first tokens and head gates, gated residual
    with depth average, biased gate / up and routing, each beside the like kernel of the other families. frac_hbm: bytes that
    must move once; frac_tc: FLOPs over measured cuBLAS bf16 (attention, products)."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    f = lambda *s: (torch.randn(*s, device="cuda") * 0.5).bfloat16()                 # noqa: E731

    def row(kernel, n, L, ms, byts=None, flops=None):
        r = dict(kernel=kernel, n_seq=n, L=L, us=round(ms * 1e3, 2), peaks=src)
        if byts:
            r["frac_hbm"] = round(byts / ms / 1e6 / hbm, 3)
        if flops:
            r["frac_tc"] = round(flops / ms / 1e9 / tf, 3)
        rows.append(r)
        print(r, flush=True)
    H, G, D, W, window = 16, 4, 128, 2048, 1024
    one, zero = torch.ones(H * D, device="cuda"), torch.zeros(H * D, device="cuda")
    for n, L in (CASE["attn"] or ((1, 1), (16, 1), (64, 1), (1, 8192), (4, 2048))):
        T = n * L
        cu, cu_host = torch.arange(0, T + 1, L, device="cuda", dtype=torch.int32), list(range(0, T + 1, L))
        slots = torch.arange(n, device="cuda", dtype=torch.int32)
        tm = timeit if L > 1 else timeit_graph
        # HGRN2, 16 heads of 128 x 128
        proj, st, low = f(T, 4 * H * D), torch.zeros(n, H, D, D, device="cuda"), torch.rand(H * D, device="cuda") * 0.9
        q, k, v, g = (proj[:, i * H * D:(i + 1) * H * D] for i in range(4))
        byts = T * 4 * H * D * 2 + st.numel() * 8
        row("forget_scan 16x128x128 (norm included)", n, L, tm(lambda: sm100.forget_scan(
            q, k, v, one, low, st, cu, slots, H, D, D, one[:D], 1e-6, max_len=L, cu_host=cu_host)), byts)
        dec = torch.full((H,), 0.99, device="cuda")
        scan = lambda: sm100.linear_scan(q, k, v, st, cu, slots, H, H, D, D, decay=dec, silu_in=True, max_len=L, cu_host=cu_host)  # noqa: E731
        row("linear_scan constant decay, same size", n, L, tm(scan), byts)
        o = scan()
        row("group_norm_gate 2048 behind it", n, L, tm(lambda: sm100.group_norm_gate(o, g, one, 1e-5)), T * H * D * 6)
        cw, hist = torch.randn(4, 3 * H * D, device="cuda"), torch.zeros(n, 3, 3 * H * D, device="cuda")
        args = (f(T, 3 * H * D), cw, hist, k, -one[:H], zero, f(T, H), st, cu, slots, H, H, D, D)
        if L == 1:
            row("channel_delta_decode, same size (convolution, norm and gate included)", n, L,
                tm(lambda: sm100.channel_delta_decode(*args, g, one[:D], 1e-6)), byts + hist.numel() * 8)
        else:
            row("channel_delta, same size (convolution included)", n, L, tm(lambda: sm100.channel_delta(*args, max_len=L)), byts)
        # attention: 16 query heads over 4 kv heads of 128, window 1024
        page, ctx = 64, max(L, 2048)
        nb = ctx // page
        kc, vc = f(n * nb, page, G, D), f(n * nb, page, G, D)
        bt = torch.arange(n * nb, device="cuda", dtype=torch.int32).view(n, nb)
        pos = torch.arange(ctx - L, ctx, device="cuda", dtype=torch.int32).repeat(n)
        cells = (bt.long()[:, :, None] * page + torch.arange(page, device="cuda")).view(n, -1)[:, ctx - L:].reshape(-1).contiguous()
        qkv, cs = f(T, (H + 2 * G) * D), torch.randn(ctx, 64, device="cuda")
        row("rotation and append 16/4 heads of 128", n, L, tm(lambda: sm100.qkv_conv_append(
            qkv, None, None, None, cu, slots, None, None, "head", 1e-6, cs, "pairs", pos, cells, kc, vc, H, max_len=L)), T * qkv.shape[1] * 4)
        row("qk_norm_rope_append, same size", n, L, tm(lambda: sm100.qk_norm_rope_append(
            qkv, H, G, D, one[:D], one[:D], 1e-6, 0.0, cs, 64, pos, cells, kc, vc)), T * qkv.shape[1] * 4)
        qq, cl, gate = f(T, H, D), torch.full((n,), ctx, device="cuda", dtype=torch.int32), f(T, H)
        ext = lambda: sm100.attention_ext(qq, kc, vc, bt, cl, cu, L, D ** -0.5, window, 4, zero[:H], gate, 0.5, max_ctx=ctx)   # noqa: E731
        if L == 1:
            kv = n * min(ctx, window) * G * D * 4
            row(f"windowed attention, sink and head gate, decode at {ctx}", n, L, tm(ext), kv)
            row(f"windowed attention, decode at {ctx}", n, L, tm(lambda: sm100.paged_decode(
                qq, kc, vc, bt, cl, D ** -0.5, window, max_ctx=ctx)), kv)
        else:
            flops = n * (L - window / 2) * window * H * D * 4
            row("windowed attention, sink and head gate, prompt", n, L, tm(ext), flops=flops)
            row("windowed attention, prompt", n, L, tm(lambda: sm100.prefill_attn(qq, kc, vc, cu, cl, bt, L, D ** -0.5, window)), flops=flops)
        # residual with gates and depth average: four layers from the 1st, 13th and 21st of 24 on
        hist = sm100.DepthHistory(torch.zeros(25, T, W, device="cuda"))
        x, y, p2, nw = torch.randn(T, W, device="cuda"), f(T, W), f(T, 2 * W), torch.zeros(W, device="cuda")
        co = [torch.ones(26, device="cuda") for _ in range(4)]

        def four(i):
            for j in range(i, i + 4):
                sm100.depth_step(x, hist, j, y, p2[:, :W], nw, y, p2[:, W:], nw, nw, co[:4 - (j - i)], nw, 1e-6, 1.0)
        for i in (0, 12, 20):
            row(f"depth_step 2048, behind layers {i} .. {i + 3}, each", n, L, tm(lambda: four(i)) / 4, T * W * (i + 22 - (i == 20) + 10))
        del hist
        X, mix = torch.randn(T, 4, W, device="cuda"), torch.eye(4, device="cuda")
        row("hyper_step 4x2048", n, L, tm(lambda: sm100.hyper_step(X, [(y, 1.0)], mix, one[:4], one[:4], nw, 1e-5, 1.0)), T * W * 36)
        row("prenorm_step 2048", n, L, tm(lambda: sm100.prenorm_step(x, [(y, 1.0)], 0.5, nw, 1e-6, 1.0, dtype=torch.bfloat16)), T * W * 12)
        # feed-forward parts
        gu, ff = f(2 * 6144, W), 6144
        gb = torch.zeros(2 * ff, device="cuda")
        for name, b in (("gate / up 6144 with biases", gb), ("gate / up 6144", None)):
            row(name, n, L, tm(lambda: sm100.gate_up_act(y, gu, ff, bias=b)), gu.numel() * 2 + T * (W + ff) * 2, 2.0 * T * gu.numel())
        rw, up, dn = f(32, W), f(32, 2 * 1024, W), f(32, W, 1024)
        rb = torch.zeros(32, device="cuda")
        seen = 32 * (1 - (1 - 4 / 32) ** T)
        for name, mode, b in (("router with logit bias + experts", "biased_softmax", rb), ("router + experts", "softmax", None)):
            def experts():
                r = sm100.router(y, rw, 4, mode, True, 1.0, b, n_local=32)
                return sm100.moe_experts(y, r.ids, r.wts, up, dn, 1024, 0, routing=r, defer_combine="pairs")
            row(name, n, L, tm(experts), seen * (up[0].numel() + dn[0].numel()) * 2 + T * W * 12, 8.0 * T * (up[0].numel() + dn[0].numel()))


class Batch:
    """The fields of a step that a planner reads."""

    def __init__(self, **kw):
        self.__dict__.update(kw)


def bench_latent(rows):
    """Latent attention of two sizes: the pieces of a decode step and of a prompt. Attention by the bytes of the latents
    (decode) or the FLOPs of the per-head form, 2 (dim + rot + vdim) per visible pair and head (prompts)."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    for H, dim, R, L, V in ((16, 128, 64, 512, 128), (32, 128, 64, 512, 128), (16, 64, 32, 256, 64)):
        for n, q_len, ctx in ((1, 1, 8192), (16, 1, 2048), (16, 1, 8192), (64, 1, 8192), (1, 8192, 8192), (1, 2048, 16384)):
            T, page = n * q_len, 64
            f = lambda *s: (torch.randn(*s, device="cuda") * 0.5).bfloat16()        # noqa: E731
            nb = n * ctx // page
            cache, bt = f(nb, page, 1, L + R), torch.arange(nb, device="cuda", dtype=torch.int32).view(n, -1)
            proj = f(T, H * (dim + R) + L + R + H * V)
            nq = H * (dim + R)
            q, kv, gate = proj[:, :nq], proj[:, nq:nq + L + R], proj[:, nq + L + R:]
            uk, uv = f(H * L, dim), f(H * V, L)
            w = torch.ones(L, device="cuda")
            cs = torch.randn(ctx, R, device="cuda")
            pos = torch.arange(ctx - q_len, ctx, device="cuda", dtype=torch.int32).repeat(n)
            slots = torch.cat([torch.arange(ctx - q_len, ctx, device="cuda") + i * ctx for i in range(n)])
            cu = torch.arange(0, T + 1, q_len, device="cuda", dtype=torch.int32)
            cl = torch.full((n,), ctx, device="cuda", dtype=torch.int32)
            pairs = n * (q_len * ctx - q_len * (q_len - 1) / 2)
            args = (uv, w, 1e-5, cs)
            if q_len == 1:
                qa = sm100.latent_queries(q, kv, uk, w, 1e-5, cs, pos, slots, cache, H, dim, R)
                fns = [("latent_attention", lambda: sm100.latent_attention(qa, cache, bt, cl, cu, 1, 0.07, L, R, max_ctx=ctx)),
                       ("latent_decode (queries, append, attention, values, gate)", lambda: sm100.latent_decode(
                           q, kv, gate, uk, *args, pos, slots, cache, bt, cl, cu, 0.07, H, dim, R, ctx))]
            else:
                part = sm100.latent_parts(Batch(cu_q=cu, ctx_lens=cl, block_table=bt, positions=pos, slots=slots, token_ids=pos,
                                                n_seqs=n, max_q_len=q_len, max_ctx=ctx, cu_q_host=list(range(0, T + 1, q_len)),
                                                ctx_host=[ctx] * n, latent_parts=None), page)[0]
                rows_uk = f(H * dim, L)

                def latent_space():
                    qs = sm100.latent_queries(q, kv, uk, w, 1e-5, cs, pos, slots, cache, H, dim, R)
                    sm100.latent_values(sm100.latent_attention(qs, cache, bt, cl, cu, q_len, 0.07, L, R, max_ctx=ctx), uv, gate)
                fns = [("latent space, all", latent_space),
                       ("latent_prompt (per head), all", lambda: sm100.latent_prompt(q, kv, gate, rows_uk, *args, cache, part, 0.07,
                                                                                     H, dim, R))]
                if R == 64:
                    kc, vc = f(nb, page, H, dim + R), f(nb, page, H, V)
                    qq = f(T, H, dim + R)
                    fns.append(("prefill_attn (its attention alone)",
                                lambda: sm100.prefill_attn(qq, kc, vc, cu, cl, bt, q_len, 0.07)))
            for name, fn in fns:
                ms = (timeit_graph if q_len == 1 else timeit)(fn)
                r = dict(kernel=name, heads=H, dims=(dim, R, L, V), n_seq=n, q_len=q_len, ctx=ctx, us=round(ms * 1e3, 2), peaks=src)
                if q_len == 1:
                    r["frac_hbm"] = round(n * ctx * (L + R) * 2 / ms / 1e6 / hbm, 3)
                else:
                    r["frac_tflops"] = round(2.0 * H * pairs * (dim + R + V) / ms / 1e9 / tf, 3)
                rows.append(r)
                print(r, flush=True)


def bench_attn_sizes(rows):
    """Attention with key and value heads of different sizes, windowed and not, beside equal sizes: prompts by FLOPs of
    the visible scores, decode by the bytes of the visible keys and values."""
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    Hq, Hkv, page = 16, 4, 64
    for n_seq, L, ctx in ((1, 8192, 8192), (16, 1, 8192)):
        for dk, dv in ((128, 128), (96, 192), (64, 128), (128, 64)):
            for window in (0, 1024):
                nb = n_seq * (ctx // page)
                kc = torch.randn(nb, page, Hkv, dk, device="cuda").bfloat16()
                vc = torch.randn(nb, page, Hkv, dv, device="cuda").bfloat16()
                bt = torch.arange(nb, device="cuda", dtype=torch.int32).view(n_seq, -1)
                q = torch.randn(n_seq * L, Hq, dk, device="cuda").bfloat16()
                cl = torch.full((n_seq,), ctx, device="cuda", dtype=torch.int32)
                seen = ctx if not window else min(window, ctx)
                r = dict(kernel="prefill_attn" if L > 1 else "paged_decode", n_seq=n_seq, ctx=ctx, heads=(Hq, Hkv, dk, dv),
                         window=window, peaks=src)
                if L > 1:
                    cu = torch.arange(0, (n_seq + 1) * L, L, device="cuda", dtype=torch.int32)
                    ms = timeit(lambda: sm100.prefill_attn(q, kc, vc, cu, cl, bt, L, dk ** -0.5, window), iters=5)
                    pairs = L * seen - seen * (seen - 1) / 2 if window else L * (L + 1) / 2
                    r.update(us=round(ms * 1e3, 1), frac_tflops=round(2.0 * n_seq * pairs * (dk + dv) * Hq / ms / 1e9 / tf, 3))
                else:
                    ms = timeit_graph(lambda: sm100.paged_decode(q, kc, vc, bt, cl, dk ** -0.5, window, max_ctx=ctx))
                    r.update(us=round(ms * 1e3, 1), frac_hbm=round(n_seq * seen * Hkv * (dk + dv) * 2 / ms / 1e6 / hbm, 3))
                rows.append(r)
                print(r, flush=True)


def bench_gemm(rows):
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    for (T, N, K) in CASE["gemm"] or [(8192, 5120, 2048), (8192, 2048, 4096), (4096, 8192, 8192), (16, 5120, 2048), (16, 2048, 4096),
                      (64, 151936, 2048), (1, 5120, 2048), (256, 17408, 5120)]:
        x = torch.randn(T, K, device="cuda").bfloat16()
        w = torch.randn(N, K, device="cuda").bfloat16()
        out = torch.empty(T, N, device="cuda", dtype=torch.bfloat16)
        ms = timeit(lambda: sm100.linear(x, w, out=out))
        ms_t = timeit(lambda: torch.matmul(x, w.t(), out=out))
        fl = 2.0 * T * N * K / ms / 1e9
        gb = (N * K + T * K + T * N) * 2 / ms / 1e6
        rows.append(dict(kernel="wgemm", T=T, N=N, K=K, ms=ms, tflops=fl, gbs=gb, frac_tflops=fl / tf, frac_hbm=gb / hbm,
                         cublas_ms=ms_t, peaks=src))
        print(rows[-1], flush=True)


def bench_moe(rows):
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    E, k, H, F = 128, 8, 2048, 768
    wgu = (torch.randn(E, 2 * F, H, device="cuda") * 0.02).bfloat16()
    wd = (torch.randn(E, H, F, device="cuda") * 0.02).bfloat16()
    for T in (CASE["tokens"] or (1, 16, 64, 1024, 8192)):
        x = torch.randn(T, H, device="cuda").bfloat16()
        logits = torch.randn(T, E, device="cuda")
        ids, wts = sm100.router_topk(logits, k)
        ms = timeit(lambda: sm100.moe_experts(x, ids, wts, wgu, wd, F))
        n_act = int(torch.unique(ids).numel())
        byts = n_act * 3 * H * F * 2
        fl = 2.0 * T * k * 3 * H * F / ms / 1e9
        rows.append(dict(kernel="moe_experts", T=T, active_experts=n_act, ms=ms, tflops=fl, weight_gbs=byts / ms / 1e6,
                         frac_tflops=fl / tf, frac_hbm=byts / ms / 1e6 / hbm, peaks=src))
        print(rows[-1], flush=True)


def bench_decode_attn(rows):
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    Hq, Hkv, D, page = 32, 4, 128, 64
    for B, ctx in (CASE["attn"] or ((1, 8192), (16, 8192), (64, 8192), (16, 1024))):
        nb = B * ((ctx + page - 1) // page)
        kc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        vc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        bt = torch.arange(nb, device="cuda", dtype=torch.int32).view(B, -1)
        q = torch.randn(B, Hq, D, device="cuda").bfloat16()
        cl = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        ms = timeit(lambda: sm100.paged_decode(q, kc, vc, bt, cl, D ** -0.5, max_ctx=ctx))
        byts = B * ctx * Hkv * D * 2 * 2
        rows.append(dict(kernel="paged_decode", B=B, ctx=ctx, ms=ms, gbs=byts / ms / 1e6, frac_hbm=byts / ms / 1e6 / hbm,
                         peaks=src))
        print(rows[-1], flush=True)


def bench_prefill_attn(rows):
    from legion_b200.ops import sm100
    hbm, tf, src = peaks()
    Hq, Hkv, D, page = CASE.get("heads") or (32, 4, 128, 64)
    for n_seq, L in (CASE["attn"] or ((1, 8192), (4, 2048), (1, 32768))):
        nb = n_seq * (L // page)
        kc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        vc = torch.randn(nb, page, Hkv, D, device="cuda").bfloat16()
        bt = torch.arange(nb, device="cuda", dtype=torch.int32).view(n_seq, -1)
        q = torch.randn(n_seq * L, Hq, D, device="cuda").bfloat16()
        cu = torch.arange(0, (n_seq + 1) * L, L, device="cuda", dtype=torch.int32)
        cl = torch.full((n_seq,), L, device="cuda", dtype=torch.int32)
        out = torch.empty_like(q)
        ms = timeit(lambda: sm100.prefill_attn(q, kc, vc, cu, cl, bt, L, D ** -0.5, out=out), iters=5)
        fl = 4.0 * n_seq * L * L / 2 * D * Hq / ms / 1e9
        rows.append(dict(kernel="prefill_attn", n_seq=n_seq, L=L, heads=(Hq, Hkv, D), ms=ms, tflops=fl,
                         frac_tflops=fl / tf, peaks=src))
        print(rows[-1], flush=True)


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--only", default="gemm,moe,decode_attn,prefill_attn")
    ap.add_argument("--json", default=None)
    ap.add_argument("--tokens", default=None, help="moe: comma list of token counts")
    ap.add_argument("--attn", default=None, help="attention: BxCTX[,BxCTX...] (decode) or SEQSxLEN (prefill)")
    ap.add_argument("--gemm", default=None, help="gemm: TxNxK[,TxNxK...]")
    ap.add_argument("--heads", default=None, help="prefill attention: HQxHKVxD (page 64), default 32x4x128")
    ap.add_argument("--iters", type=int, default=None)
    ap.add_argument("--warmup-iters", type=int, default=None)
    a = ap.parse_args(argv)
    ITERS["iters"], ITERS["warmup"] = a.iters, a.warmup_iters
    if a.tokens:
        CASE["tokens"] = tuple(int(x) for x in a.tokens.split(","))
    if a.attn:
        CASE["attn"] = tuple(tuple(int(y) for y in x.split("x")) for x in a.attn.split(","))
    if a.heads:
        hq, hkv, d = (int(x) for x in a.heads.split("x"))
        CASE["heads"] = (hq, hkv, d, 64)
    if a.gemm:
        CASE["gemm"] = [tuple(int(y) for y in x.split("x")) for x in a.gemm.split(",")]
    rows = []
    table = {"forget": bench_forget, "delta": bench_delta, "resid": bench_resid, "diag": bench_diag, "latent": bench_latent, "linear": bench_linear, "hyper": bench_hyper, "attn_sizes": bench_attn_sizes, "moe_nv4": bench_moe_nv4, "gdn": bench_gdn, "moe_fp8": bench_moe_fp8, "mla": bench_mla, "moe_nvfp4": bench_moe_nvfp4, "layer_parts": bench_layer_parts, "decode_pages": bench_decode_pages, "gemm": bench_gemm, "moe": bench_moe, "decode_attn": bench_decode_attn, "prefill_attn": bench_prefill_attn}
    for name in a.only.split(","):
        table[name](rows)
    from legion_b200.ops.sm100 import Workspace
    torch.cuda.synchronize()
    print("status word:", Workspace.get("cuda").check())
    if a.json:
        json.dump(rows, open(a.json, "w"), indent=1)


if __name__ == "__main__":
    main(sys.argv[1:])
