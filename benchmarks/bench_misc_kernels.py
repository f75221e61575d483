"""Device timings of the sampling, gated-delta-net, conv, LoRA and MTP-glue kernels (CUDA events, L2 flushed
between iterations, 3 warm-ups), reported against the algorithmic bytes and the measured copy bandwidth.

    python benchmarks/bench_misc_kernels.py [--case sample|gdn|recurrence|stream|sandwich|postnorm|latent|conv|lora|all] [--small]

``--small`` shrinks every case to a few hundred MB so that a profiler capture of one launch ends quickly."""
import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from vllm_kunlun_b200 import ops  # noqa: E402

PEAK_GBS = 6548.5
try:
    with open(os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")) as f:
        PEAK_GBS = float(json.load(f).get("hbm_gbs", PEAK_GBS))
except Exception:  # noqa: BLE001
    pass


def timeit(fn, iters=10, warm=3):
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(iters):
        flush.fill_(1)
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1))
    ts.sort()
    return ts[len(ts) // 2] * 1e-3


def report(name, sec, nbytes, extra=""):
    gbs = nbytes / sec / 1e9
    print(json.dumps({"kernel": name, "us": round(sec * 1e6, 1), "GB/s": round(gbs, 1),
                      "frac_of_measured_copy_bw": round(gbs / PEAK_GBS, 3), "note": extra}))


def case_sample(small):
    B, V = (16, 151936) if not small else (16, 32000)
    logits = torch.randn(B, V, device="cuda").to(torch.bfloat16)
    t = torch.full((B,), 0.8, device="cuda")
    k = torch.full((B,), 50, dtype=torch.int32, device="cuda")
    p = torch.full((B,), 0.9, device="cuda")
    sec = timeit(lambda: ops.topk_topp_sample(logits, t, k, p, seed=1))
    report("topk_topp_sample_kernel", sec, B * V * 2, f"B={B} V={V}; 11 passes over the row, L2 resident after the first")
    g = torch.zeros(B, device="cuda")
    sec = timeit(lambda: ops.topk_topp_sample(logits, g, None, None))
    report("topk_topp_sample_kernel(greedy)", sec, B * V * 2, f"B={B} V={V}")

    def torch_path():
        lg = logits.float() / 0.8
        from vllm_kunlun_b200.ops.reference import misc as ref
        lg = ref.apply_top_k_top_p(lg, k.long(), p)
        pr = lg.softmax(-1)
        return (pr / torch.empty_like(pr).exponential_()).argmax(-1)
    sec = timeit(torch_path)
    report("sort-based torch sampler (comparison)", sec, B * V * 2)


def case_gdn(small):
    Hk, Hv, D = 16, 32, 128
    for name, R, L in (("decode", 16, 1), ("prefill", 16 if not small else 4, 2048 if not small else 512)):
        T = R * L
        C = 2 * Hk * D + Hv * D
        mixed = torch.randn(T, C, device="cuda").to(torch.bfloat16)
        q, k = mixed[:, :Hk * D].view(T, Hk, D), mixed[:, Hk * D:2 * Hk * D].view(T, Hk, D)
        v = mixed[:, 2 * Hk * D:].view(T, Hv, D)
        g = -torch.rand(T, Hv, device="cuda")
        beta = torch.rand(T, Hv, device="cuda")
        states = torch.zeros(R, Hv, D, D, device="cuda")
        cu = (torch.arange(R + 1, device="cuda") * L).int()
        idx = torch.arange(R, device="cuda").int()
        init = torch.ones(R, device="cuda").int()
        sec = timeit(lambda: ops.gated_delta_rule(q, k, v, g, beta, states, cu, idx, init))
        nbytes = 2 * states.numel() * 4 + T * C * 2 + T * Hv * D * 2
        report(f"gdn_recurrent_kernel({name})", sec, nbytes, f"R={R} L={L}; {T * Hv * 3 * D * D * 2 / sec / 1e12:.2f} TFLOP/s fp32 FMA")


def case_recurrence(small):
    """Linear recurrences of the layer-list designs: fixed decay per head and delta rule with a decay per key channel."""
    H, D = 32, 128
    for name, R, L in (("decode", 16, 1), ("prefill", 4, 2048 if not small else 512)):
        T = R * L
        mixed = torch.randn(T, 3 * H * D, device="cuda").to(torch.bfloat16)
        q, k, v = (mixed[:, i * H * D:(i + 1) * H * D].as_strided((T, H, D), (3 * H * D, D, 1), i * H * D) for i in range(3))
        states = torch.zeros(R, H, D, D, device="cuda")
        cu = (torch.arange(R + 1, device="cuda") * L).int()
        idx, init = torch.arange(R, device="cuda").int(), torch.ones(R, device="cuda").int()
        nd = R if L == 1 else 0
        decay = torch.linspace(0.9, 0.999, H, device="cuda")
        nbytes = 2 * states.numel() * 4 + T * 3 * H * D * 2 + T * H * D * 4
        sec = timeit(lambda: ops.fixed_decay_attention(q, k, v, decay, states, cu, idx, init, L, nd))
        report(f"fixed_decay_attention({name})", sec, nbytes, f"R={R} L={L}")
        a = torch.randn(T, H * D, device="cuda").to(torch.bfloat16)
        b = torch.randn(T, H, device="cuda").to(torch.bfloat16)
        A_log, dt = torch.zeros(H, device="cuda"), torch.full((H * D,), -3.0, device="cuda")
        f, bias, low = torch.randn(T, H * D, device="cuda").to(torch.bfloat16), torch.full((H * D,), 3.0, device="cuda"), \
            torch.rand(H * D, device="cuda")
        sec = timeit(lambda: ops.gated_write_attention(q, v, f, bias, low, states, cu, idx, init, L, nd))
        report(f"gated_write_attention({name})", sec, nbytes, f"R={R} L={L}")
        sec = timeit(lambda: ops.channel_delta_rule(q, k, v, a, b, A_log, dt, states, cu, idx, init, D ** -0.5, 1e-6, L, nd))
        report(f"channel_delta_rule({name})", sec, nbytes + T * H * D * 2, f"R={R} L={L}")


def case_stream(small):
    """fp32-stream kernels: post-norm residual step, unit-RMS split with cache write, gated group norm."""
    T, W, H, G, D = (8192 if not small else 4096), 4096, 32, 8, 128
    x = torch.randn(T, W, device="cuda")
    y1, y2 = (torch.randn(T, W, device="cuda").to(torch.bfloat16) for _ in range(2))
    w = torch.ones(W, device="cuda")
    sec = timeit(lambda: ops.layernorm_residual(x, torch.bfloat16, [(y1, 1.0), (y2, 0.5)], w, 1e-5))
    report("layernorm_residual_kernel", sec, T * W * (8 + 2 + 2 + 2), f"T={T} W={W}, two summands")
    proj = torch.randn(T, (H + 2 * G) * D, device="cuda").to(torch.bfloat16)
    cache = torch.zeros(T // 64, 2, G, 64, D, device="cuda", dtype=torch.bfloat16)
    slots = torch.arange(T, device="cuda")
    sec = timeit(lambda: ops.qk_unit_norm_cache(proj[:, :H * D], proj[:, H * D:(H + G) * D], proj[:, (H + G) * D:], cache,
                                                slots, H, G, 1e-5))
    report("qk_unit_norm_cache_kernel", sec, 2 * T * (H + 2 * G) * D * 2, f"T={T} {H}/{G} heads of {D}")
    out = torch.empty(T, W, device="cuda", dtype=torch.bfloat16)
    for n, name in ((W, "whole row"), (D, f"groups of {D}")):
        sec = timeit(lambda: ops.gated_group_rmsnorm(x, y1, w[:n], 1e-5, out))
        report("gated_group_rmsnorm_kernel", sec, T * W * 8, f"T={T} W={W}, {name}")
    ids, pos = torch.randint(0, 32000, (T,), device="cuda"), torch.arange(T, device="cuda")
    table, turns = torch.randn(32000, W, device="cuda").to(torch.bfloat16), ops.position_turns(W, 10000.0).cuda()
    sec = timeit(lambda: ops.embed_positions_layernorm(ids, pos, table, turns, w, 1e-5))
    report("embed_layernorm_kernel", sec, T * W * 8, f"T={T} W={W}")


def case_sandwich(small):
    """Norms around every sublayer, polynomial activation, attention with a bias by distance and output gates (32 / 8 heads
    of 128) beside the same kernels without, experts on weighted inputs: 4 prompts of 2048 tokens, 16 tokens behind 2080."""
    W, F, H, G, D, E, k, ff = 4096, 12288, 32, 8, 128, 32, 4, 1536
    dev, bf = "cuda", torch.bfloat16

    def rnd(*shape):
        return torch.randn(*shape, device=dev).to(bf)

    w, coeff, bias = torch.rand(W, device=dev), torch.rand(4, device=dev), torch.randn(H, 400, device=dev)
    w13, w2, router = rnd(E, 2 * ff, W) * 0.02, rnd(E, W, ff) * 0.02, rnd(E, W) * 0.02
    for tag, B, n, ctx in (("prompts", 4, 2048 if not small else 512, 0), ("single tokens", 16, 1, 2080)):
        T, blocks = B * n, -(-(ctx + n) // 64)
        x, y, z = torch.randn(T, W, device=dev), rnd(T, W), rnd(T, F)
        sec = timeit(lambda: ops.sandwich_rmsnorm(x, y, w, w, 1e-5))
        report("sandwich_rmsnorm_kernel", sec, T * W * 12, tag)
        rows, pos = rnd(T * k, W), torch.randperm(T * k, device=dev).int()
        sec = timeit(lambda: ops.sandwich_rmsnorm(x, (rows, pos), w, w, 1e-5))
        report("sandwich_rmsnorm_kernel (experts' rows)", sec, T * W * (10 + 2 * k), tag)
        res, yy = rnd(T, W), y.clone()
        sec = timeit(lambda: ops.add_rmsnorm(yy, res, w.to(bf), 1e-5))
        report("rmsnorm_kernel (with residual add)", sec, T * W * 8, tag)
        sec = timeit(lambda: ops.poly_norm(z, coeff, F, 1e-5))
        report("poly_norm_kernel", sec, T * F * 4, tag)
        z2 = rnd(T, 2 * F)
        sec = timeit(lambda: ops.act_and_mul(z2, "silu"))
        report("act_and_mul_kernel", sec, T * F * 6, tag)
        proj, gate = rnd(T, (H + 2 * G) * D), rnd(T, H)
        cache = rnd(B * blocks, 2, G, 64, D)
        bt = torch.arange(B * blocks, dtype=torch.int32, device=dev).view(B, blocks)
        p = (torch.arange(T, device=dev) % n) + ctx
        slots = torch.cat([bt[b].long()[p[b * n:(b + 1) * n] // 64] * 64 + p[b * n:(b + 1) * n] % 64 for b in range(B)])
        keep = rnd(T, G * D)
        sec = timeit(lambda: ops.attn_prep_cache(proj[:, :H * D], proj[:, H * D:(H + G) * D], proj[:, (H + G) * D:], cache,
                                                 slots, p, H, G, 1e-5, (0.1, 1024), None, keep, 0.4))
        report("attn_prep_cache_kernel", sec, T * (2 * (H + 2 * G) + G) * D * 2, tag)
        lens = torch.full((B,), ctx + n, dtype=torch.int32, device=dev)
        qsl = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        q, nd = rnd(T, H, D), B if n == 1 else 0
        flops = sum(min(i + 1, ctx + n) for i in range(ctx, ctx + n)) * B * H * D * 4
        for name, b, gt in (("bias and gate", bias, gate), ("neither", None, None)):
            sec = timeit(lambda: ops.paged_attention(q, cache, bt, lens, qsl, 0.09, n, ctx + n, num_decodes=nd,
                                                     num_decode_tokens=nd, bias=b, gate=gt))
            report(f"attention ({name})", sec, B * (ctx + n) * G * D * 4 + T * H * D * 4,
                   f"{tag}; {flops / sec / 1e12:.0f} TFLOP/s of visible scores")
        h = rnd(T, W)
        wt, ids = ops.router_and_route(h, router, None, k, "sigmoid", False, fp32=True)
        sec = timeit(lambda: ops.router_and_route(h, router, None, k, "sigmoid", False, fp32=True))
        report("router + route", sec, T * W * 2 + E * W * 2, tag)
        if n > 1:
            for name, fn in (("fp32 output", lambda: ops.router_gemm(h, router, fp32=True)), ("16-bit output", lambda: ops.linear(h, router))):
                report(f"router GEMM ({name})", timeit(fn), T * W * 2 + E * W * 2, tag)
        touched = min(E, T * k) * 3 * ff * W * 2
        for name, fn in (("weighted inputs", lambda: ops.experts_on_weighted_input(h, w13, w2, wt, ids, "swiglu_limit", 7.0)),
                         ("weighted outputs", lambda: ops.fused_moe(h, w13, w2, wt, ids))):
            sec = timeit(fn)
            report(f"experts ({name})", sec, touched + T * W * 4, f"{tag}; {T * k * 6 * ff * W / sec / 1e12:.0f} TFLOP/s")


def case_postnorm(small):
    """Norms on the sublayers' outputs with convolutions of their inputs, minGRU, sigmoid attention (32 / 8 heads of 128, window of
    1024 and 4 kept keys, or all keys) beside softmax attention, corrected routing, ungated experts: 4 prompts of 2048 tokens, 16
    tokens behind 2080."""
    from vllm_kunlun_b200.attention.metadata import AttentionMetadata
    W, H, G, D, E, I, k, ff, taps = 4096, 32, 8, 128, 28, 4, 4, 1536, 3
    dev, bf = "cuda", torch.bfloat16

    def rnd(*shape):
        return torch.randn(*shape, device=dev).to(bf)

    w, conv_w, corr = torch.rand(W, device=dev), torch.randn(taps, W, device=dev), torch.randn(E + I, device=dev) * 0.01
    up, down, router = rnd(E, ff, W) * 0.02, rnd(E, W, ff) * 0.02, rnd(E + I, W) * 0.02
    qn, pb = torch.rand(D, device=dev), torch.full((H, 1), -3.0, device=dev)
    turns = ops.position_turns(64, 10000.0).to(dev)
    for tag, B, n, ctx in (("prompts", 4, 2048 if not small else 512, 0), ("single tokens", 16, 1, 2080)):
        T, blocks = B * n, -(-(ctx + n) // 64)
        i32 = lambda t: t.to(torch.int32)  # noqa: E731
        p = (torch.arange(T, device=dev) % n) + ctx
        bt = i32(torch.arange(B * blocks, device=dev)).view(B, blocks)
        lens, qsl = i32(torch.full((B,), ctx + n, device=dev)), i32(torch.arange(0, T + 1, n, device=dev))
        idx, init = i32(torch.arange(B, device=dev)), i32(torch.ones(B, device=dev))
        slots = torch.cat([bt[b].long()[p[b * n:(b + 1) * n] // 64] * 64 + p[b * n:(b + 1) * n] % 64 for b in range(B)])
        md = AttentionMetadata(num_tokens=T, num_reqs=B, positions=p, slot_mapping=slots, block_tables=bt, seq_lens=lens,
                               query_start_loc=qsl, max_query_len=n, max_seq_len=ctx + n, state_indices=idx,
                               has_initial_state=init)
        nd = B if n == 1 else 0
        x, y, h = torch.randn(T, W, device=dev), rnd(T, W), rnd(T, W)
        conv = (conv_w, torch.zeros(B, taps - 1, W, device=dev))
        ids = torch.cat([torch.randperm(E + I, device=dev)[:k].view(1, k) for _ in range(T)]).int()
        wt = torch.rand(T, k, device=dev)
        rows, places = ops.expert_rows(h, up, down, ids, "relu2", choices=E + I)
        parts = ops.ChoicesSum(y, rows, places, wt, h)
        kept = 12 * (taps - 1) / n                        # state of a request, read and written
        for name, part, nbytes in (("row", y, 10), ("experts", parts, 10 + 2 * k)):
            if n == 1:
                sec = timeit(lambda: ops.postnorm_input_conv(x, part, w, 1e-5, bf, conv, md))
                report(f"postnorm_kernel with convolution ({name})", sec, T * W * (nbytes + 2 + kept), tag)
            else:
                sec = timeit(lambda: ops._c().postnorm(x, None, *(part if isinstance(part, ops.ChoicesSum) else (part,) + (None,) * 4),
                                                       w, 1e-5, None, None, None, None, None, None))
                report(f"postnorm_kernel ({name})", sec, T * W * nbytes, tag)
        if n > 1:
            report("input_conv_kernel", timeit(lambda: ops.input_conv(x, bf, conv, md)), T * W * 6, tag)
        sec = timeit(lambda: ops.layernorm_residual(x, bf, [(y, 1.0)], w, 1e-5))
        report("layernorm_residual_kernel", sec, T * W * 12, tag)
        z = rnd(T, 3 * W)
        zb, state, out = torch.full((W,), -2.0, device=dev), torch.zeros(B, W, device=dev), torch.empty(T, W, dtype=bf, device=dev)
        sec = timeit(lambda: ops.gated_blend(z[:, :W], z[:, W:2 * W], z[:, 2 * W:], zb, zb, state, qsl, idx, init, out, n, nd))
        report("gated_blend", sec, T * W * 8 + B * W * 8, tag)
        proj, cache = rnd(T, (H + 2 * G) * D), rnd(B * blocks, 2, G, 64, D)
        table = ops.rotary_table(p, turns)
        split = (proj[:, :H * D], proj[:, H * D:(H + G) * D], proj[:, (H + G) * D:])
        sec = timeit(lambda: ops.attn_prep_cache(*split, cache, slots, p, H, G, 1e-5, v_norm=False, qk_norm=(qn, qn), table=table))
        report("attn_prep_cache_kernel (norms, rotation)", sec, 2 * T * (H + 2 * G) * D * 2, tag)
        sec = timeit(lambda: ops.attn_prep_cache(*split, cache, slots, p, H, G, 1e-5))
        report("attn_prep_cache_kernel (value norm)", sec, 2 * T * (H + 2 * G) * D * 2, tag)
        q = rnd(T, H, D)
        for window, keep in ((None, 0), (1024, 4)):
            seen = lambda i: i + 1 if window is None else min(i + 1, window + keep)  # noqa: E731
            flops = sum(seen(i) for i in range(ctx, ctx + n)) * B * H * D * 4
            keys = ctx + n if window is None or n > 1 else window + keep
            for name, kw in (("sigmoid", dict(bias=pb, sigmoid=True, keep_first=keep)), ("softmax", {})):
                sec = timeit(lambda: ops.paged_attention(q, cache, bt, lens, qsl, 0.09, n, keys, window, num_decodes=nd,
                                                         num_decode_tokens=nd, **kw))
                report(f"attention ({name}, window {window})", sec, B * keys * G * D * 4 + T * H * D * 4,
                       f"{tag}; {flops / sec / 1e12:.0f} TFLOP/s of visible scores")
        for name, kw in (("groups, correction", dict(bias=corr, n_group=4, topk_group=2, group_top=1)), ("plain", {})):
            sec = timeit(lambda: ops.router_and_route(h, router, None, k, "softmax", False, fp32=True, **kw))
            report(f"router + route ({name})", sec, T * W * 2 + (E + I) * W * 2, tag)
        touched = min(E, T * k) * 2 * ff * W * 2
        sec = timeit(lambda: ops.expert_rows(h, up, down, ids, "relu2", choices=E + I))
        report("experts (squared relu)", sec, touched + T * W * 2 + T * k * W * 2,
               f"{tag}; {int((places >= 0).sum()) * 4 * ff * W / sec / 1e12:.0f} TFLOP/s")


def case_latent(small):
    """Kernels around latent attention (32 heads, 128 + 64 / 128, latents of 1536 and 512) and the gated fp32 stream of
    width 4096: 4 prompts of 2048 tokens, and 16 single tokens behind a context of 2080."""
    from types import SimpleNamespace
    W, H, Q, C, R, win = (4096, 32, 1536, 512, 64, 1024) if not small else (4096, 32, 1536, 512, 64, 256)
    dev, bf = "cuda", torch.bfloat16

    def rnd(*shape):
        return torch.randn(*shape, device=dev).to(bf)

    w, mix = torch.randn(W, device=dev), torch.rand(W, device=dev)
    table, bigram = rnd(32000, W), rnd(65522, W)
    up = rnd(H * 256, C)
    w_uk, w_uv = up.view(H, 256, C)[:, :128], up.view(H, 256, C)[:, 128:]
    qn, kn, sinks = torch.randn(Q, device=dev), torch.randn(C, device=dev), torch.randn(H, device=dev)
    turns = ops.position_turns(R, 10000.0).to(dev)
    for tag, B, n, ctx in (("prompts", 4, 2048 if not small else 512, 0), ("single tokens", 16, 1, 2080)):
        T, blocks = B * n, -(-(ctx + n) // 64)
        lens = torch.full((B,), ctx + n, dtype=torch.int32, device=dev)
        qsl = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        md = SimpleNamespace(req_id_per_token=torch.arange(B, device=dev).repeat_interleave(n).int(), query_start_loc=qsl,
                             state_indices=torch.arange(B, dtype=torch.int32, device=dev),
                             has_initial_state=torch.full((B,), int(ctx > 0), dtype=torch.int32, device=dev))
        shift = (mix, torch.randn(B, W, device=dev))
        x, y1, y2, g = torch.randn(T, W, device=dev), rnd(T, W), rnd(T, W), rnd(T, 2 * W)
        parts = [(y1, g[:, :W]), (y2, g[:, W:])]
        sec = timeit(lambda: ops.gated_residual_layernorm(x, parts, w, 1e-6, bf, shift, md))
        report("stream_layernorm (gated sum)", sec, T * W * 20, tag)
        ids = torch.randint(0, 32000, (T,), device=dev)
        rows = torch.randint(0, 65521, (T,), device=dev)
        sec = timeit(lambda: ops.embed_stream_layernorm(ids, table, 64.0, (rows, bigram), w, 1e-6, shift, md))
        report("stream_layernorm (embedding)", sec, T * W * 12, tag)
        pos = (torch.arange(T, device=dev) % n) + ctx
        tab = ops.rotary_table(pos, turns)
        cache = rnd(B * blocks, 64, C + R)
        bt = torch.arange(B * blocks, dtype=torch.int32, device=dev).view(B, blocks)
        slots = torch.cat([bt[b].long()[pos[b * n:(b + 1) * n] // 64] * 64 + pos[b * n:(b + 1) * n] % 64 for b in range(B)])
        down = rnd(T, Q + C + R + 32)
        sec = timeit(lambda: ops.latent_prep(down[:, :Q], down[:, Q:Q + C + R], qn, kn, tab, cache, slots, C, Q, 1e-6))
        report("latent_prep", sec, T * (2 * Q + 2 * C + 2 * R) * 2, tag)
        q, gate = rnd(T, H, 192), down[:, Q + C + R:]
        if n > 1:
            sec = timeit(lambda: ops.rotate_heads(q, tab, 128))
            report("rotate_heads", sec, T * H * R * 4, tag)
            starts, klens = qsl[:-1].contiguous(), torch.full((B,), n, dtype=torch.int32, device=dev)
            sec = timeit(lambda: ops.gather_window(cache, bt, lens, starts, klens, T, n))
            report("gather_window", sec, T * (C + R) * 4, tag)
            got = ops.gather_window(cache, bt, lens, starts, klens, T, n)
            kv, out = rnd(T, H * 256), rnd(T, H, 128)
            for name, wd, s in (("window and sinks", win, sinks), ("all positions", None, None)):
                keys = sum(min(i + 1, wd or n) for i in range(n)) * B
                sec = timeit(lambda: ops.mla_prefill_attention(q, kv, got[:, C:], starts, klens, qsl, True, 0.07, n, out=out,
                                                               window=wd, sinks=s, want_lse=False))
                report(f"prefill_umma_kernel (latent, {name})", sec, T * H * 256 * 2,
                       f"{tag}; {keys * H * 640 / sec / 1e12:.0f} TFLOP/s of visible scores")
        else:
            sec = timeit(lambda: ops.absorb_query(q, w_uk, tab, C, C + R))
            report("absorb_query", sec, H * 128 * C * 2 + T * H * (192 + 576) * 2, tag)
            qa = ops.absorb_query(q, w_uk, tab, C, C + R)
            for name, wd, s in (("window and sinks", win, sinks), ("all positions", None, None)):
                sec = timeit(lambda: ops.mla_attention(qa, cache, bt, lens, qsl, 0.07, C, 1, ctx + 1, window=wd, sinks=s))
                report(f"mla_decode_umma_kernel ({name})", sec, B * min(ctx + 1, wd or ctx + 1) * 1152, tag)
            o = rnd(T, H, C)
            sec = timeit(lambda: ops.expand_value(o, w_uv, gate))
            report("expand_value", sec, H * 128 * C * 2 + T * H * (512 + 128) * 2, tag)


def case_conv(small):
    C, W = 8192, 4
    T = 32768 if not small else 4096
    x = torch.randn(T, C, device="cuda").to(torch.bfloat16)
    w = torch.randn(C, W, device="cuda").to(torch.bfloat16)
    R = 16
    cu = (torch.arange(R + 1, device="cuda") * (T // R)).int()
    states = torch.zeros(R, W - 1, C, device="cuda", dtype=torch.bfloat16)
    idx = torch.arange(R, device="cuda").int()
    init = torch.zeros(R, device="cuda").int()
    sec = timeit(lambda: ops.causal_conv1d_fn(x, w, None, cu, states, idx, init, True))
    report("conv1d_fwd_kernel + conv1d_state_kernel", sec, 2 * T * C * 2, f"T={T} C={C}")
    xb = torch.randn(16, C, device="cuda").to(torch.bfloat16)
    sec = timeit(lambda: ops.causal_conv1d_update(xb, states, w, None, idx, True))
    report("conv1d_update_kernel", sec, 2 * 16 * C * 2 + 2 * states.numel() * 2, "B=16")


def case_lora(small):
    K, N, r, L = 4096, 6144, 16, 4
    T = 8192 if not small else 1024
    x = torch.randn(T, K, device="cuda").to(torch.bfloat16)
    A = torch.randn(L, r, K, device="cuda").to(torch.bfloat16)
    Bm = torch.randn(L, N, r, device="cuda").to(torch.bfloat16)
    out = torch.zeros(T, N, device="cuda", dtype=torch.bfloat16)
    # prefill: runs of 512 tokens per adapter; decode-like: an adapter drawn per token
    patterns = (("segments of 512", (torch.arange(T, device="cuda") // 512 % L).int()),
                ("adapter per token", torch.randint(0, L, (T,), device="cuda", dtype=torch.int32)))
    for name, ids in patterns:
        sec = timeit(lambda: ops.lora_shrink(x, A, ids, 1.0))
        report("lora_shrink_kernel", sec, T * K * 2 + T * r * 4, f"T={T} K={K} r={r}, {name}")
        h = ops.lora_shrink(x, A, ids, 1.0)
        sec = timeit(lambda: ops.lora_expand(h, Bm, ids, out, 0, True))
        report("lora_expand_kernel", sec, 2 * T * N * 2 + T * r * 4, f"T={T} N={N} r={r}, {name}")


def case_gemm_splits(small):
    """Decode-sized bf16 GEMMs of an 8B dense model at TP 1-8: default K split against forced 1-8 equal parts."""
    from vllm_kunlun_b200.ops.gemm_cuda import gemm_bf16
    shapes = [("qkv tp8", 768, 4096), ("qkv tp4", 1536, 4096), ("qkv tp2", 3072, 4096), ("qkv tp1", 6144, 4096),
              ("o tp1", 4096, 4096), ("o tp2", 4096, 2048), ("o tp4", 4096, 1024), ("down tp1", 4096, 14336),
              ("down tp2", 4096, 7168), ("down tp4", 4096, 3584), ("down tp8", 4096, 1792),
              ("gate_up tp8", 3584, 4096)]
    for name, N, K in shapes[:3] if small else shapes:
        x = torch.randn(16, K, device="cuda").bfloat16()
        w = (torch.randn(N, K, device="cuda") * 0.05).bfloat16()
        out = torch.empty(16, N, device="cuda", dtype=torch.bfloat16)
        res = {"default": timeit(lambda: gemm_bf16(x, w, None, out), iters=15, warm=4)}
        for sp in (1, 2, 3, 4, 6, 8):
            res[str(sp)] = timeit(lambda: gemm_bf16(x, w, None, out, splits=sp), iters=15, warm=4)
        print(json.dumps({"kernel": "gemm_bf16", "shape": f"16x{N}x{K}", "name": name, "tiles": (N + 127) // 128,
                          "us_by_splits": {k: round(v * 1e6, 1) for k, v in res.items()}}))


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--case", default="all")
    ap.add_argument("--small", action="store_true")
    a = ap.parse_args()
    cases = {"sample": case_sample, "gdn": case_gdn, "recurrence": case_recurrence, "stream": case_stream, "sandwich": case_sandwich,
             "postnorm": case_postnorm, "latent": case_latent, "conv": case_conv, "lora": case_lora}
    explicit = {"gemm_splits": case_gemm_splits}  # not part of "all"
    with torch.inference_mode():
        for n, fn in cases.items():
            if a.case in ("all", n):
                fn(a.small)
        if a.case in explicit:
            explicit[a.case](a.small)
