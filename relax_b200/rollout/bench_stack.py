"""Serving benchmark of composed stacks beside the engine's existing models at equal size (``bench.py --stack-bench``).

Two tables, random weights, bf16, one GPU:

* kernels: device time per launch, algorithmic bytes or FLOPs, fraction of the measured copy bandwidth / cuBLAS rate
  (``--peaks``), each kernel of the composed stack beside the like kernel of the existing models;
* models: prefill and decode tokens/s through the engine's scheduler - a Talizen stack beside the Gated-DeltaNet hybrid and
  the dense softmax model, a Ketolorn stack beside the mixture-of-experts model, a Zupupel stack beside a Ketolorn stack, or a Zoguzen
  stack beside a Zupupel stack, with the same width, heads, feed-forward bytes and depth.

Times come from CUDA events after warm-up; every kernel rotates through inputs larger than the L2 cache.
"""
from __future__ import annotations

import json
import os

import torch

FP32_FMA_PER_CLOCK_SM = 128


def _time(fns, iters=30, warmup=5):
    """Mean ms of one call, cycling through ``fns`` (independent buffers)."""
    for i in range(max(warmup, len(fns))):
        fns[i % len(fns)]()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for i in range(iters):
        fns[i % len(fns)]()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def _copies(nbytes: int) -> int:
    return max(2, min(16, int(3e8 // max(1, nbytes)) + 1))


def _graph(fn):
    """One captured call: launch gaps of the host do not count against a kernel of a few microseconds."""
    fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        fn()
    return lambda: (g.replay(), fn)[0]      # the closure keeps the captured buffers alive


@torch.no_grad()
def kernel_rows(H=32, d=128, R=512, W=4096, F=12288, groups=8, only=""):
    """``(kernel, case, ms, bytes, flops)`` for decode batches and prompts of one real-sized layer."""
    from .. import ops
    from .composed import SegmentBatch, query_blocks, recurrent_spans

    dev, bf = "cuda", torch.bfloat16
    rows = []
    mk = lambda *s: torch.randn(*s, device=dev).to(bf)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    want = lambda section: not only or section in only.split(",")
    for B in (16, 128):
        # recurrent step: the state is read and written once
        sbytes = B * H * d * d * 4
        fb, lo, nw = mk(H * d), torch.rand(H * d, device=dev).to(bf), mk(d)
        ctx = torch.full((B,), 9, dtype=torch.int32, device=dev)
        fns = []
        for _ in range(_copies(2 * sbytes) if want("step") else 0):
            st, x, sl = torch.randn(B, H, d, d, device=dev), mk(B, 3 * H * d), torch.randperm(B, device=dev).to(torch.int32)
            fns.append(_graph(lambda st=st, x=x, sl=sl: ops.hgrn2(x, fb, lo, nw, st, sl, ctx, None, H, d, d, 1e-5)))
        if fns:
            rows.append(("hgrn2_step", f"batch {B}", _time(fns), 2 * sbytes + B * 4 * H * d * 2, None))
        del fns
        for L, page in () if not want("attn") else ((2048, 16), (2048, 64), (8192, 16), (8192, 64)):
            nb = L // page
            bt = torch.randperm(B * nb, device=dev).to(torch.int32).view(B, nb)
            cl = torch.full((B,), L, dtype=torch.int32, device=dev)
            fns = []
            for _ in range(_copies(B * L * R * 2)):
                pool, q, g = mk(B * L, R), mk(B, H, R), mk(B, H)
                b = SegmentBatch(None, None, cl, bt, None, max_ctx=L)
                fns.append(_graph(lambda pool=pool, q=q, g=g, b=b: ops.latent_attention(q, pool, b, page, 0.05, g)))
            rows.append(("latent_attn decode", f"batch {B}, context {L}, pages of {page}", _time(fns), B * L * R * 2, 4.0 * B * L * R * H))
            del fns
            if page != 16:
                continue
            kvh = 8
            fns = []
            for _ in range(_copies(B * L * kvh * d * 4)):
                kc, vc, q = mk(B * nb, 16, kvh, d), mk(B * nb, 16, kvh, d), mk(B, H, d)
                fns.append(_graph(lambda kc=kc, vc=vc, q=q: ops.paged_decode_attention(q, kc, vc, bt, cl)))
            rows.append(("  like: paged decode attention", f"batch {B}, context {L}", _time(fns), B * L * kvh * d * 4, None))
            del fns
        if not want("gemm"):
            continue
        q, o = mk(B, H, d), mk(B, H, R)
        ukc = [mk(H, d, R) for _ in range(_copies(H * d * R * 2))]
        rows.append(("head_gemm fold", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(q, w, False)) for w in ukc]),
                     H * d * R * 2 + B * H * (d + R) * 2, 2.0 * B * H * d * R))
        rows.append(("head_gemm unfold", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(o, w, True)) for w in ukc]),
                     H * d * R * 2 + B * H * (d + R) * 2, 2.0 * B * H * d * R))
        wc = [mk(W, W) for _ in range(_copies(W * W * 2))]
        x = mk(B, W)
        rows.append(("  like: decode GEMM 4096 x 4096", f"batch {B}", _time([_graph(lambda w=w: ops.linear(x, w)) for w in wc]), W * W * 2 + 2 * B * W * 2, None))
        wc = [mk(2 * F, W) for _ in range(2)]
        rows.append(("decode GEMM + gelu unit", f"batch {B}", _time([_graph(lambda w=w: ops.linear_glu(x, w, "gelu_tanh")) for w in wc]), 2 * F * W * 2, None))
        rows.append(("  like: decode GEMM + SwiGLU", f"batch {B}", _time([_graph(lambda w=w: ops.linear_swiglu(x, w)) for w in wc]), 2 * F * W * 2, None))
        del wc
    for T in (128, 8192) if want("norm") else ():
        n = _copies(T * W * 12)
        w = mk(W)
        buf = [(torch.randn(T, W, device=dev), mk(T, W)) for _ in range(n)]
        rows.append(("norm_add (fp32 stream)", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.norm_add(r, y, w, W, groups, 1e-5)) for r, y in buf]), T * W * 12, None))
        b2 = [(mk(T, W), mk(T, W)) for _ in range(n)]
        rows.append(("  like: add_rmsnorm (bf16 stream)", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.add_rmsnorm(y, r, w, 1e-5)) for r, y in b2]), T * W * 8, None))
        del buf, b2
    fb, lo, nw = mk(H * d), torch.rand(H * d, device=dev).to(bf), mk(d)
    for S, L in ((1, 8192), (4, 2048), (32, 256)) if want("prompt") else ():
        T = S * L
        x, st = mk(T, 3 * H * d), torch.zeros(S, H, d, d, device=dev)
        spans = recurrent_spans([L] * S, H)
        spans = None if spans is None else (i32(spans[0]), i32(spans[1]))
        cu, ctx, sl = i32([i * L for i in range(S + 1)]), i32([L] * S), i32(list(range(S)))
        rows.append(("hgrn2 prompt", f"{S} x {L}", _time([lambda: ops.hgrn2(x, fb, lo, nw, st, sl, ctx, cu, H, d, d, 1e-5, spans)], 10), T * H * d * 4 * 2, 6.0 * T * H * d * d))
        q, k, v, g = mk(T, H, d), mk(T, H, d), mk(T, H, d), mk(T, H)
        first, tiles = i32([i * L for i in range(S)]), i32(query_blocks([L] * S, [L] * S, 128))
        rows.append(("flash + gate (prompt)", f"{S} x {L}", _time([lambda: ops.dense_flash(q, k, v, first, tiles, 0.08, g)], 10), T * H * d * 8, 2.0 * T * L * H * d))
        rows.append(("  like: flash attention", f"{S} x {L}", _time([lambda: ops.attention_varlen(q, k, v, cu, True, 0.08, cu, L)], 10), T * H * d * 8, 2.0 * T * L * H * d))
    for n, L in ((4, 2048), (64, 2048)) if want("attn") else ():
        from .composed import attention_items

        S, R_ = 16, R
        nb = L // 16
        bt = torch.randperm(S * nb, device=dev).to(torch.int32).view(S, nb)
        q, pool, g = mk(S * n, H, R_), mk(S * L, R_), mk(S * n, H)
        b = SegmentBatch(None, None, i32([L] * S), bt, None, cu=i32([0]), max_ctx=L, items={H: i32(attention_items([n] * S, [L] * S, H))})
        rows.append(("latent_attn portions", f"{S} x {n} tokens, context {L}", _time([_graph(lambda: ops.latent_attention(q, pool, b, 16, 0.05, g))]),
                     S * L * R_ * 2, 4.0 * S * n * L * R_ * H))
    return rows


@torch.no_grad()
def ketolorn_kernel_rows(W=2048, H=32, G=4, d=128, E=128, k=8, F=1152, only=""):
    """The kernels of one real-sized Ketolorn layer, each beside the like kernel of the existing models."""
    from .. import ops
    from ..models.config import LayerSpec, MoESpec
    from .composed import SegmentBatch, query_blocks, tile_tokens

    dev, bf = "cuda", torch.bfloat16
    rows = []
    mk = lambda *s: torch.randn(*s, device=dev).to(bf)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    want = lambda section: not only or section in only.split(",")
    sink, scale = mk(H), d ** -0.5
    for B in (16, 128) if want("attn") else ():
        for L in (2048, 8192):
            nbytes = B * L * G * d * 4
            cl = torch.full((B,), L, dtype=torch.int32, device=dev)
            for page, like in ((64, False), (16, True)):
                bt = torch.randperm(B * L // page, device=dev).to(torch.int32).view(B, L // page)
                fns = []
                for _ in range(_copies(nbytes)):
                    kc, vc, q = mk(B * L, G, d), mk(B * L, G, d), mk(B, H, d)
                    if like:
                        kv = kc.view(-1, page, G, d), vc.view(-1, page, G, d)
                        fns.append(_graph(lambda q=q, kv=kv: ops.paged_decode_attention(q, *kv, bt, cl)))
                    else:
                        b = SegmentBatch(None, None, cl, bt, None, max_ctx_one=L)
                        fns.append(_graph(lambda q=q, kc=kc, vc=vc, b=b: ops.paged_attention(q, kc, vc, b, page, scale, sink, d)))
                rows.append(("  like: paged decode attention" if like else "attention decode + sink", f"batch {B}, context {L}, pages of {page}", _time(fns), nbytes, None))
                del fns, kc, vc, q
    spec = LayerSpec("attention", heads=H, dim=d, vdim=d, kv_heads=G)
    for S, n, L in ((1, 8192, 8192), (4, 2048, 2048), (32, 256, 256), (16, 64, 2048), (16, 4, 2048)) if want("prompt") else ():
        T, page = S * n, 64
        nb = L // page
        bt = torch.randperm(S * nb, device=dev).to(torch.int32).view(S, nb)
        q, kc, vc = mk(T, H, d), mk(S * L, G, d), mk(S * L, G, d)
        t = tile_tokens(spec)
        b = SegmentBatch(None, None, i32([L] * S), bt, None, cu=i32([i * n for i in range(S + 1)]), multi_segs=S, multi_rows=T,
                         blocks={t: i32(query_blocks([n] * S, [L] * S, t))})
        flops = 4.0 * S * H * d * sum(L - n + i + 1 for i in range(n))
        rows.append(("paged flash + sink", f"{S} x {n} tokens, context {L}", _time([_graph(lambda: ops.paged_attention(q, kc, vc, b, page, scale, sink, d))], 10),
                     T * H * d * 4 + S * L * G * d * 4, flops))
        cq, ck = i32([i * n for i in range(S + 1)]), i32([i * L for i in range(S + 1)])
        rows.append(("  like: flash attention", f"{S} x {n} tokens, context {L}", _time([_graph(lambda: ops.attention_varlen(q, kc, vc, cq, True, scale, ck, n))], 10),
                     T * H * d * 4 + S * L * G * d * 4, flops))
    for T in (128, 8192) if want("prep") else ():
        n = _copies(T * (H + 2 * G) * d * 4)
        freq = torch.tensor([1e6 ** (-2 * i / 64) for i in range(32)], dtype=torch.float64, device=dev)
        pos, slots = torch.arange(T, device=dev).to(torch.int32), torch.randperm(T, device=dev)
        tab, kp, vp = ops.rope_table(pos, 0, freq), mk(T, G, d), mk(T, G, d)
        xs = [mk(T, (H + 2 * G) * d) for _ in range(n)]
        nb = T * (H + 2 * G) * d * 4
        rows.append(("rotation + norm + cache write", f"{T} rows", _time([_graph(lambda x=x: ops.attention_inputs(x, tab, H, G, d, d, d, 64, 1e-6, kp, vp, slots)) for x in xs]), nb, None))
        cos, sin = torch.randn(T, d // 2, device=dev), torch.randn(T, d // 2, device=dev)
        qw, kc, vc = mk(d), kp.view(-1, 16, G, d), vp.view(-1, 16, G, d)
        rows.append(("  like: qkv_post", f"{T} rows", _time([_graph(lambda x=x: ops.qkv_post(x, H, G, qw, qw, cos, sin, 1e-6, kc, vc, slots, False)) for x in xs]), nb, None))
        rows.append(("rope_table (once per forward)", f"{T} rows", _time([_graph(lambda: ops.rope_table(pos, 0, freq))]), T * 32 * 8, None))
        del xs
    moe = MoESpec(experts=E, top=k, ff=F, groups=8, keep=4)
    for T in (1, 16, 128, 8192) if want("moe") else ():
        R, h = T * k, mk(T, W)
        up, down = mk(E, F, W), mk(E, W, F)
        plans = [ops.moe_route(torch.randn(T, E, device=dev), moe, bf) for _ in range(1 if T > 1000 else 4)]      # each touches other experts
        hit = [int((p.offset[1:] > p.offset[:-1]).sum()) for p in plans]
        nb, fl = sum(hit) / len(hit) * 2 * F * W * 2 + R * (2 * W + 2 * F) * 2, 4.0 * R * F * W
        rows.append(("expert products (gather, up, relu^2, down)", f"{T} rows", _time([_graph(lambda p=p: ops.moe_experts(h, p, up, down, "relu2")) for p in plans], 10), nb, fl if T > 1000 else None))
        from ..models.moe import grouped_swiglu_mlp

        w1, w2 = mk(E, 2 * 768, W), mk(E, W, 768)
        sorts = [torch.rand(T, E, device=dev).topk(k, -1).indices for _ in range(len(plans))]
        hit = [x.unique().numel() for x in sorts]
        nb2, fl2 = sum(hit) / len(hit) * 3 * 768 * W * 2 + R * (2 * W + 3 * 768) * 2, 6.0 * R * 768 * W
        rows.append(("  like: grouped SwiGLU experts with their permutation", f"{T} rows",
                     _time([_graph(lambda i=i: grouped_swiglu_mlp(h.repeat_interleave(k, 0), i.reshape(-1), w1, w2)) for i in sorts], 10), nb2, fl2 if T > 1000 else None))
        if T > 1000:      # the products alone: rows laid out beforehand
            cap = R // E // 128 * 128 * E
            x, te = mk(cap, W), torch.arange(E, device=dev).to(torch.int32).repeat_interleave(cap // E // 128)
            er = (torch.arange(E + 1, device=dev) * (cap // E)).to(torch.int32)
            rows.append(("  like: grouped GEMM alone", f"{cap} sorted rows", _time([_graph(lambda: ops.grouped_linear(x, w1, te, er))], 10), cap * (W + 1536) * 2 + E * 1536 * W * 2, 2.0 * cap * 1536 * W))
            y = mk(cap, 768)
            rows.append(("  like: grouped GEMM alone (down)", f"{cap} sorted rows", _time([_graph(lambda: ops.grouped_linear(y, w2, te, er))], 10), cap * (W + 768) * 2 + E * 768 * W * 2, 2.0 * cap * 768 * W))
        z = torch.randn(T, E, device=dev)
        rows.append(("routing and layout of the experts' rows", f"{T} rows", _time([_graph(lambda: ops.moe_route(z, moe, bf))]), T * E * 4 + R * 16, None))
        rows.append(("  like: softmax top-k", f"{T} rows", _time([_graph(lambda: ops.topk_router(z, k))]), T * E * 8 + R * 12, None))
        from ..models.moe import padded_expert_layout

        rows.append(("  like: softmax top-k and padded_expert_layout", f"{T} rows",
                     _time([_graph(lambda: padded_expert_layout(ops.topk_router(z, k)[1].reshape(-1), E))]), T * E * 8 + R * 28, None))
        wr = mk(E, W)
        rows.append(("router logits (fp32)", f"{T} rows", _time([_graph(lambda: ops.linear_fp32(h, wr))]), T * W * 2 + E * W * 2 + T * E * 4, None))
        rows.append(("  like: GEMM of that size", f"{T} rows", _time([_graph(lambda: ops.linear(h, wr))]), T * W * 2 + E * W * 2 + T * E * 2, None))
        del up, down, w1, w2
    for T in (128, 8192) if want("norm") else ():
        n = _copies(T * W * (12 + 2 * k))
        w = mk(W)
        plan = ops.moe_route(torch.randn(T, E, device=dev), moe, bf)
        buf = [(torch.randn(T, W, device=dev), mk(T, W), mk(T * k, W)) for _ in range(n)]
        rows.append(("norm_add with expert rows", f"{T} rows", _time([_graph(lambda r=r, y=y, e=e: ops.norm_add(r, y, w, W, 1, 1e-6, None, (e, plan))) for r, y, e in buf]), T * W * (12 + 2 * k), None))
        rows.append(("norm_add", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.norm_add(r, y, w, W, 1, 1e-6)) for r, y, _ in buf]), T * W * 12, None))
        rows.append(("  like: add_rmsnorm (bf16 stream)", f"{T} rows", _time([_graph(lambda y=y, e=e: ops.add_rmsnorm(y, e[:T], w, 1e-6)) for _, y, e in buf]), T * W * 8, None))
        del buf
    for T in (16, 128, 8192) if want("gemm") else ():
        x = mk(T, W)
        wc = [mk(2 * F, W) for _ in range(_copies(2 * F * W * 2))]
        fl = 4.0 * T * F * W if T > 1000 else None
        rows.append(("GEMM + squared relu (shared expert)", f"{T} rows", _time([_graph(lambda w=w: ops.linear_act(x, w, "relu2")) for w in wc], 10), 2 * F * W * 2 + T * (W + 2 * F) * 2, fl))
        rows.append(("  like: GEMM + SwiGLU", f"{T} rows", _time([_graph(lambda w=w: ops.linear_glu(x, w, "silu")) for w in wc], 10), 2 * F * W * 2 + T * (W + F) * 2, fl))
        del wc
    return rows


@torch.no_grad()
def zupupel_kernel_rows(W=2048, H=32, G=4, d=128, window=1024, R=512, rot=64, E=128, I=16, k=8, F=768, only=""):
    """The kernels of one real-sized Zupupel layer of each kind, each beside the like kernel of Ketolorn or Talizen stacks."""
    from dataclasses import replace

    from .. import ops
    from ..models.config import LayerSpec, MoESpec
    from .composed import SegmentBatch, attention_items, query_blocks, tile_tokens

    dev, bf = "cuda", torch.bfloat16
    rows = []
    mk = lambda *s: torch.randn(*s, device=dev).to(bf)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    want = lambda section: not only or section in only.split(",")
    freq = torch.tensor([1e6 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=dev)
    sink, scale, page = mk(H), d ** -0.5, 64
    for B in (16, 128) if want("attn") else ():
        for L, win in ((8192, window), (window, 0)):
            seen = min(L, window)
            nbytes = B * seen * G * d * 4
            bt = torch.randperm(B * L // page, device=dev).to(torch.int32).view(B, L // page)
            b = SegmentBatch(None, None, torch.full((B,), L, dtype=torch.int32, device=dev), bt, None, max_ctx_one=L)
            fns = []
            for _ in range(_copies(nbytes) if B * L < 1 << 20 else 2):
                kc, vc, q, g = mk(B * L, G, d), mk(B * L, G, d), mk(B, H, d), mk(B, H * d)
                extra = dict(window=win, gate=g) if win else {}
                fns.append(_graph(lambda q=q, kc=kc, vc=vc, extra=extra: ops.paged_attention(q, kc, vc, b, page, scale, None if win else sink, d, **extra)))
            name = f"attention decode, window {win}, gate" if win else "  like: attention decode + sink (Ketolorn)"
            rows.append((name, f"batch {B}, context {L}", _time(fns), nbytes, None))
            del fns, kc, vc, q
    spec = LayerSpec("attention", heads=H, dim=d, vdim=d, kv_heads=G)
    for S, n, L in ((1, 8192, 8192), (4, 2048, 2048), (32, 256, 256), (16, 64, 2048), (16, 4, 2048)) if want("prompt") else ():
        T, nb, t = S * n, L // page, tile_tokens(spec)
        bt = torch.randperm(S * nb, device=dev).to(torch.int32).view(S, nb)
        q, kc, vc, g = mk(T, H, d), mk(S * L, G, d), mk(S * L, G, d), mk(T, H * d)
        b = SegmentBatch(None, None, i32([L] * S), bt, None, cu=i32([i * n for i in range(S + 1)]), multi_segs=S, multi_rows=T,
                         blocks={t: i32(query_blocks([n] * S, [L] * S, t))})
        for win in (window, 0):
            flops = 4.0 * S * H * d * sum(min(win or L, L - n + i + 1) for i in range(n))
            extra = dict(window=win, gate=g) if win else {}
            rows.append((f"paged flash, window {win}, gate" if win else "  like: paged flash + sink (Ketolorn)", f"{S} x {n} tokens, context {L}",
                         _time([_graph(lambda: ops.paged_attention(q, kc, vc, b, page, scale, None if win else sink, d, **extra))], 10),
                         T * H * d * (6 if win else 4) + S * min(L, (win or L) + n) * G * d * 4, flops))
    for B, L in ((16, 2048), (16, 8192), (128, 2048), (128, 8192)) if want("latent") else ():
        bt = torch.randperm(B * L // page, device=dev).to(torch.int32).view(B, L // page)
        b = SegmentBatch(None, None, torch.full((B,), L, dtype=torch.int32, device=dev), bt, None, max_ctx=L)
        for r, name in ((rot, "latent decode, rotated part"), (0, "  like: latent decode + gate (Talizen)")):
            fns = []
            for _ in range(_copies(B * L * (R + r) * 2)):
                pool, q, g = mk(B * L, R + r), mk(B, H, R + r), mk(B, H)
                fns.append(_graph(lambda pool=pool, q=q, g=g, r=r: ops.latent_attention(q, pool, b, page, 0.05, None if r else g, R)))
            rows.append((name, f"batch {B}, context {L}", _time(fns), B * L * (R + r) * 2, None))
            del fns, pool
    for n, L in ((4, 2048), (64, 2048)) if want("latent") else ():
        S = 16
        bt = torch.randperm(S * L // page, device=dev).to(torch.int32).view(S, L // page)
        for r, name in ((rot, "latent portions, rotated part"), (0, "  like: latent portions + gate (Talizen)")):
            width = ops.latent_columns(R + r, R)
            q, pool, g = mk(S * n, H, R + r), mk(S * L, R + r), mk(S * n, H)
            b = SegmentBatch(None, None, i32([L] * S), bt, None, cu=i32([0]), max_ctx=L, items={H: i32(attention_items([n] * S, [L] * S, H, width))},
                             item_width={H: width})
            rows.append((name, f"{S} x {n} tokens, context {L}", _time([_graph(lambda r=r: ops.latent_attention(q, pool, b, page, 0.05, None if r else g, R))]),
                         S * L * (R + r) * 2, 2.0 * S * n * L * (2 * R + r) * H))
    for S, L in ((1, 8192), (4, 2048), (32, 256)) if want("latent") else ():
        T = S * L
        first, tiles = i32([i * L for i in range(S)]), i32(query_blocks([L] * S, [L] * S, 128))
        for r, name in ((rot, "flash of a latent prompt, rotated part, feature gate"), (0, "  like: flash + head gate (Talizen)")):
            q, kk, v, g = mk(T, H, d + r), mk(T, H, d + r), mk(T, H, d), mk(T, H * d if r else H)
            rows.append((name, f"{S} x {L}", _time([_graph(lambda r=r: ops.dense_flash(q, kk, v, first, tiles, 0.08, g, bool(r)))], 10),
                         T * H * (4 * d + 2 * r) * 2, 1.0 * S * L * (L + 1) * H * (2 * d + r)))
    for T in (16, 128, 8192) if want("prep") else ():
        n = _copies(T * (H + 2 * G) * d * 4)
        pos, slots = torch.arange(T, device=dev).to(torch.int32), torch.randperm(T, device=dev)
        tab, kp, vp, qw, kw = ops.rope_table(pos, 0, freq), mk(T, G, d), mk(T, G, d), mk(H * d), mk(G * d)
        xs = [mk(T, (H + 2 * G) * d) for _ in range(n)]
        nb = T * (H + 2 * G) * d * 4
        rows.append(("projection norms + rotation + cache write", f"{T} rows",
                     _time([_graph(lambda x=x: ops.projection_inputs(x, qw, kw, tab, H, G, d, d, d, rot, True, 1e-6, kp, vp, slots)) for x in xs]), nb, None))
        rows.append(("  like: rotation + head norm + cache write (Ketolorn)", f"{T} rows",
                     _time([_graph(lambda x=x: ops.attention_inputs(x, tab, H, G, d, d, d, rot, 1e-6, kp, vp, slots)) for x in xs]), nb, None))
        del xs
        pool, w = mk(T, R + rot), mk(R)
        xs = [mk(T, H * (d + rot) + R + rot) for _ in range(n)]
        parts = lambda x: x.split([H * (d + rot), R, rot], 1)
        rows.append(("latent row: norm, rotation, queries' rotation", f"{T} rows",
                     _time([_graph(lambda x=x: ops.latent_write(parts(x)[1], w, R, 1e-6, pool, slots, (parts(x)[0].view(T, H, d + rot), parts(x)[2], tab, R, rot, d)))
                            for x in xs]), T * (R * 4 + rot * 4 + H * rot * 4), None))
        plain = mk(T, R)
        rows.append(("  like: latent row: norm (Talizen)", f"{T} rows", _time([_graph(lambda x=x: ops.latent_write(parts(x)[1], w, R, 1e-6, plain, slots)) for x in xs]),
                     T * R * 4, None))
        del xs
    for B in (16, 128) if want("gemm") else ():
        x, o, g = mk(B, H, d + rot), mk(B, H, R), mk(B, H * d)
        wide, narrow = [mk(H, d + rot, R + rot) for _ in range(_copies(H * d * R * 2))], [mk(H, d, R) for _ in range(_copies(H * d * R * 2))]
        alg = H * d * R * 2 + B * H * (d + R + 2 * rot) * 2      # (the identity rows of the key map are not counted)
        rows.append(("head_gemm fold with the rotated part", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(x, w, False)) for w in wide]), alg, None))
        y = x[..., :d].contiguous()
        rows.append(("  like: head_gemm fold (Talizen)", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(y, w, False)) for w in narrow]),
                     H * d * R * 2 + B * H * (d + R) * 2, None))
        rows.append(("head_gemm unfold + feature gate", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(o, w, True, g)) for w in narrow]),
                     H * d * R * 2 + B * H * (2 * d + R) * 2, None))
        rows.append(("  like: head_gemm unfold (Talizen)", f"batch {B}", _time([_graph(lambda w=w: ops.head_linear(o, w, True)) for w in narrow]),
                     H * d * R * 2 + B * H * (d + R) * 2, None))
    mine = MoESpec(experts=E, top=k, ff=F, groups=8, keep=4, act="clamped_swish", limit=7.0, renormalize=True, score="softmax", correction=True, identity=I,
                   group_best=1)
    like = MoESpec(experts=E, top=k, ff=F * 3 // 2, groups=8, keep=4)
    corr = torch.zeros(E + I, device=dev, dtype=bf)
    route = lambda spec, z: ops.moe_route(z, spec, bf, None, corr if spec.correction else None)
    for T in (1, 16, 128, 8192) if want("moe") else ():
        h = mk(T, W)
        for spec, name in ((mine, "gated expert products (gather, both halves, unit, down)"), (like, "  like: squared-relu expert products (Ketolorn)")):
            up, down = mk(E, 2 * F if spec.gated else F * 3 // 2, W), mk(E, W, spec.ff)
            plans = [route(spec, torch.randn(T, spec.outputs, device=dev)) for _ in range(1 if T > 1000 else 4)]      # each touches other experts
            hit = [int((p.offset[1:] > p.offset[:-1]).sum()) for p in plans]
            used = sum(int(p.offset[-1]) for p in plans) / len(plans)
            nb = sum(hit) / len(hit) * 3 * F * W * 2 + used * (2 * W + 2 * spec.ff) * 2
            rows.append((name, f"{T} rows ({used:.0f} expert rows)",
                         _time([_graph(lambda p=p: ops.moe_experts(h, p, up, down, spec.act, spec.limit)) for p in plans], 10), nb,
                         6.0 * used * F * W if T > 1000 else None))
            del up, down
        for spec, name in ((mine, "routing (softmax, correction, identity) and layout"), (like, "  like: routing and layout (Ketolorn)")):
            z = torch.randn(T, spec.outputs, device=dev)
            rows.append((name, f"{T} rows", _time([_graph(lambda: route(spec, z))]), T * spec.outputs * 4 + T * k * 16, None))
    for T in (16, 128, 8192) if want("norm") else ():
        n = _copies(T * W * (12 + 2 * k))
        w, bias = mk(W), mk(W)
        plans = {s: route(s, torch.randn(T, s.outputs, device=dev)) for s in (mine, replace(like, shared_ff=8))}
        buf = [(torch.randn(T, W, device=dev), mk(T, W), mk(T * k, W)) for _ in range(n)]
        pm, pl = plans.values()
        used = int(pm.offset[-1])
        rows.append(("sum_norm with expert rows", f"{T} rows", _time([_graph(lambda r=r, e=e: ops.sum_norm(r, None, w, bias, W, 1.5, 1e-6, None, 1.0, (e, pm))) for r, _, e in buf]),
                     T * W * 10 + used * W * 2, None))
        rows.append(("  like: norm_add with expert rows (Ketolorn)", f"{T} rows",
                     _time([_graph(lambda r=r, e=e: ops.norm_add(r, None, w, W, 1, 1e-6, None, (e, pl))) for r, _, e in buf]), T * W * (10 + 2 * k), None))
        rows.append(("sum_norm", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.sum_norm(r, y, w, bias, W, 1.5, 1e-6)) for r, y, _ in buf]), T * W * 12, None))
        rows.append(("  like: norm_add", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.norm_add(r, y, w, W, 1, 1e-6)) for r, y, _ in buf]), T * W * 12, None))
        rows.append(("sum_norm and the final norm", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.sum_norm(r, y, w, bias, W, 1.5, 1e-6, (w, bias), 0.1)) for r, y, _ in buf]),
                     T * W * 12, None))
        rows.append(("  like: norm_add and the final norm", f"{T} rows", _time([_graph(lambda r=r, y=y: ops.norm_add(r, y, w, W, 1, 1e-6, w)) for r, y, _ in buf]),
                     T * W * 12, None))
        del buf
    return rows


def zoguzen_kernel_rows(W=2048, H=32, G=4, d=128, chunk=1024, Hl=16, Hr=16, dk=64, width=4096, side=256, E=128, k=8, F=768, only=""):
    """The kernels of one real-sized Zoguzen layer of each kind, each beside the like kernel of Zupupel or Talizen stacks."""
    from .. import ops
    from ..models.config import LayerSpec, MoESpec
    from .composed import ComposedForward, SegmentBatch, query_blocks, recurrent_spans, tile_tokens

    dev, bf = "cuda", torch.bfloat16
    rows = []
    mk = lambda *s: torch.randn(*s, device=dev).to(bf)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    want = lambda section: not only or section in only.split(",")
    one, talk, scale, page = torch.zeros(H, device=dev, dtype=bf), mk(H, H), d ** -0.5, 64
    chunked = dict(chunk=chunk, softcap=30.0, talk=talk)
    for B in (16, 128) if want("attn") else ():
        L = 8 * chunk
        bt = torch.randperm(B * L // page, device=dev).to(torch.int32).view(B, L // page)
        b = SegmentBatch(None, None, torch.full((B,), L, dtype=torch.int32, device=dev), bt, None, max_ctx_one=L)
        for heads, name, kw, s in ((H, "attention decode, chunk, cap, mixed heads", chunked, one), (H, "  like: attention decode, window, gate (Zupupel)", dict(window=chunk), None),
                                   (Hl, "attention decode, window, first tokens, gate", dict(window=chunk, keep=16), None),
                                   (Hl, "  like: attention decode, window, gate (Zupupel)", dict(window=chunk), None)):
            fns = []
            for _ in range(2 if B * L >= 1 << 20 else _copies(B * chunk * G * d * 4)):
                kc, vc, q, g = mk(B * L, G, d), mk(B * L, G, d), mk(B, heads, d), mk(B, heads * d)
                extra = dict(kw, gate=None if "talk" in kw else g)
                fns.append(_graph(lambda q=q, kc=kc, vc=vc, extra=extra, s=s: ops.paged_attention(q, kc, vc, b, page, scale, s, d, **extra)))
            rows.append((name, f"batch {B}, {heads} heads, {chunk} of {L} positions", _time(fns), B * chunk * G * d * 4, None))
            del fns, kc, vc, q
    for S, n, L in ((1, 8192, 8192), (4, 2048, 2048), (32, 256, 256), (16, 64, 2048), (16, 4, 2048)) if want("prompt") else ():
        T, nb = S * n, L // page
        bt = torch.randperm(S * nb, device=dev).to(torch.int32).view(S, nb)
        for heads, name, kw, s in ((H, "paged flash, chunk, cap, mixed heads", chunked, one), (H, "  like: paged flash, window, gate (Zupupel)", dict(window=chunk), None),
                                   (Hl, "paged flash, window, first tokens, gate", dict(window=chunk, keep=16), None),
                                   (Hl, "  like: paged flash, window, gate (Zupupel)", dict(window=chunk), None)):
            t = tile_tokens(LayerSpec("attention", heads=heads, dim=d, vdim=d, kv_heads=G))
            q, kc, vc, g = mk(T, heads, d), mk(S * L, G, d), mk(S * L, G, d), mk(T, heads * d)
            b = SegmentBatch(None, None, i32([L] * S), bt, None, cu=i32([i * n for i in range(S + 1)]), multi_segs=S, multi_rows=T,
                             blocks={t: i32(query_blocks([n] * S, [L] * S, t))})
            mixes = "talk" in kw
            seen = lambda p: p % chunk + 1 if mixes else min(chunk, p + 1)
            pairs = S * heads * sum(seen(L - n + i) for i in range(n))
            extra = dict(kw, gate=None if mixes else g)
            rows.append((name, f"{S} x {n} tokens, context {L}, {heads} heads", _time([_graph(lambda: ops.paged_attention(q, kc, vc, b, page, scale, s, d, **extra))], 10),
                         T * heads * d * (4 if mixes else 6) + S * min(L, chunk + n) * G * d * 4, pairs * (4.0 * d + (2.0 * heads if mixes else 0.0))))
    rot, freq = d, torch.tensor([1e6 ** (-2 * i / d) for i in range(d // 2)], dtype=torch.float64, device=dev)
    for T in (16, 128, 8192) if want("prep") else ():
        C = (H + 2 * G) * d
        n = _copies(T * C * 4)
        pos, slots = torch.arange(T, device=dev).to(torch.int32), torch.randperm(T, device=dev)
        tab, kp, vp, qw, kw, bias, taps = ops.rope_table(pos, 0, freq), mk(T, G, d), mk(T, G, d), mk(H * d), mk(G * d), mk(C), mk(C, 4)
        if T > 1000:
            b = SegmentBatch(None, slots, i32([T // 4] * 4), None, i32([0, 1, 2, 3]), cu=i32([i * T // 4 for i in range(5)]),
                             seg_of=(torch.arange(T, device=dev) // (T // 4)).to(torch.int32), pos=(torch.arange(T, device=dev) % (T // 4)).to(torch.int32))
        else:
            b = SegmentBatch(None, slots, i32([900] * T), None, torch.arange(T, device=dev).to(torch.int32))
        xs, nb = [mk(T, C) for _ in range(n)], T * C * 4
        state = mk(T if T < 1000 else 4, 3, C)
        rows.append(("bias, convolution, head norm, cache write", f"{T} rows", _time([_graph(lambda x=x: ops.conv_inputs(
            x, bias, taps, state, b, qw[:d], kw[:d], None, H, G, d, d, d, 0, 1e-6, kp, vp)) for x in xs]), nb + (T * 6 * C * 2 if T < 1000 else 0), None))
        rows.append(("convolution, rotation, cache write", f"{T} rows", _time([_graph(lambda x=x: ops.conv_inputs(
            x, None, taps, state, b, None, None, tab, H, G, d, d, d, rot, 0.0, kp, vp)) for x in xs]), nb + (T * 6 * C * 2 if T < 1000 else 0), None))
        rows.append(("  like: projection norms, rotation, cache write (Zupupel)", f"{T} rows",
                     _time([_graph(lambda x=x: ops.projection_inputs(x, qw, kw, tab, H, G, d, d, d, rot, True, 1e-6, kp, vp, slots)) for x in xs]), nb, None))
        del xs, state
    gla = LayerSpec("gla", heads=Hr, dim=dk, vdim=d, decay_rank=16)
    at = ComposedForward.gla_columns(gla)
    zb, zw, fb, lower, nw = mk(width), mk(width), mk(Hr * dk), torch.rand(Hr * dk, device=dev).to(bf), mk(d)
    for B in (16, 128) if want("step") else ():
        ids, ctx = torch.arange(B, device=dev).to(torch.int32), i32([900] * B)
        n = _copies(B * Hr * dk * d * 8)
        states = [torch.randn(B, Hr, dk, d, device=dev) for _ in range(n)]
        x, z, q = mk(B, at["end"]), torch.randn(B, Hr * dk, device=dev), mk(B, Hr * (2 * dk + d))
        nb = B * Hr * dk * d * 8
        rows.append(("linear attention step", f"batch {B}", _time([_graph(lambda s=s: ops.gla(x, z, fb, nw, s, ids, ctx, None, Hr, dk, d, at["g"], 1e-6, 16.0)) for s in states]),
                     nb, None))
        rows.append(("  like: hgrn2 step (Talizen)", f"batch {B}", _time([_graph(lambda s=s: ops.hgrn2(q, fb, lower, nw, s, ids, ctx, None, Hr, dk, d, 1e-6)) for s in states]),
                     nb, None))
        del states
        n = _copies(B * width * 16)
        states, xs = [torch.randn(B, 1, 1, width, device=dev) for _ in range(n)], [mk(B, 3 * width) for _ in range(n)]
        b = SegmentBatch(None, None, ctx, None, ids)
        rows.append(("running mean step", f"batch {B}", _time([_graph(lambda s=s, x=x: ops.mingru(x, zb, zw, s, b, width)) for s, x in zip(states, xs)]), B * width * 16, None))
        del states, xs
    for S, L in ((1, 8192), (4, 2048), (32, 256)) if want("step") else ():
        T = S * L
        cu, ids, ctx = i32([i * L for i in range(S + 1)]), torch.arange(S, device=dev).to(torch.int32), i32([L] * S)
        both = lambda c: None if c is None else (i32(c[0]), i32(c[1]))
        spans = both(recurrent_spans([L] * S, Hr))
        state, x, z, q = torch.zeros(S, Hr, dk, d, device=dev), mk(T, at["end"]), torch.randn(T, Hr * dk, device=dev), mk(T, Hr * (2 * dk + d))
        rows.append(("linear attention of a prompt", f"{S} x {L}", _time([_graph(lambda: ops.gla(x, z, fb, nw, state, ids, ctx, cu, Hr, dk, d, at["g"], 1e-6, 16.0, spans))], 10),
                     T * (at["a1"] * 2 + Hr * (dk * 4 + d * 2)), 6.0 * T * Hr * dk * d))
        rows.append(("  like: hgrn2 of a prompt (Talizen)", f"{S} x {L}", _time([_graph(lambda: ops.hgrn2(q, fb, lower, nw, state, ids, ctx, cu, Hr, dk, d, 1e-6, spans))], 10),
                     T * Hr * (2 * dk + 2 * d) * 2, 6.0 * T * Hr * dk * d))
        xs, mean = [mk(T, 3 * width) for _ in range(2)], torch.zeros(S, 1, 1, width, device=dev)
        b = SegmentBatch(None, None, ctx, None, ids, cu=cu)
        rows.append(("running mean of a prompt", f"{S} x {L}", _time([_graph(lambda x=x: ops.mingru(x, zb, zw, mean, b, width)) for x in xs], 10), T * width * 8, None))
        del xs
    mine = MoESpec(experts=E, top=k, ff=F, act="swiglu", score="softmax", renormalize=True)
    like = MoESpec(experts=E, top=k, ff=F, groups=8, keep=4, act="clamped_swish", limit=7.0, renormalize=True, score="softmax", correction=True, group_best=1)
    corr = torch.zeros(E, device=dev, dtype=bf)
    route = lambda spec, z: ops.moe_route(z, spec, bf, None, corr if spec.correction else None)
    for T in (1, 16, 128, 8192) if want("moe") else ():
        h, up, down = mk(T, W), mk(E, 2 * F, W), mk(E, W, F)
        zs = [torch.randn(T, E, device=dev) for _ in range(1 if T > 1000 else 4)]      # each touches other experts
        for spec, name in ((mine, "expert products (gather, both halves, silu unit, down)"), (like, "  like: bounded units (Zupupel)")):
            plans = [route(spec, z) for z in zs]
            hit = sum(int((p.offset[1:] > p.offset[:-1]).sum()) for p in plans) / len(plans)
            rows.append((name, f"{T} rows", _time([_graph(lambda p=p: ops.moe_experts(h, p, up, down, spec.act, spec.limit)) for p in plans], 10),
                         hit * 3 * F * W * 2 + T * k * (2 * W + 2 * F) * 2, 6.0 * T * k * F * W if T > 1000 else None))
        for spec, name in ((mine, "routing and layout"), (like, "  like: routing and layout, groups and correction (Zupupel)")):
            rows.append((name, f"{T} rows", _time([_graph(lambda: route(spec, zs[0]))]), T * E * 4 + T * k * 16, None))
        del up, down
    for T in (16, 128, 8192) if want("norm") else ():
        n = _copies(T * W * (12 + 2 * k))
        w, mu, bias = mk(W), mk(W), mk(W)
        plan, other = (route(s, torch.randn(T, E, device=dev)) for s in (mine, like))
        buf = [(torch.randn(T, W, device=dev), mk(T, W), mk(T, W), mk(T * k, W)) for _ in range(n)]
        many = T > 1000
        b = SegmentBatch(None, None, i32([T // 4] * 4) if many else i32([900] * T), None, torch.arange(4 if many else T, device=dev).to(torch.int32),
                         cu=i32([i * T // 4 for i in range(5)]) if many else None, seg_of=(torch.arange(T, device=dev) // max(1, T // 4)).to(torch.int32))
        state = mk(4 if many else T, W)
        run = lambda f: _time([_graph(lambda a=a: f(*a)) for a in buf])
        rows.append(("stream step: mixer, expert rows", f"{T} rows", run(lambda r, y, _, e: ops.stream_step(r, W, 1e-6, [y], None, (e, plan))), T * W * (12 + 2 * k), None))
        rows.append(("stream step: pair of normed mixers, expert rows", f"{T} rows", run(lambda r, y, x, e: ops.stream_step(r, W, 1e-6, [y, x], (w, bias), (e, plan))),
                     T * W * (14 + 2 * k), None))
        rows.append(("stream step: second embedding, two norms, shift", f"{T} rows", run(lambda r, y, _, e: ops.stream_step(r, W, 1e-6, [y], (w,), None, (w, bias), (mu, state, b))),
                     T * W * (18 if many else 18), None))
        rows.append(("  like: sum_norm with expert rows (Zupupel)", f"{T} rows", run(lambda r, y, _, e: ops.sum_norm(r, y, w, bias, W, 1.5, 1e-6, None, 1.0, (e, other))),
                     T * W * (12 + 2 * k), None))
        rows.append(("  like: sum_norm and the final norm (Zupupel)", f"{T} rows", run(lambda r, y, _, e: ops.sum_norm(r, y, w, bias, W, 1.5, 1e-6, (w, bias), 0.1)), T * W * 12, None))
        ids, table = torch.randint(0, 64000, (T,), device=dev), mk(64000, 4 * side)
        zs = [mk(T, side) for _ in range(n)]
        rows.append(("second embedding: gelu and product", f"{T} rows", _time([_graph(lambda z=z: ops.side_gate(z, table, ids, side, side)) for z in zs]), T * side * 6, None))
        xs = [mk(T, 2 * side) for _ in range(n)]
        rows.append(("  like: gated unit", f"{T} rows", _time([_graph(lambda x=x: ops.glu(x, "gelu_tanh")) for x in xs]), T * side * 6, None))
        if not many:
            zs = [torch.randn(T, 64000, device=dev) for _ in range(_copies(T * 64000 * 8))]
            rows.append(("capped logits", f"{T} rows of 64000", _time([_graph(lambda z=z: ops.softcap(z, 30.0)) for z in zs]), T * 64000 * 8, None))
        del buf, zs, xs
    return rows


def _zoguzen_models(layers: int, W: int, H: int, G: int, experts: int, top: int, ff: int, vocab: int):
    """A Zoguzen stack and a Zupupel stack of the same width, heads, window, depth and experts."""
    from ..models.config import LayerSpec, MoESpec, chunk_mean_pair_layers, composed_config

    d = 128
    att = LayerSpec("attention", heads=H, dim=d, vdim=d, kv_heads=G, scale=d ** -0.5, chunk=1024, softcap=30.0, unit_sink=True, talk=True, qkv_bias=True, conv=4,
                    head_norm=True)
    pair = LayerSpec("pair", pair=(LayerSpec("attention", heads=H // 2, dim=d, vdim=d, kv_heads=G, scale=d ** -0.5, window=1024, keep_first=16, rot_dims=d, rot_base=5e5,
                                             rot_scaling=(8.0, 1.0, 4.0, 8192.0), conv=4, out_gate=True),
                                   LayerSpec("gla", heads=H // 2, dim=64, vdim=d, decay_rank=16, decay_root=16.0)))
    mine = MoESpec(experts=experts, top=top, ff=ff, act="swiglu", score="softmax", renormalize=True)
    return {"zoguzen": composed_config("zoguzen", chunk_mean_pair_layers(layers, att, LayerSpec("mingru", vdim=2 * W), pair, mine), W, vocab, pre_norm=True,
                                       token_shift=True, side_dim=256, logit_softcap=30.0, tie_word_embeddings=True),
            "zupupel": _zupupel_models(layers, W, H, G, experts, top, ff, vocab)["zupupel"]}


def _zupupel_models(layers: int, W: int, H: int, G: int, experts: int, top: int, ff: int, vocab: int):
    """A Zupupel stack and a Ketolorn stack with experts of the same bytes in every layer (no shared expert)."""
    from dataclasses import replace

    from ..models.config import LayerSpec, MoESpec, composed_config, window_latent_layers

    d = 128
    att = LayerSpec("attention", heads=H, dim=d, vdim=d, kv_heads=G, scale=d ** -0.5, rot_dims=64, rot_base=1e6)
    lat = LayerSpec("latent_attention", heads=H, dim=d, vdim=d, kv_rank=512, scale=192 ** -0.5, rot_dims=64, rot_base=1e6, out_gate=True)
    mine = MoESpec(experts=experts, top=top, ff=ff, groups=8, keep=4, act="clamped_swish", limit=7.0, renormalize=True, score="softmax", correction=True,
                   identity=experts // 8, group_best=1)
    like = MoESpec(experts=experts, top=top, ff=ff * 3 // 2, groups=8, keep=4)
    return {"zupupel": composed_config("zupupel", window_latent_layers(layers, replace(att, rot_halves=True, proj_norm=True, window=1024, out_gate=True), lat, mine), W,
                                       vocab, norm_sum=True, sum_alpha=2.0, embed_scale=W ** 0.5, logit_scale=W ** -0.5),
            "ketolorn": composed_config("ketolorn", [replace(att, qk_norm=True, sink=True, moe=like) for _ in range(layers)], W, vocab, embed_norm=True)}


def _ketolorn_models(layers: int, W: int, H: int, G: int, experts: int, top: int, ff: int, dense_ff: int, vocab: int):
    """A Ketolorn stack (squared-relu experts of 3 / 2 the width: the same bytes as gated ones) and the mixture-of-experts model."""
    from ..models.config import LayerSpec, ModelConfig, MoESpec, composed_config, shared_kv_layers

    d = 128
    att = LayerSpec("attention", heads=H, dim=d, vdim=d, kv_heads=G, scale=d ** -0.5, rot_dims=64, rot_base=1e6, qk_norm=True, sink=True, act="silu")
    moe = MoESpec(experts=experts, top=top, ff=ff * 3 // 2, groups=8, keep=4, shared_ff=ff * 3)
    return {"ketolorn": composed_config("ketolorn", shared_kv_layers(layers, layers // 2, att, dense_ff, moe), W, vocab, embed_norm=True, tie_word_embeddings=True),
            "mixture of experts": ModelConfig(name="moe", num_layers=layers, hidden_size=W, num_attention_heads=H, num_query_groups=G, head_dim=d,
                                              ffn_hidden_size=dense_ff, vocab_size=vocab, num_experts=experts, moe_top_k=top, moe_ffn_hidden_size=ff,
                                              moe_first_dense_layers=1, moe_shared_expert_ffn=2 * ff, moe_router_score="sigmoid",
                                              tie_word_embeddings=True)}


def _models(layers: int, W: int, H: int, ff: int, vocab: int):
    from ..models.config import LayerSpec, ModelConfig, composed_config, talizen_layers

    d = 128
    rec = LayerSpec("hgrn2", heads=H, dim=d, vdim=d, ff=ff)
    att = LayerSpec("latent_attention", heads=H, dim=d, vdim=d, kv_rank=512, scale=d ** -0.5, ff=ff)
    common = dict(num_layers=layers, hidden_size=W, num_attention_heads=H, num_query_groups=H // 4, head_dim=d, ffn_hidden_size=ff, vocab_size=vocab)
    return {"talizen": composed_config("talizen", talizen_layers(layers, 4, rec, att), W, vocab, norm_groups=8),
            "gdn hybrid": ModelConfig(name="gdn-hybrid", linear_attention_freq=4, gdn_k_heads=H, gdn_v_heads=H, gdn_head_dim=d, **common),
            "dense softmax": ModelConfig(name="dense", **common)}


@torch.no_grad()
def model_rows(size: str, only=None, decode_batches=(1, 32, 128), prompt=2048, design="talizen"):
    """``(model, workload, tokens/s, ms)`` through ``RolloutEngine.step``."""
    from .engine import RolloutEngine, SamplingParams

    if design == "zoguzen":
        models = _zoguzen_models(*{"1b": (8, 2048, 32, 4, 128, 8, 768), "5b": (8, 4096, 64, 8, 128, 8, 1536)}[size], 64000)
    elif design == "zupupel":
        models = _zupupel_models(*{"1b": (9, 2048, 32, 4, 128, 8, 768), "5b": (9, 4096, 64, 8, 128, 8, 1536)}[size], 64000)
    elif design == "ketolorn":
        models = _ketolorn_models(*{"1b": (8, 2048, 32, 4, 128, 8, 768, 6144), "5b": (8, 4096, 64, 8, 128, 8, 1536, 12288)}[size], 64000)
    else:
        models = _models(*{"1b": (8, 2048, 16, 8192), "5b": (8, 4096, 32, 12288)}[size], 64000)
    out = []
    for name, cfg in models.items():
        if only and name not in only:
            continue
        slow = name == "gdn hybrid"
        page = 64 if cfg.is_composed else 16
        eng = RolloutEngine(cfg, device="cuda", dtype=torch.bfloat16, num_kv_blocks=(max(decode_batches) + 8) * (prompt + 256) // page,
                            block_size=page, max_running=136,
                            max_model_len=prompt + 256, memory_saver=False)
        eng.weights.flat.normal_(0, 0.02)
        if design in ("zupupel", "zoguzen"):      # rows of unit size and no bias of the choice: tokens spread over the experts
            for key, t in eng.weights.p.items():
                if key.endswith(("norm", "norm1", "norm2")):
                    t.fill_(1.0)
                elif key.endswith(("norm_b", "moe_correction")):
                    t.zero_()
        g = torch.Generator().manual_seed(0)
        prm = lambda n: torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist()

        def run(fn):
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            return a.elapsed_time(b)

        for S, L in ((1, 8192 if not slow else 2048), (4, 2048), (32, 256)):
            if L > eng.max_model_len and S * L > eng.bm.num_free * page:
                continue
            ps = [prm(L) for _ in range(S)]
            go = lambda: eng.generate(ps, SamplingParams(max_new_tokens=1, ignore_eos=True))
            go()
            ms = min(run(go) for _ in range(1 if slow else 3))
            out.append((name, f"prefill {S} x {L}", S * L / ms * 1e3, ms))
        for B in decode_batches:
            for _ in range(B):
                eng.add_request(prm(prompt), SamplingParams(max_new_tokens=160, ignore_eos=True))
            while any(not r.output for r in eng.running) or eng.waiting:
                eng.step()
            eng.step()                                     # warm-up window (captures the step)
            n0 = eng.stats["decode_tokens"]
            ms = run(lambda: [eng.step() for _ in range(3)])
            n = eng.stats["decode_tokens"] - n0
            out.append((name, f"decode batch {B}, context {prompt}", n / ms * 1e3, ms * B / n))
            eng.abort_all()
        eng.close()
        del eng
        torch.cuda.empty_cache()
    return out


def main(size: str = "5b", peaks: str = "MEASURED_PEAKS.json", kernels: bool = True, models: bool = True, only: str = "", design: str = "talizen") -> int:
    from ..ops import cuda as C

    assert C.available()
    pk = json.load(open(peaks)) if os.path.exists(peaks) else {}
    hbm, tf = pk.get("hbm_gbs"), pk.get("bf16_tflops")
    if kernels:
        print("kernel | case | us | GB/s (of measured copy) | TFLOP/s (of measured GEMM)")
        for k, case, ms, nb, fl in {"talizen": kernel_rows, "ketolorn": ketolorn_kernel_rows, "zupupel": zupupel_kernel_rows, "zoguzen": zoguzen_kernel_rows}[design](only=only):
            gb = nb / ms / 1e6
            t = f"{gb:7.0f}" + (f" ({gb / hbm:.2f})" if hbm else "")
            if fl:
                v = fl / ms / 1e9
                t += f" | {v:7.1f}" + (f" ({v / tf:.2f})" if tf else "")
            print(f"{k} | {case} | {ms * 1e3:.1f} | {t}", flush=True)
    if models:
        for name, what, tps, ms in model_rows(size, design=design):
            print(f"[{size}] {name} | {what} | {tps:,.0f} tokens/s | {ms:.3f} ms", flush=True)
    C.check_error_flag()
    return 0


if __name__ == "__main__":
    import argparse

    ap = argparse.ArgumentParser(description="kernel table of composed stacks")
    ap.add_argument("--design", choices=["talizen", "ketolorn", "zupupel", "zoguzen"], default="talizen")
    ap.add_argument("--only", default="", help="sections, with commas: step, attn, gemm, norm, prompt (talizen); attn, prompt, prep, moe, norm, gemm (ketolorn); "
                                               "attn, prompt, latent, prep, gemm, moe, norm (zupupel); attn, prompt, prep, step, moe, norm (zoguzen)")
    ap.add_argument("--peaks", default="MEASURED_PEAKS.json")
    a = ap.parse_args()
    raise SystemExit(main(peaks=a.peaks, models=False, only=a.only, design=a.design))
