"""Serving benchmark of composed stacks beside the engine's existing models at equal size (``bench.py --stack-bench``).

Two tables, random weights, bf16, one GPU:

* kernels: device time per launch, algorithmic bytes or FLOPs, fraction of the measured copy bandwidth / cuBLAS rate
  (``--peaks``), each kernel of the composed stack beside the like kernel of the existing models;
* models: prefill and decode tokens/s through the engine's scheduler - a Talizen stack, the Gated-DeltaNet hybrid and
  the dense softmax model with the same width, heads, feed-forward and depth.

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
    from .composed import SegmentBatch, recurrent_spans

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
        rows.append(("flash + gate (prompt)", f"{S} x {L}", _time([lambda: ops.flash_gated(q, k, v, cu, cu, 0.08, L, g)], 10), T * H * d * 8, 2.0 * T * L * H * d))
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
def model_rows(size: str, only=None, decode_batches=(1, 32, 128), prompt=2048):
    """``(model, workload, tokens/s, ms)`` through ``RolloutEngine.step``."""
    from .engine import RolloutEngine, SamplingParams

    layers, W, H, ff = {"1b": (8, 2048, 16, 8192), "5b": (8, 4096, 32, 12288)}[size]
    out = []
    for name, cfg in _models(layers, W, H, ff, 64000).items():
        if only and name not in only:
            continue
        slow = name == "gdn hybrid"
        page = 64 if cfg.is_composed else 16
        eng = RolloutEngine(cfg, device="cuda", dtype=torch.bfloat16, num_kv_blocks=(max(decode_batches) + 8) * (prompt + 256) // page,
                            block_size=page, max_running=136,
                            max_model_len=prompt + 256, memory_saver=False)
        eng.weights.flat.normal_(0, 0.02)
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


def main(size: str = "5b", peaks: str = "MEASURED_PEAKS.json", kernels: bool = True, models: bool = True, only: str = "") -> int:
    from ..ops import cuda as C

    assert C.available()
    pk = json.load(open(peaks)) if os.path.exists(peaks) else {}
    hbm, tf = pk.get("hbm_gbs"), pk.get("bf16_tflops")
    if kernels:
        print("kernel | case | us | GB/s (of measured copy) | TFLOP/s (of measured GEMM)")
        for k, case, ms, nb, fl in kernel_rows(only=only):
            gb = nb / ms / 1e6
            t = f"{gb:7.0f}" + (f" ({gb / hbm:.2f})" if hbm else "")
            if fl:
                v = fl / ms / 1e9
                t += f" | {v:7.1f}" + (f" ({v / tf:.2f})" if tf else "")
            print(f"{k} | {case} | {ms * 1e3:.1f} | {t}", flush=True)
    if models:
        for name, what, tps, ms in model_rows(size):
            print(f"[{size}] {name} | {what} | {tps:,.0f} tokens/s | {ms:.3f} ms", flush=True)
    C.check_error_flag()
    return 0


if __name__ == "__main__":
    import argparse

    ap = argparse.ArgumentParser(description="kernel table of composed stacks")
    ap.add_argument("--only", default="", help="sections, with commas: step, attn, gemm, norm, prompt")
    ap.add_argument("--peaks", default="MEASURED_PEAKS.json")
    raise SystemExit(main(peaks=ap.parse_args().peaks, models=False, only=ap.parse_args().only))
