"""Autograd wrappers around the in-tree sm_100a extension (``relax_b200/_C.so``).

Importing this module on a machine with a GPU but without the built extension
raises: CUDA tensors never fall back to library kernels silently.
"""
from __future__ import annotations

import importlib.util
import math
import os
from typing import Optional

import torch

_SO = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "_C.so")
_SO_SERVING = _SO.replace("_C.so", "_C_serving.so")      # serving subset (ops/build.py)
_C = None
_ERR: dict = {}
_MN_OK: Optional[bool] = None


def _load(path: Optional[str] = None):
    """The extension module: the full one, else the serving subset (whose missing operators raise when called)."""
    global _C
    if _C is not None:
        return _C
    so = path or (_SO if os.path.exists(_SO) else _SO_SERVING)
    if not os.path.exists(so):
        raise RuntimeError(f"{_SO} is missing: build it with `python __graft_entry__.py` (nvcc, sm_100a)")
    spec = importlib.util.spec_from_file_location("relax_b200." + os.path.basename(so)[:-3], so)
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    if os.environ.get("RELAX_B200_CRASH_TRACE", "0") == "1":
        mod.install_crash_handler()
    _C = mod
    return mod


def available() -> bool:
    if not torch.cuda.is_available():
        return False
    _load()
    return True


def err_flag(device=None) -> torch.Tensor:
    dev = torch.device(device if device is not None else torch.cuda.current_device())
    if dev.type != "cuda":
        dev = torch.device("cuda", torch.cuda.current_device())
    idx = dev.index if dev.index is not None else torch.cuda.current_device()
    if idx not in _ERR:
        _ERR[idx] = torch.zeros(1, dtype=torch.int32, device=f"cuda:{idx}")
    return _ERR[idx]


def check_error_flag(device=None):
    """Raise if any kernel recorded an error status (e.g. a bounded wait that ran out)."""
    f = err_flag(device)
    v = int(f.item())
    if v != 0:
        f.zero_()
        raise RuntimeError(f"sm_100a kernel reported error status {v} (1 = barrier wait timed out, 3 = peer wait timed out)")


# --------------------------------------------------------------------------- GEMM


_PAIR = os.environ.get("RELAX_B200_GEMM_PAIR", "1") == "1"


def gemm_raw(a, b, out, M, N, K, lda, ldb, ldc, a_mn=False, b_mn=False, accumulate=False, bias=None, force_bn=0,
             lbo_a=0, sbo_a=0, lbo_b=0, sbo_b=0, pair=None):
    """One GEMM launch.  Problems with at least one full 256-row pair tile go to the CTA-pair kernel
    (csrc/gemm2_sm100.cu: ``cta_group::2``, TMA-store / TMA-reduce epilogue); the rest, and anything with a bias,
    a forced tile width or a non-default descriptor, to the single-CTA kernel (csrc/gemm_sm100.cu)."""
    L = _load()
    use_pair = _PAIR if pair is None else pair
    if (use_pair and bias is None and force_bn == 0 and M >= 256 and N >= 128 and a.dtype == torch.bfloat16
            and not (lbo_a or sbo_a or lbo_b or sbo_b) and (out.dtype == torch.float32 or not accumulate)):
        if L.gemm_pair(a, b, out, M, N, K, lda, ldb, ldc, a_mn, b_mn, accumulate, 256 if N >= 256 else 128,
                       err_flag(a.device)):
            return out
    L.gemm(a, b, out, bias, M, N, K, lda, ldb, ldc, a_mn, b_mn, accumulate, force_bn, lbo_a, sbo_a, lbo_b, sbo_b,
           err_flag(a.device))
    return out


def _rowmajor_2d(t):
    """Return (tensor, ld) such that the tensor is a row-major matrix with 16-byte aligned pitch."""
    if t.stride(-1) != 1 or t.stride(0) % 8 or t.stride(0) < t.shape[1] or t.data_ptr() % 16:
        t = t.contiguous()
        if t.shape[1] % 8:
            raise ValueError(f"GEMM operand inner dimension {t.shape[1]} must be a multiple of 8")
    return t, t.stride(0)


def mn_major_ok() -> bool:
    """One-time numerical self-check of the MN-major (transposed operand) tensor-core path
    against the K-major path on explicitly transposed copies."""
    global _MN_OK
    if _MN_OK is None:
        if os.environ.get("RELAX_B200_DISABLE_MN_MAJOR", "0") == "1":
            _MN_OK = False
            return False
        g = torch.Generator(device="cuda").manual_seed(1)
        M, N, K = 256, 192, 320
        at = torch.randn(K, M, device="cuda", generator=g).bfloat16()   # A stored transposed
        bt = torch.randn(K, N, device="cuda", generator=g).bfloat16()
        ref = torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
        gemm_raw(at.t().contiguous(), bt.t().contiguous(), ref, M, N, K, K, K, N)
        out = torch.empty_like(ref)
        gemm_raw(at, bt, out, M, N, K, M, N, N, a_mn=True, b_mn=True)
        _MN_OK = bool(torch.allclose(out.float(), ref.float(), atol=1e-2, rtol=1e-2))
    return _MN_OK


def matmul_nt(x, w, bias=None, out_dtype=None, out=None, accumulate=False):
    """x[M,K] @ w[N,K]^T."""
    x, lda = _rowmajor_2d(x)
    w, ldb = _rowmajor_2d(w)
    M, K = x.shape
    N = w.shape[0]
    if out is None:
        out = torch.empty(M, N, dtype=out_dtype or x.dtype, device=x.device)
    return gemm_raw(x, w, out, M, N, K, lda, ldb, out.stride(0), bias=bias, accumulate=accumulate)


def matmul_nn(a, b, out=None, out_dtype=None):
    """a[M,K] @ b[K,N]  (b row-major: the MN-major B operand)."""
    a, lda = _rowmajor_2d(a)
    M, K = a.shape
    N = b.shape[1]
    if out is None:
        out = torch.empty(M, N, dtype=out_dtype or a.dtype, device=a.device)
    if mn_major_ok() and N % 8 == 0:
        b, ldb = _rowmajor_2d(b)
        return gemm_raw(a, b, out, M, N, K, lda, ldb, out.stride(0), b_mn=True)
    bt = b.t().contiguous()
    return gemm_raw(a, bt, out, M, N, K, lda, bt.stride(0), out.stride(0))


def matmul_tn(a, b, out=None, out_dtype=None, accumulate=False):
    """a[K,M]^T @ b[K,N] -> [M,N]  (both operands MN-major: weight gradients)."""
    K, M = a.shape
    N = b.shape[1]
    if out is None:
        out = torch.empty(M, N, dtype=out_dtype or a.dtype, device=a.device)
    if mn_major_ok() and M % 8 == 0 and N % 8 == 0:
        a, lda = _rowmajor_2d(a)
        b, ldb = _rowmajor_2d(b)
        return gemm_raw(a, b, out, M, N, K, lda, ldb, out.stride(0), a_mn=True, b_mn=True, accumulate=accumulate)
    at, bt = a.t().contiguous(), b.t().contiguous()
    return gemm_raw(at, bt, out, M, N, K, at.stride(0), bt.stride(0), out.stride(0), accumulate=accumulate)


class _Linear(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, w, bias):
        ctx.save_for_backward(x, w)
        ctx.has_bias = bias is not None
        return matmul_nt(x, w, bias)

    @staticmethod
    def backward(ctx, dy):
        x, w = ctx.saved_tensors
        dy = dy.contiguous()
        dx = matmul_nn(dy, w) if ctx.needs_input_grad[0] else None
        dw = None
        if ctx.needs_input_grad[1]:
            mg = getattr(w, "main_grad", None)
            if mg is not None and mg.dtype == torch.float32 and mg.shape == w.shape and mg.stride(-1) == 1:
                # weight-gradient GEMM accumulates straight into the fp32 gradient buffer of the
                # distributed optimizer: no temporary, no separate add pass
                matmul_tn(dy, x, out=mg, accumulate=True)
            else:
                dw = matmul_tn(dy, x)
        db = dy.sum(0) if ctx.has_bias and ctx.needs_input_grad[2] else None
        return dx, dw, db


def linear(x, w, bias=None):
    shp = x.shape
    x2 = x.reshape(-1, shp[-1])
    if x2.dtype == torch.float32 and w.dtype == torch.float32 and not torch.is_grad_enabled():
        y = torch.empty(x2.shape[0], w.shape[0], dtype=torch.float32, device=x.device)      # 32-bit inference: CUDA cores, true fp32
        _load().simt_gemm(x2[None], w[None], y[None], False)
        return (y if bias is None else y + bias).reshape(*shp[:-1], w.shape[0])
    if x2.dtype not in (torch.bfloat16, torch.float16):
        raise TypeError("the sm_100a GEMM takes bf16/fp16 inputs (fp32 in inference only)")
    if w.dim() != 2:
        raise ValueError("weight must be 2-D")
    if x2.shape[0] <= 256 and not (torch.is_grad_enabled() and (x2.requires_grad or w.requires_grad)) \
            and w.is_contiguous() and w.shape[0] % 64 == 0:
        y = matmul_nt_skinny(x2, w, bias)
        bias = None
    elif not w.is_contiguous() and w.t().is_contiguous():
        # y = x @ (w^T stored row-major)  ->  NN product
        y = _LinearNN.apply(x2, w.t())
    else:
        y = _Linear.apply(x2, w, bias)
        bias = None
    if bias is not None:
        y = y + bias
    return y.reshape(*shp[:-1], y.shape[-1])


_DECODE_GEMM = os.environ.get("RELAX_B200_DECODE_GEMM", "1") == "1"


GLU_ACT = {"silu": 1, "gelu_tanh": 2}


def _decode_gemm(x, w, glu_act: int):
    """Weight-streaming decode GEMM (csrc/gemm_decode_sm100.cu) when the shape is in its range, else None.  ``glu_act``: 0 none,
    1 and 2 gated units (:data:`GLU_ACT`), 3 squared relu without a gate, 4 fp32 results."""
    if not _DECODE_GEMM or x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or x.shape[0] > 128:
        return None     # above 128 rows the 2-stage ring of the 256-column variant loses to the other paths (measured)
    if w.stride(1) != 1 or w.stride(0) % 8 or w.data_ptr() % 16:
        return None
    N = w.shape[0]
    out = torch.empty(x.shape[0], N // 2 if glu_act in (1, 2) else N, dtype=torch.float32 if glu_act == 4 else x.dtype, device=x.device)
    if _load().decode_gemm(x, w, out, glu_act, 0, err_flag(x.device)):
        return out
    return None


def _wide_pair_gemm(x, w):
    """129..256 token rows against a wide weight (N >= 6144: at least 24 pair tiles of 256 x 256): one row of CTA-pair
    tiles of the training GEMM beats split-K here (measured on B200 at 160 and 256 rows: 33 vs 52 us at N = 12288,
    31 vs 50 us at N = 6144; below that split-K wins).  Returns None when the shape is outside that range."""
    M, K = x.shape
    N = w.shape[0]
    if not (_PAIR and 128 < M <= 256 and N >= 6144 and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16
            and w.is_contiguous()):
        return None
    out = torch.empty(M, N, dtype=x.dtype, device=x.device)
    if _load().gemm_pair(x, w, out, M, N, K, x.stride(0), w.stride(0), N, False, False, False, 256, err_flag(x.device)):
        return out
    return None


def matmul_nt_skinny(x, w, bias=None, residual=None):
    """x[M, K] @ w[N, K]^T for decode (a few hundred rows at most): when the N tiles alone cannot fill the SMs the
    reduction dimension is split across CTAs (fp32 partials in a workspace, one small reduce
    kernel that also adds bias / residual)."""
    x, _ = _rowmajor_2d(x)
    M, K = x.shape
    N = w.shape[0]
    C = _load()
    if bias is None and residual is None:
        y = _decode_gemm(x, w, 0)
        if y is None:
            y = _wide_pair_gemm(x, w)
        if y is not None:
            return y
    splits, bn = C.gemm_splitk_plan(M, N, K)
    out = torch.empty(M, N, dtype=x.dtype, device=x.device)
    if splits <= 1:
        gemm_raw(x, w, out, M, N, K, x.stride(0), w.stride(0), N, bias=bias)
        return out if residual is None else out + residual
    ws = torch.empty(splits * M * N, dtype=torch.float32, device=x.device)
    C.gemm_splitk(x, w, out, bias, residual, ws, splits, bn, err_flag(x.device))
    return out


def linear_swiglu_skinny(x, w):
    """``swiglu(x @ w.T)`` for decode (``w`` = [gate; up] rows): split-K partial sums, then ONE kernel that
    reduces them and applies the activation, instead of reduce + swiglu."""
    x, _ = _rowmajor_2d(x)
    M, K = x.shape
    N = w.shape[0]
    C = _load()
    y = _decode_gemm(x, w, 1)
    if y is not None:
        return y
    y = _wide_pair_gemm(x, w)
    if y is not None:
        return swiglu(y)
    splits, bn = C.gemm_splitk_plan(M, N, K)
    if splits <= 1 or x.dtype != torch.bfloat16 or (N // 2) % 4:
        return swiglu(linear(x, w))
    ws = torch.empty(splits * M * N, dtype=torch.float32, device=x.device)
    C.gemm_splitk_partial(x, w, ws, splits, bn, err_flag(x.device))
    out = torch.empty(M, N // 2, dtype=x.dtype, device=x.device)
    C.splitk_swiglu(ws, out, splits)
    return out


def glu(gate_up, act: str = "silu"):
    """``act(gate) * up`` on ``[gate | up]`` rows (inference only)."""
    gu = gate_up.reshape(-1, gate_up.shape[-1])
    out = torch.empty(gu.shape[0], gu.shape[1] // 2, dtype=gu.dtype, device=gu.device)
    _load().glu(gu, out, GLU_ACT[act] - 1)
    return out.reshape(*gate_up.shape[:-1], out.shape[1])


def linear_glu(x, w, act: str = "silu"):
    """``glu(x @ w.T)``: the activation joins the decode GEMM's reduction for up to 128 rows."""
    if x.dtype == torch.bfloat16 and x.shape[0] <= 128:
        x, _ = _rowmajor_2d(x)
        y = _decode_gemm(x, w, GLU_ACT[act])
        if y is not None:
            return y
    return glu(linear(x, w), act)


def linear_relu2(x, w):
    """``relu(x @ w.T) ** 2``: the activation joins the decode GEMM's reduction for up to 128 rows."""
    if x.dtype == torch.bfloat16 and x.shape[0] <= 128:
        x, _ = _rowmajor_2d(x)
        y = _decode_gemm(x, w, 3)
        if y is not None:
            return y
    y = linear(x, w)
    _load().relu2(y)
    return y


def linear_fp32(x, w):
    """``x @ w.T`` with fp32 results from bf16 (or fp32) operands."""
    if x.dtype == torch.float32:
        return linear(x, w)
    x, ld = _rowmajor_2d(x)
    y = _decode_gemm(x, w, 4)
    return matmul_nt(x, w, out_dtype=torch.float32) if y is None else y


# --------------------------------------------------------------------------- composed stacks (inference)


def embed_rows(tokens, w, norm_w=None, width=0, groups=1, eps=0.0, scale=1.0):
    res = torch.empty(tokens.shape[0], w.shape[1], dtype=torch.float32, device=w.device)
    h = torch.empty(tokens.shape[0], w.shape[1], dtype=w.dtype, device=w.device)
    if norm_w is None:
        _load().embed_rows(tokens, w, res, h, float(scale))
    else:
        _load().embed_norm(tokens, w, norm_w, res, h, int(width), int(groups), float(eps))
    return res, h


def norm_add(res, y, w, width, groups, eps, next_w=None, experts=None):
    h = torch.empty(res.shape, dtype=w.dtype, device=w.device)
    if experts is None:
        _load().norm_add(res, y, w, next_w, h, int(width), int(groups), float(eps))
    else:
        rows, plan = experts
        _load().norm_add_experts(res, y, rows, plan.expert, plan.place, plan.offset, plan.weight, w, next_w, h, int(width), int(groups), float(eps))
    return h


def sum_norm(res, y, w, b, width, alpha, eps, nxt=None, scale=1.0, experts=None):
    h = torch.empty(res.shape, dtype=w.dtype, device=w.device)
    rows, plan = experts if experts is not None else (None, None)
    e = (None,) * 4 if plan is None else (plan.expert, plan.place, plan.offset, plan.weight)
    _load().sum_norm(res, y, rows, *e, w, b, *(nxt if nxt is not None else (None, None)), h, int(width), b is not None, float(alpha), float(eps),
                     float(scale))
    return h


def rope_table(positions, offset, inv_freq):
    out = torch.empty(positions.shape[0], inv_freq.shape[0], 2, dtype=torch.float32, device=positions.device)
    _load().rope_table(positions, int(offset), inv_freq, out)
    return out


def attention_inputs(qkv, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps, k_pool, v_pool, slots):
    q = torch.empty(qkv.shape[0], heads, dp, dtype=qkv.dtype, device=qkv.device)
    _load().attention_inputs(qkv, table, q, k_pool, v_pool, slots, int(kv_heads), int(dim), int(vdim), int(rot_dims), float(eps))
    return q


def projection_inputs(qkv, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, halves, eps, k_pool, v_pool, slots):
    q = torch.empty(qkv.shape[0], heads, dp, dtype=qkv.dtype, device=qkv.device)
    _load().projection_inputs(qkv, q_w, k_w, table, q, k_pool, v_pool, slots, int(kv_heads), int(dim), int(vdim), int(rot_dims), bool(halves), float(eps))
    return q


def conv_inputs(qkv, bias, taps, state, b, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps, k_pool, v_pool):
    q = torch.empty(qkv.shape[0], heads, dp, dtype=qkv.dtype, device=qkv.device)
    _load().conv_inputs(qkv, bias, taps, state, q_w, k_w, table, q, k_pool, v_pool, b.slots, b.ctx, b.state_slot, b.cu, b.seg_of, b.pos, int(kv_heads),
                        int(dim), int(vdim), int(rot_dims), float(eps))
    return q


def decode_splits(rows: int, kv_heads: int, max_ctx: int) -> int:
    """Parts of the context that run side by side: enough CTAs to fill the machine twice, at least 512 positions each, none
    when the batch alone fills it."""
    ctas, splits = rows * kv_heads, 1
    if ctas >= 148:
        return 1
    while ctas * splits < 296 and (max_ctx + splits - 1) // splits > 512 and splits < 32:
        splits *= 2
    return splits


def paged_attention(q, k_pool, v_pool, b, block_size, scale, sink, out_width, window=0, gate=None, keep=0, chunk=0, softcap=0.0, talk=None):
    """bf16 heads of up to 128 features: segments of several rows on the flash kernel, single rows on the decode kernel (the
    flash kernel when more than 16 heads share keys); anything else, and fp32, on CUDA cores."""
    if talk is not None:
        return _mixed_attention(q, k_pool, v_pool, b, block_size, scale, sink, out_width, window, keep, chunk, softcap, talk)
    T, H, dp = q.shape
    G = k_pool.shape[1]
    L, err = _load(), err_flag(q.device)
    out = torch.empty(T, H * out_width, dtype=q.dtype, device=q.device)
    n, s = (0, 0) if b.cu is None else (b.multi_rows, b.multi_segs)
    see = (int(window), int(keep), int(chunk))

    def tensor_cores() -> bool:
        if n and not L.paged_flash(q[:n], k_pool, v_pool, b.block_tables, b.ctx, b.blocks[128 // (H // G)], sink, None if gate is None else gate[:n], out[:n],
                                   int(block_size), *see, False, float(scale), float(softcap), err):
            return False
        if n == T:
            return True
        bt, ctx, g = b.block_tables[s:], b.ctx[s:], None if gate is None else gate[n:]
        if H // G > 16:
            return L.paged_flash(q[n:], k_pool, v_pool, bt, ctx, None, sink, g, out[n:], int(block_size), *see, False, float(scale), float(softcap), err)
        most = _most_seen(b.max_ctx_one, block_size, *see)
        splits = decode_splits(T - n, G, most)
        po = ml = None
        if splits > 1:
            po = torch.empty(splits * (T - n) * H * 128, dtype=torch.float32, device=q.device)
            ml = torch.empty(splits * (T - n) * H * 2, dtype=torch.float32, device=q.device)
        return L.paged_decode(q[n:], k_pool, v_pool, bt, ctx, sink, g, out[n:], po, ml, int(block_size), int(most), *see, splits, float(scale),
                              float(softcap), err)

    if not (q.dtype == torch.bfloat16 and max(dp, v_pool.shape[2]) <= 128 and H // G <= 128 and tensor_cores()):
        L.gqa_attn(q, k_pool, v_pool, b.block_tables, b.seg_of, b.pos, b.ctx, sink, gate, out, int(block_size), *see, False, float(scale), float(softcap))
    return out


def _most_seen(max_ctx: int, page: int, window: int, keep: int, chunk: int) -> int:
    """Most positions that a single row sees, pages that count in part as a whole."""
    return min(max_ctx, chunk + page if chunk else window + keep + 2 * page if window else max_ctx)


def _mixed_attention(q, k_pool, v_pool, b, block_size, scale, sink, out_width, window, keep, chunk, softcap, talk):
    """Heads whose weights are mixed: ``sum_g T[h, g] (P_g V) = (sum_g T[h, g] P_g) V``, so every head's weights meet the values of every
    group, and the outputs are mixed (single rows: when the splits are merged).  Capped scores (caps up to 80) have kernels that keep
    several groups' accumulators; the others take the flash kernel once per group."""
    T, H, dp = q.shape
    G, dv = k_pool.shape[1], v_pool.shape[2]
    L, err = _load(), err_flag(q.device)
    out = torch.empty(T, H * out_width, dtype=q.dtype, device=q.device)
    n, s = (0, 0) if b.cu is None else (b.multi_rows, b.multi_segs)
    see, fl = (int(window), int(keep), int(chunk)), (float(scale), float(softcap))
    tensor = q.dtype == torch.bfloat16 and max(dp, dv) <= 128 and H // G <= 128
    done = T                                     # rows that are still to do: in front of here
    if tensor and n < T and 0 < softcap <= 80:
        cols, groups = L.talk_decode_plan(H, G, dp, dv)
        if cols:
            most = _most_seen(b.max_ctx_one, block_size, *see)
            splits = max(1, min(148 // ((T - n) * -(-G // groups)), -(-most // 128)))      # one CTA per SM; tiles of 128 positions
            po = torch.empty((T - n) * splits * G * cols * 128, dtype=torch.float32, device=q.device)
            pl = torch.empty((T - n) * splits * cols, dtype=torch.float32, device=q.device)
            if L.talk_decode(q[n:], k_pool, v_pool, b.block_tables[s:], b.ctx[s:], sink, talk, out[n:], po, pl, int(block_size), int(most), *see, splits, *fl, err):
                done = n
    if done == 0:
        return out
    wide = torch.empty(done, H * G * out_width, dtype=q.dtype, device=q.device)

    def flash(lo, hi, bt, ctx, blocks) -> bool:
        a = (q[lo:hi], k_pool, v_pool, bt, ctx, blocks, sink)
        if 0 < softcap <= 80 and L.talk_flash(*a, wide[lo:hi], int(block_size), *see, *fl, err):
            return True
        return L.paged_flash(*a, None, wide[lo:hi], int(block_size), *see, True, *fl, err)

    if not (tensor and (n == 0 or flash(0, n, b.block_tables, b.ctx, b.blocks[128 // (H // G)])) and
            (done == n or flash(n, done, b.block_tables[s:], b.ctx[s:], None))):
        if done < T:      # (single rows are done, the segments of several rows are not)
            L.gqa_attn(q[:n], k_pool, v_pool, b.block_tables, b.seg_of[:n], b.pos[:n], b.ctx, sink, None, wide, int(block_size), *see, True, *fl)
        else:
            L.gqa_attn(q, k_pool, v_pool, b.block_tables, b.seg_of, b.pos, b.ctx, sink, None, wide, int(block_size), *see, True, *fl)
    L.mix_heads(wide, talk, out[:done], G)
    return out


class ExpertPlan:
    """Device description of one layer's routing: per row and choice ``expert``, ``weight`` and ``place`` (its row among the expert's
    rows), the token of every expert row, the experts' first sorted rows, and the tile list of the grouped GEMMs."""
    __slots__ = ("expert", "weight", "place", "row_token", "offset", "tiles", "n_tiles")


def route_counters(layers, experts, device):
    return torch.zeros(layers, experts + 1, dtype=torch.int32, device=device)


def moe_route(logits, spec, tile_rows, count=None, correction=None):
    T, E, k, dev = logits.shape[0], spec.experts, spec.top, logits.device
    p = ExpertPlan()
    i32 = lambda *s: torch.empty(*s, dtype=torch.int32, device=dev)
    p.expert, p.place, p.row_token, p.offset, p.n_tiles = i32(T, k), i32(T, k), i32(E, T), i32(E + 1), i32(1)
    p.weight = torch.empty(T, k, dtype=torch.float32, device=dev)
    p.tiles = i32(min(T * k, E) + T * k // tile_rows, 4)
    if count is None:
        count = route_counters(1, E, dev)[0]
    _load().moe_route(logits, correction, p.expert, p.weight, p.place, p.row_token, count, p.offset, p.tiles, p.n_tiles, E, spec.outputs, spec.groups,
                      spec.keep, spec.group_best, tile_rows, bool(spec.renormalize), spec.score == "softmax", float(spec.weight_scale))
    return p


def _moe_plan(rows: int, experts: int, n: int) -> tuple:
    """``(columns per tile, whether most tiles have many rows)``: wide tiles when they fill the machine twice (measured)."""
    tiles = min(rows, experts) + rows // 128
    return (256 if tiles * ((n + 255) // 256) >= 296 else 128), rows >= 16 * experts


EXPERT_ACT = {"relu2": 1, "clamped_swish": 2, "swiglu": 3}


def moe_experts(h, plan, up, down, act, limit=0.0):
    """Sorted expert rows ``[T top, W]``: gather, up-projection and activation in one grouped GEMM, down-projection in a second.
    Gated experts: ``up`` holds gate and up rows in alternating runs (:func:`relax_b200.ops.glu_rows`)."""
    R, E, err, code = plan.expert.numel(), up.shape[0], err_flag(h.device), EXPERT_ACT[act]
    mid = torch.empty(R, up.shape[1] // (2 if code >= 2 else 1), dtype=h.dtype, device=h.device)
    out = torch.empty(R, down.shape[1], dtype=h.dtype, device=h.device)
    L = _load()
    L.moe_gemm(h, up, mid, plan.tiles, plan.n_tiles, plan.row_token, code, float(limit), *_moe_plan(R, E, up.shape[1]), err)
    L.moe_gemm(mid, down, out, plan.tiles, plan.n_tiles, None, 0, 0.0, *_moe_plan(R, E, down.shape[1]), err)
    return out


def hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, eps, spans=None):
    T = qfv.shape[0]
    sp, first = spans if spans is not None else (None, None)
    out = torch.empty(T, (heads * vdim + 7) // 8 * 8, dtype=qfv.dtype, device=qfv.device)
    st = gt = None
    if sp is not None and qfv.dtype == torch.bfloat16:
        st = torch.empty(sp.shape[0], *state.shape[1:], dtype=torch.float32, device=qfv.device)
        gt = torch.empty(sp.shape[0], heads, dim, dtype=torch.float32, device=qfv.device)
    run = lambda raw: _load().hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, raw, sp, first, st, gt, out, int(dim),
                                    int(vdim), float(eps))
    if (cu is None or qfv.dtype == torch.bfloat16) and run(None):      # decode step, or segments on the tensor cores
        return out
    run(torch.empty(T, heads, vdim, dtype=torch.float32, device=qfv.device))      # 32-bit mode and head sizes of odd shape
    return out


def mingru(zxg, z_b, x_b, state, b, width):
    out = torch.empty(zxg.shape[0], (width + 7) // 8 * 8, dtype=zxg.dtype, device=zxg.device)
    _load().mingru(zxg, z_b, x_b, state, b.state_slot, b.ctx, b.cu, out, int(width))
    return out


def gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, gate_col, eps, root, spans=None):
    T = rows.shape[0]
    sp, first = spans if spans is not None else (None, None)
    out = torch.empty(T, (heads * vdim + 7) // 8 * 8, dtype=rows.dtype, device=rows.device)
    st = gt = None
    if sp is not None and rows.dtype == torch.bfloat16:
        st = torch.empty(sp.shape[0], *state.shape[1:], dtype=torch.float32, device=rows.device)
        gt = torch.empty(sp.shape[0], heads, dim, dtype=torch.float32, device=rows.device)
    run = lambda raw: _load().gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, raw, sp, first, st, gt, out, int(dim), int(vdim), int(gate_col),
                                  float(eps), float(root))
    if (cu is None or rows.dtype == torch.bfloat16) and run(None):      # decode step, or segments on the tensor cores
        return out
    run(torch.empty(T, heads, vdim, dtype=torch.float32, device=rows.device))      # 32-bit mode and head sizes of odd shape
    return out


def stream_step(res, width, eps, y=None, norm_w=None, experts=None, norms=(), shift=None):
    dt = norms[0].dtype if norms else y[0].dtype
    h = [torch.empty(res.shape, dtype=dt, device=res.device) for _ in norms or (None,)]
    rows, plan = experts if experts is not None else (None, None)
    e = (None,) * 4 if plan is None else (plan.expert, plan.place, plan.offset, plan.weight)
    mu, state, b = shift if shift is not None else (None, None, None)
    one = b is not None and b.cu is None      # one row per sequence: shifted in the same pass
    _load().stream_step(res, list(y or ()), list(norm_w or ()), rows, *e, list(norms), h, mu if one else None, state if one else None,
                        b.state_slot if one else None, b.ctx if one else None, int(width), float(eps))
    if b is not None and not one:
        n, h[0] = h[0], torch.empty_like(h[0])
        _load().token_shift(n, mu, state, h[0], b.state_slot, b.ctx, b.cu, b.seg_of)
    return h


def side_gate(z, embed, tokens, first, dim):
    out = torch.empty(z.shape[0], (dim + 7) // 8 * 8, dtype=z.dtype, device=z.device)
    _load().side_gate(z, embed, tokens, out, int(first), int(dim))
    return out


def softcap(z, cap):
    _load().softcap(z, float(cap))
    return z


def latent_write(raw, w, rank, eps, pool, slots, turned=None):
    if turned is None:
        _load().latent_write(raw, None, None, None, w, pool, slots, int(rank), 0, 0, 0, float(eps))
    else:
        q, k_rot, table, part, rot, dim = turned
        _load().latent_write(raw, k_rot, q, table, w, pool, slots, int(rank), int(part), int(rot), int(dim), float(eps))


def head_linear(x, w, transposed, gate=None):
    T, H, _ = x.shape
    out = torch.empty(T, H, w.shape[1] if transposed else w.shape[2], dtype=x.dtype, device=x.device)
    if x.dtype == torch.bfloat16 and _load().head_gemm(x, w, gate, out, not transposed, err_flag(x.device)):
        return out
    _load().simt_gemm(x.transpose(0, 1), w, out.transpose(0, 1), not transposed)      # 32-bit mode
    if gate is not None:
        _load().gate_outputs(out, gate)
    return out


LATENT_TILE = 128      # positions per tile of the tensor-core latent attention


def latent_columns(row: int, rank: int) -> int:
    """Most (token, head) columns a CTA of the tensor-core latent attention serves: 64, fewer when the queries of that many and the
    tiles of one step (``row`` features, the first ``rank`` of them values) do not fit its shared memory together; 0: rows too wide."""
    if row % 64 or rank % 64 or row > 640 or rank > 512:
        return 0
    pairs = (row // 64 + 1) // 2
    return next((n for n in (64, 32, 16) if pairs * 32768 + row // 64 * n * 128 + 512 * n + 2560 <= 227 * 1024), 0)


def latent_attention(q, pool, b, block_size, scale, gate, rank=None):
    """Tensor cores for bf16 with ranks up to 512 and pages of 16 to 128 tokens, CUDA cores otherwise (32-bit mode)."""
    q = q.contiguous()
    T, H, R = q.shape
    rank = rank or R
    out = torch.empty(T, H, rank, dtype=q.dtype, device=q.device)
    n = b.long_segs
    bt, ctx = b.block_tables[n:], b.ctx[n:]
    most = latent_columns(R, rank) if q.dtype == torch.bfloat16 and block_size in (16, 32, 64, 128) else 0
    if most:
        items = b.items[H] if b.items is not None else None
        if items is None and b.cu is not None:
            raise ValueError("a batch of segments needs its column groups (attention_items)")
        width = (b.item_width or {}).get(H, 64) if items is not None else min(most, 64 if H > 32 else (16 if H <= 16 else 32))
        groups = items.shape[0] if items is not None else T * ((H + width - 1) // width)
        splits = max(1, min(148 // groups, (b.max_ctx + LATENT_TILE - 1) // LATENT_TILE, 32))
        po = ml = None
        if splits > 1:
            po = torch.empty(splits * T * H * rank, dtype=torch.float32, device=q.device)
            ml = torch.empty(splits * T * H * 2, dtype=torch.float32, device=q.device)
        if _load().latent_attn_tc(q, pool, bt, items, ctx, gate, out, po, ml, int(block_size), width, splits, float(scale), err_flag(q.device)):
            return out
    _load().latent_attn(q, pool, bt, b.row_seg, b.row_pos, ctx, gate, out, int(block_size), float(scale))
    return out


def dense_flash(q, k, v, first, blocks, scale, gate=None, features=False):
    out = torch.empty(q.shape[0], q.shape[1] * v.shape[2], dtype=q.dtype, device=q.device)
    if not _load().dense_flash(q, k, v, first, blocks, gate, bool(features), out, float(scale), err_flag(q.device)):
        raise ValueError(f"no kernel for heads of {q.shape[2]} / {v.shape[2]} features, {q.dtype}")
    return out


def qkv_post(qkv, nq, nkv, q_norm_w, k_norm_w, cos, sin, eps, k_cache=None, v_cache=None, slots=None, dense_kv=True):
    """Per-head q/k RMSNorm (optional) + rotary embedding + KV-cache write in one launch.
    Returns ``(q, k, v)`` as ``[T, heads, 128]``; ``k``/``v`` are None unless ``dense_kv``."""
    T = qkv.shape[0]
    q = torch.empty(T, nq, 128, dtype=qkv.dtype, device=qkv.device)
    k = torch.empty(T, nkv, 128, dtype=qkv.dtype, device=qkv.device) if dense_kv else None
    v = torch.empty(T, nkv, 128, dtype=qkv.dtype, device=qkv.device) if dense_kv else None
    _load().qkv_post(qkv, q_norm_w, k_norm_w, cos.contiguous(), sin.contiguous(), q, k, v, k_cache, v_cache, slots, nq, nkv,
                     float(eps))
    return q, k, v


def quantize_rows_fp8(x, block: int = 128):
    """Per-row, per-``block`` columns e4m3 quantisation of activations: ``(q [M, K] float8_e4m3fn, scale [M, K/block])``
    with ``x ~ q * scale``."""
    M, K = x.shape
    kb = (K + block - 1) // block
    xp = torch.nn.functional.pad(x.float(), (0, kb * block - K)).view(M, kb, block)
    scale = xp.abs().amax(-1).clamp_min(1e-12) / 448.0
    q = (xp / scale.unsqueeze(-1)).clamp(-448.0, 448.0).to(torch.float8_e4m3fn).view(M, kb * block)[:, :K].contiguous()
    return q, scale.contiguous()


def fp8_linear(x, w_q, w_scale_inv, x_q=None, x_scale=None):
    """``x @ dequant(w_q)^T`` on the fp8 tensor cores with block scaling: weights are e4m3 with one scale per
    128 x 128 block (``weight_scale_inv`` of :func:`blockwise_cast_to_fp8`), activations are quantised per row and
    128 columns here unless given.  Output bf16."""
    x2 = x.reshape(-1, x.shape[-1])
    if x_q is None:
        x_q, x_scale = quantize_rows_fp8(x2)
    out = torch.empty(x2.shape[0], w_q.shape[0], dtype=torch.bfloat16, device=x.device)
    _load().gemm_fp8(x_q, x_scale.float().contiguous(), w_q, w_scale_inv.float().contiguous(), out, err_flag(x.device))
    return out.reshape(*x.shape[:-1], w_q.shape[0])


class _LinearNN(torch.autograd.Function):
    """y = x @ b with b[K,N] row-major (used when the caller passes ``w.t()``)."""

    @staticmethod
    def forward(ctx, x, b):
        ctx.save_for_backward(x, b)
        return matmul_nn(x, b)

    @staticmethod
    def backward(ctx, dy):
        x, b = ctx.saved_tensors
        dy = dy.contiguous()
        dx = matmul_nt(dy, b) if ctx.needs_input_grad[0] else None
        db = matmul_tn(x, dy) if ctx.needs_input_grad[1] else None
        return dx, db


# --------------------------------------------------------------------------- norms / elementwise


class _RMSNorm(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, w, eps):
        x = x.contiguous()
        cols = x.shape[-1]
        rows = x.numel() // cols
        y = torch.empty_like(x)
        _load().rmsnorm_fwd(x, None, w, y, None, rows, cols, eps)
        ctx.save_for_backward(x, w)
        ctx.eps = eps
        return y

    @staticmethod
    def backward(ctx, dy):
        x, w = ctx.saved_tensors
        cols = x.shape[-1]
        rows = x.numel() // cols
        dy = dy.contiguous()
        dx = torch.empty_like(x)
        dw = torch.empty_like(w)
        C = _load()
        scratch = torch.empty(C.rmsnorm_bwd_parts(rows, cols) * cols, dtype=torch.float32, device=x.device)
        C.rmsnorm_bwd(x, w, dy, dx, dw, scratch, rows, cols, ctx.eps)
        return dx, dw, None


def rmsnorm(x, w, eps=1e-6):
    return _RMSNorm.apply(x, w, eps)


class _AddRMSNorm(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, res, w, eps):
        x, res = x.contiguous(), res.contiguous()
        cols = x.shape[-1]
        rows = x.numel() // cols
        y, r = torch.empty_like(x), torch.empty_like(x)
        _load().rmsnorm_fwd(x, res, w, y, r, rows, cols, eps)
        ctx.save_for_backward(r, w)
        ctx.eps = eps
        return y, r

    @staticmethod
    def backward(ctx, dy, dr):
        r, w = ctx.saved_tensors
        cols = r.shape[-1]
        rows = r.numel() // cols
        dx = torch.empty_like(r)
        dw = torch.empty_like(w)
        C = _load()
        scratch = torch.empty(C.rmsnorm_bwd_parts(rows, cols) * cols, dtype=torch.float32, device=r.device)
        C.rmsnorm_bwd(r, w, dy.contiguous(), dx, dw, scratch, rows, cols, ctx.eps)
        if dr is not None:
            dx = dx + dr
        return dx, dx, dw, None


def add_rmsnorm(x, res, w, eps=1e-6):
    return _AddRMSNorm.apply(x, res, w, eps)


class _Rope(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, cos, sin):
        x = x.contiguous()
        T, H, D = x.shape
        y = torch.empty_like(x)
        cos, sin = cos.contiguous(), sin.contiguous()
        _load().rope(x, y, cos, sin, T, H, D, False)
        ctx.save_for_backward(cos, sin)
        return y

    @staticmethod
    def backward(ctx, dy):
        cos, sin = ctx.saved_tensors
        dy = dy.contiguous()
        T, H, D = dy.shape
        dx = torch.empty_like(dy)
        _load().rope(dy, dx, cos, sin, T, H, D, True)
        return dx, None, None


def apply_rope(x, cos, sin):
    return _Rope.apply(x, cos.float(), sin.float())


class _SwiGLU(torch.autograd.Function):
    @staticmethod
    def forward(ctx, gu):
        gu = gu.contiguous()
        F = gu.shape[-1] // 2
        rows = gu.numel() // (2 * F)
        out = torch.empty(*gu.shape[:-1], F, dtype=gu.dtype, device=gu.device)
        _load().swiglu_fwd(gu, out, rows, F)
        ctx.save_for_backward(gu)
        return out

    @staticmethod
    def backward(ctx, dout):
        (gu,) = ctx.saved_tensors
        F = gu.shape[-1] // 2
        rows = gu.numel() // (2 * F)
        din = torch.empty_like(gu)
        _load().swiglu_bwd(gu, dout.contiguous(), din, rows, F)
        return din


def swiglu(gate_up):
    return _SwiGLU.apply(gate_up)


# --------------------------------------------------------------------------- optimizer / misc


def fused_adam(pshard, master, gshard, exp_avg, exp_avg_sq, step, lr, b1, b2, eps, wd, gscale, split):
    _load().adam(pshard, master, gshard, exp_avg, exp_avg_sq, step, lr, b1, b2, eps, wd, gscale, split)


def sumsq(x) -> torch.Tensor:
    out = torch.zeros(1, dtype=torch.float32, device=x.device)
    _load().sumsq(x.contiguous().view(-1), out)
    return out


def kv_scatter(k, v, k_cache, v_cache, slots):
    """k/v ``[T, H, D]`` (possibly strided views of a fused qkv buffer) -> cache rows ``slots[T]``."""
    T = k.shape[0]
    row = k.shape[1] * k.shape[2]
    if k.stride(2) != 1 or k.stride(1) != k.shape[2]:
        k = k.contiguous()
    if v.stride(2) != 1 or v.stride(1) != v.shape[2]:
        v = v.contiguous()
    _load().kv_scatter(k, v, k_cache, v_cache, slots, T, row, k.stride(0), v.stride(0))


def fake_int4_quant(x, block_m, block_n, sym=True):
    x = x.contiguous()
    M, N = x.shape
    gm, gn = (M + block_m - 1) // block_m, (N + block_n - 1) // block_n
    out = torch.empty_like(x)
    scale = torch.empty(gm, gn, dtype=x.dtype, device=x.device)
    zero = torch.empty(gm, gn, dtype=x.dtype, device=x.device)
    _load().int4_fake_quant(x, out, scale, zero, block_m, block_n, sym)
    return out, scale, zero


def blockwise_cast_to_fp8(w, block=128, ue8m0=False):
    w = w.contiguous()
    M, N = w.shape
    q = torch.empty(M, N, dtype=torch.float8_e4m3fn, device=w.device)
    scale = torch.empty((M + block - 1) // block, (N + block - 1) // block, dtype=torch.float32, device=w.device)
    _load().fp8_block_cast(w, q, scale, block, ue8m0)
    return q, scale


def blockwise_dequant_fp8(q, scale_inv, block=128, dtype=torch.bfloat16):
    out = torch.empty(q.shape, dtype=dtype, device=q.device)
    _load().fp8_block_dequant(q.contiguous(), scale_inv.contiguous(), out, block)
    return out


# --------------------------------------------------------------------------- weight-sync copy table


class CopyTable:
    def __init__(self, table, chunk_start, n_desc, total_chunks, chunk_rows, elem_size, keepalive):
        self.table, self.chunk_start = table, chunk_start
        self.n_desc, self.total_chunks, self.chunk_rows, self.elem_size = n_desc, total_chunks, chunk_rows, elem_size
        self.keepalive = keepalive


def build_copy_table_raw(entries, device, elem_size: int, chunk_bytes: int = 1 << 18) -> CopyTable:
    """entries: (src_ptr, dst_ptr, rows, cols, src_ld, dst_ld) in elements.  Large blocks are
    split into chunks of about ``chunk_bytes`` so the copy spreads over all SMs."""
    import struct

    raw = bytearray()
    starts, total = [], 0
    chunk_rows_list = []
    # one global chunk_rows keeps the kernel simple: rows per chunk chosen from the widest block
    max_cols = max((e[3] for e in entries), default=1)
    chunk_rows = max(1, chunk_bytes // max(1, max_cols * elem_size))
    for (s, d, rows, cols, sld, dld) in entries:
        raw += struct.pack("<QQiiii", s, d, rows, cols, sld, dld)
        starts.append(total)
        total += (rows + chunk_rows - 1) // chunk_rows
    table = torch.frombuffer(raw, dtype=torch.uint8).to(device)
    cs = torch.tensor(starts, dtype=torch.int32, device=device)
    return CopyTable(table, cs, len(entries), total, chunk_rows, elem_size, None)


def copy_entries(blocks, trainer_params: dict, dst_params: dict) -> list:
    """Raw ``(src_ptr, dst_ptr, rows, cols, src_ld, dst_ld)`` entries of plan blocks; ``dst_params`` maps rollout
    parameter names to tensors, which may be views of ANOTHER GPU's memory mapped into this process."""
    entries = []
    es = next(iter(trainer_params.values())).element_size()
    for b in blocks:
        src = trainer_params[b.src_name]
        dst = dst_params[b.dst_name]
        s2 = src[b.src_batch] if src.dim() == 3 else (src.view(1, -1) if src.dim() == 1 else src)
        d2 = dst[b.dst_batch] if dst.dim() == 3 else (dst.view(1, -1) if dst.dim() == 1 else dst)
        sp = s2.data_ptr() + (b.src_row * s2.stride(0) + b.src_col) * es
        dp = d2.data_ptr() + (b.dst_row * d2.stride(0) + b.dst_col) * es
        entries.append((sp, dp, b.rows, b.cols, s2.stride(0), d2.stride(0)))
    return entries


def build_copy_table(blocks, trainer_params: dict, rollout_weights) -> CopyTable:
    es = next(iter(trainer_params.values())).element_size()
    t = build_copy_table_raw(copy_entries(blocks, trainer_params, rollout_weights.p), rollout_weights.device, es)
    t.keepalive = (trainer_params, rollout_weights)
    return t


def run_copy_table(t: CopyTable):
    _load().copy_table(t.table, t.n_desc, t.chunk_start, t.total_chunks, t.chunk_rows, t.elem_size)


# --------------------------------------------------------------------------- flash attention (training / prefill)


def _tok_head_view(t):
    """[T, H, 128] with unit inner stride and 16-byte aligned outer strides, else a contiguous copy."""
    if t.stride(2) != 1 or t.stride(0) % 8 or t.stride(1) % 8 or t.data_ptr() % 16:
        t = t.contiguous()
    return t


class _FlashAttn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, q, k, v, cu_q, cu_k, causal, scale, max_q_blocks, max_kv_blocks):
        q, k, v = _tok_head_view(q), _tok_head_view(k), _tok_head_view(v)
        Tq, Hq, D = q.shape
        o = torch.empty(Tq, Hq, D, dtype=q.dtype, device=q.device)
        lse = torch.empty(Hq, Tq, dtype=torch.float32, device=q.device)
        _load().fa_fwd(q, k, v, o, lse, cu_q, cu_k, max_q_blocks, causal, scale, err_flag(q.device))
        ctx.save_for_backward(q, k, v, o, lse, cu_q, cu_k)
        ctx.causal, ctx.scale, ctx.max_kv_blocks = causal, scale, max_kv_blocks
        return o

    @staticmethod
    def backward(ctx, do):
        q, k, v, o, lse, cu_q, cu_k = ctx.saved_tensors
        q, k, v, do = q.contiguous(), k.contiguous(), v.contiguous(), do.contiguous()
        Tq, Hq, D = q.shape
        dq, dk, dv = torch.empty_like(q), torch.empty_like(k), torch.empty_like(v)
        delta = torch.empty(Hq, Tq, dtype=torch.float32, device=q.device)
        dq_acc = torch.empty(Tq, Hq, D, dtype=torch.float32, device=q.device)
        _load().fa_bwd(q, k, v, o, do, lse, dq, dk, dv, delta, dq_acc, cu_q, cu_k, ctx.max_kv_blocks, ctx.causal,
                       ctx.scale, err_flag(q.device))
        return dq, dk, dv, None, None, None, None, None, None


def attention_varlen(q, k, v, cu_seqlens, causal=True, scale=None, cu_seqlens_k=None, max_seqlen=None):
    """Packed varlen attention; q [Tq, Hq, 128], k/v [Tk, Hkv, 128] bf16."""
    if q.dtype != torch.bfloat16 or q.shape[-1] != 128:
        raise NotImplementedError("the sm_100a attention kernel handles bf16 with head_dim 128")
    cu_q = cu_seqlens.to(torch.int32)
    cu_k = cu_q if cu_seqlens_k is None else cu_seqlens_k.to(torch.int32)
    scale = scale if scale is not None else 1.0 / math.sqrt(q.shape[-1])
    nseq = cu_q.numel() - 1
    # upper bounds of the tile counts (no host sync): every sequence adds at most one partial tile
    max_q_blocks = (q.shape[0] + 127) // 128 + nseq
    max_kv_blocks = (k.shape[0] + 127) // 128 + nseq
    return _FlashAttn.apply(q, k, v, cu_q, cu_k, bool(causal), float(scale), max_q_blocks, max_kv_blocks)


# --------------------------------------------------------------------------- rollout kernels


def paged_decode_attention(q, k_cache, v_cache, block_tables, context_lens, scale=None, max_ctx=None, splits=None,
                           version=None):
    B, Hq, D = q.shape
    Hkv = k_cache.shape[2]
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    if max_ctx is None:
        max_ctx = block_tables.shape[1] * k_cache.shape[1]
    C = _load()
    if splits is None:
        splits = int(os.environ.get("RELAX_B200_DECODE_SPLITS", "0")) or C.decode_attn_splits(B, Hkv, max_ctx)
        if B * Hkv >= 148:
            splits = 1   # enough CTAs already; splitting only adds the combine pass
    if version is None:
        version = int(os.environ.get("RELAX_B200_DECODE_ATTN_VERSION", "3"))
    if version == 3 and k_cache.shape[1] != 16:
        version = 1   # the tensor-core kernel gathers 16-token pages
    out = torch.empty_like(q)
    po = pm = None
    if splits > 1:
        po = torch.empty(B * Hq * splits * D, dtype=torch.float32, device=q.device)
        pm = torch.empty(B * Hq * splits * 2, dtype=torch.float32, device=q.device)
    C.decode_attn(q.contiguous(), k_cache, v_cache, block_tables.to(torch.int32).contiguous(),
                  context_lens.to(torch.int32).contiguous(), out, po, pm, max_ctx, scale, splits, version,
                  err_flag(q.device))
    return out


def sample(logits, temperature, top_k, top_p, uniform):
    """Rows of bf16 or fp32 logits (unit inner stride; any row pitch) -> ``(token int64 [B], log-prob fp32 [B])``."""
    if logits.dtype not in (torch.bfloat16, torch.float32):
        logits = logits.float()
    if logits.stride(1) != 1:
        logits = logits.contiguous()
    B, V = logits.shape
    tok = torch.empty(B, dtype=torch.int64, device=logits.device)
    lp = torch.empty(B, dtype=torch.float32, device=logits.device)
    _load().sample_v2(logits, temperature.float().contiguous(), top_k.to(torch.int64).contiguous(),
                      top_p.float().contiguous(), uniform.float().contiguous(), tok, lp, V)
    return tok, lp


def decode_advance(tok_new, lp_new, st, block_size: int):
    """Device-side tail of one decode step (see :func:`relax_b200.ops.reference.decode_advance` for the statement)."""
    _load().decode_advance(tok_new, lp_new, st["tok"], st["pos"], st["ctx"], st["slots"], st["bt"], int(block_size),
                           st["active"], st["remain"], st["eos"], st["stop"], st["out_tok"], st["out_lp"], st["counter"],
                           st["u_all"], st["u"])


class _TopKRouter(torch.autograd.Function):
    @staticmethod
    def forward(ctx, logits, k, norm):
        logits = logits.float().contiguous()
        T, E = logits.shape
        w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
        idx = torch.empty(T, k, dtype=torch.int64, device=logits.device)
        probs = torch.empty(T, E, dtype=torch.float32, device=logits.device)
        _load().topk_router(logits, k, norm, w, idx, probs)
        ctx.save_for_backward(probs, idx, w)
        ctx.norm = norm
        ctx.mark_non_differentiable(idx)
        return w, idx, probs

    @staticmethod
    def backward(ctx, dw, _didx, dprobs):
        probs, idx, w = ctx.saved_tensors
        # gradient w.r.t. probs from the (optionally renormalised) selected weights
        gp = torch.zeros_like(probs) if dprobs is None else dprobs.clone()
        if dw is not None:
            if ctx.norm:
                sel = probs.gather(-1, idx)
                ssum = sel.sum(-1, keepdim=True)
                dsel = (dw - (dw * w).sum(-1, keepdim=True)) / ssum
            else:
                dsel = dw
            gp.scatter_add_(-1, idx, dsel)
        # softmax backward
        dlogits = probs * (gp - (gp * probs).sum(-1, keepdim=True))
        return dlogits, None, None


def topk_router(logits, top_k, norm_topk_prob=True):
    return _TopKRouter.apply(logits, int(top_k), bool(norm_topk_prob))


# --------------------------------------------------------------------------- fused LM head + log-prob / entropy


class _FusedLMHead(torch.autograd.Function):
    CHUNK = 4096
    _dlogits: dict = {}       # (device, dtype) -> flat scratch for the chunk's d(logits), reused by every backward

    @staticmethod
    def forward(ctx, hidden, weight, targets, tp_group, vocab_start, with_entropy, temperature):
        import torch.distributed as dist

        C = _load()
        h = hidden if (hidden.stride(1) == 1 and hidden.stride(0) % 8 == 0) else hidden.contiguous()
        w = weight if (weight.stride(1) == 1 and weight.stride(0) % 8 == 0) else weight.contiguous()
        T, V = h.shape[0], w.shape[0]
        inv_t = 1.0 / float(temperature)
        tp = tp_group is not None and dist.is_initialized() and dist.get_world_size(tp_group) > 1
        if T == 0:
            z = torch.zeros(0, dtype=torch.float32, device=h.device)
            ctx.save_for_backward(h, w, targets, z, z)
            ctx.meta = (tp_group, vocab_start, inv_t, with_entropy, weight)
            return z, z.clone()
        splits = C.lm_head_splits(T, V)
        part = torch.empty(T, splits, 4, dtype=torch.float32, device=h.device)
        C.lm_head_logprob(h, w, targets.contiguous(), part, vocab_start, inv_t, splits, err_flag(h.device))
        m = part[..., 0]
        gm = m.max(1).values
        if tp:
            dist.all_reduce(gm, op=dist.ReduceOp.MAX, group=tp_group)
        sc = torch.exp(m - gm[:, None])
        zt = part[..., 3].max(1).values
        found = torch.isfinite(zt)
        acc = torch.stack([(part[..., 1] * sc).sum(1), (part[..., 2] * sc).sum(1), torch.where(found, zt, torch.zeros_like(zt))])
        if tp:
            dist.all_reduce(acc, group=tp_group)
        s, u, zt = acc[0], acc[1], acc[2]
        logz = gm + torch.log(s)
        ez = u / s
        lp = zt - logz
        ent = logz - ez if with_entropy else torch.zeros_like(lp)
        ctx.save_for_backward(h, w, targets, logz, ez)
        ctx.meta = (tp_group, vocab_start, inv_t, with_entropy, weight)
        return lp, ent

    @staticmethod
    def backward(ctx, g_lp, g_ent):
        h, w, targets, logz, ez = ctx.saved_tensors
        tp_group, vocab_start, inv_t, with_entropy, weight = ctx.meta
        C = _load()
        T, H = h.shape
        V = w.shape[0]
        dh = torch.empty_like(h)
        main_grad = getattr(weight, "main_grad", None)
        direct = main_grad is not None and main_grad.dtype == torch.float32 and main_grad.shape == weight.shape \
            and w.data_ptr() == weight.data_ptr()
        dw32 = main_grad if direct else torch.zeros(V, H, dtype=torch.float32, device=h.device)
        if main_grad is not None and not direct and main_grad.dtype == torch.float32 and w.shape[0] < weight.shape[0] \
                and w.data_ptr() == weight.data_ptr():
            dw32, direct = main_grad[:V], True   # vocabulary padding rows sliced off by the caller
        stats = torch.stack([logz, ez], 1).contiguous()
        g_lp = (g_lp if g_lp is not None else torch.zeros_like(logz)).float().contiguous()
        g_en = g_ent.float().contiguous() if (with_entropy and g_ent is not None) else None
        tg = targets.contiguous()
        ck = _FusedLMHead.CHUNK
        # d(logits) of one chunk: up to 4096 x V (1.2 GB at V = 152k).  Kept across calls: a fresh allocation of that
        # size per micro-batch does not fit the blocks the caching allocator has left and costs a cudaMalloc every
        # time (about 12 ms during which the device runs dry - measured)
        key = (h.device, h.dtype)
        buf = _FusedLMHead._dlogits.get(key)
        need = min(ck, T) * V
        if buf is None or buf.numel() < need:
            buf = None
            _FusedLMHead._dlogits.pop(key, None)
            buf = _FusedLMHead._dlogits[key] = torch.empty(need, dtype=h.dtype, device=h.device)
        buf = buf[:need].view(min(ck, T), V)
        for s in range(0, T, ck):
            e = min(T, s + ck)
            d = buf[: e - s]
            C.lm_head_dlogits(h[s:e], w, tg[s:e], stats[s:e], g_lp[s:e], None if g_en is None else g_en[s:e], d,
                              vocab_start, inv_t, err_flag(h.device))
            matmul_nn(d, w, out=dh[s:e])
            matmul_tn(d, h[s:e], out=dw32, accumulate=True)
        dw = None if direct else dw32.to(weight.dtype)
        if dw is not None and dw.shape != weight.shape:
            full = torch.zeros_like(weight)
            full[: dw.shape[0]] = dw
            dw = full
        return dh, dw, None, None, None, None, None


def fused_lm_head_logprob(hidden, weight, targets, tp_group=None, vocab_start=0, with_entropy=True, temperature=1.0):
    if hidden.dtype != torch.bfloat16:
        raise TypeError("fused LM head expects bf16 hidden states")
    return _FusedLMHead.apply(hidden, weight, targets, tp_group, vocab_start, with_entropy, temperature)


# --------------------------------------------------------------------------- fused policy loss


class _PolicyLoss(torch.autograd.Function):
    @staticmethod
    def forward(ctx, ppo_kl, adv, eps_clip, eps_clip_high, eps_clip_c):
        kl = ppo_kl.detach().float().contiguous()
        loss, clip, g = (torch.empty_like(kl) for _ in range(3))
        _load().policy_loss(kl, adv.detach().float().contiguous().expand_as(kl).contiguous(), loss, clip, g,
                            float(eps_clip), float(eps_clip_high), float(eps_clip_c or 0.0))
        ctx.save_for_backward(g)
        ctx.mark_non_differentiable(clip)
        return loss, clip

    @staticmethod
    def backward(ctx, dloss, _dclip):
        (g,) = ctx.saved_tensors
        return dloss * g, None, None, None, None


def policy_loss(ppo_kl, advantages, eps_clip, eps_clip_high, eps_clip_c=None):
    """``(loss, clipfrac)`` per token of the PPO clipped surrogate in one kernel; the same pass writes
    d loss / d ppo_kl, so backward is one multiply.  Advantages are treated as constants."""
    return _PolicyLoss.apply(ppo_kl, advantages, eps_clip, eps_clip_high, eps_clip_c)


# --------------------------------------------------------------------------- grouped (MoE expert) GEMM


class _GroupedLinear(torch.autograd.Function):
    """``y[row] = x[row] @ w[expert(row)].T`` over an expert-sorted, 128-row aligned token buffer: ONE kernel launch
    per product for all local experts, tile -> expert map read on the device (csrc/grouped_gemm_sm100.cu)."""

    @staticmethod
    def forward(ctx, x, w, tile_expert, expert_rows):
        x = x.contiguous()
        wc = w if w.is_contiguous() else w.contiguous()
        y = torch.empty(x.shape[0], w.shape[1], dtype=x.dtype, device=x.device)
        _load().grouped_gemm_fwd(x, wc, y, tile_expert, err_flag(x.device))
        ctx.save_for_backward(x, wc, tile_expert, expert_rows)
        ctx.weight = w
        return y

    @staticmethod
    def backward(ctx, dy):
        x, wc, tile_expert, expert_rows = ctx.saved_tensors
        w = ctx.weight
        dy = dy.contiguous()
        L = _load()
        dx = None
        if ctx.needs_input_grad[0]:
            dx = torch.empty_like(x)
            L.grouped_gemm_dgrad(dy, wc, dx, tile_expert, err_flag(x.device))
        dw = None
        if ctx.needs_input_grad[1]:
            mg = getattr(w, "main_grad", None)
            if mg is not None and mg.dtype == torch.float32 and mg.shape == w.shape and mg.is_contiguous():
                L.grouped_gemm_wgrad(dy, x, mg, expert_rows, True, err_flag(x.device))
            else:
                dw = torch.empty_like(wc)
                L.grouped_gemm_wgrad(dy, x, dw, expert_rows, False, err_flag(x.device))
        return dx, dw, None, None


def grouped_linear(x, w, tile_expert, expert_rows):
    if x.dtype != torch.bfloat16 or x.shape[0] % 128 or w.shape[1] % 64 or w.shape[2] % 64:
        raise ValueError("grouped GEMM: bf16, token rows padded to 128 per expert, expert dims multiples of 64")
    return _GroupedLinear.apply(x, w, tile_expert, expert_rows)


def launch_count() -> int:
    """Number of kernels of this extension launched since the last reset (all threads)."""
    return int(_load().launch_count())


def reset_launch_count():
    _load().reset_launch_count()
