"""Operator entry points.

CUDA tensors go to the hand-written sm_100a kernels in the in-tree extension
(:mod:`relax_b200.ops.cuda`); CPU tensors go to the PyTorch statements in
:mod:`relax_b200.ops.reference`.  There is no silent fallback on a GPU: if the
extension is missing, a CUDA call raises.  ``RELAX_B200_FORCE_REFERENCE=1``
routes CUDA tensors through the PyTorch/library path on purpose - that is the
"unfused NCCL + cuBLAS" baseline arm used for A/B timing.
"""
from __future__ import annotations

import torch

import os

from . import reference as ref


def _force_ref() -> bool:
    return os.environ.get("RELAX_B200_FORCE_REFERENCE", "0") == "1"


def _use_cuda(t) -> bool:
    return t.is_cuda and not _force_ref()


def _cuda():
    from . import cuda as _c

    return _c


def _vec_ok(t) -> bool:
    """Rows of ``t`` split into 16-byte vectors (what the elementwise kernels load)."""
    return t.shape[-1] % (16 // t.element_size()) == 0


def rmsnorm(x, w, eps=1e-6):
    return _cuda().rmsnorm(x, w, eps) if _use_cuda(x) and _vec_ok(x) else ref.rmsnorm(x, w, eps)


def add_rmsnorm(x, residual, w, eps=1e-6):
    if _use_cuda(x) and _vec_ok(x):
        return _cuda().add_rmsnorm(x, residual, w, eps)
    return ref.add_rmsnorm(x, residual, w, eps)


def swiglu(gate_up):
    if _use_cuda(gate_up) and (gate_up.shape[-1] // 2) % (16 // gate_up.element_size()) == 0:
        return _cuda().swiglu(gate_up)
    return ref.swiglu(gate_up)


def glu(gate_up, act: str = "silu"):
    """Gated unit ``act(gate) * up`` on ``[gate | up]`` rows; ``act``: ``silu`` or ``gelu_tanh``."""
    return _cuda().glu(gate_up, act) if _use_cuda(gate_up) else ref.glu(gate_up, act)


def linear_glu(x, w, act: str = "silu"):
    """``glu(x @ w.T)`` with ``w = [gate; up]``: one fused kernel for decode shapes."""
    return _cuda().linear_glu(x, w, act) if _use_cuda(x) else ref.glu(ref.linear(x, w), act)


def linear_act(x, w, act: str):
    """``act(x @ w.T)`` without a gate (``act``: ``relu2``); joins the decode GEMM's reduction for decode shapes."""
    if act != "relu2":
        raise ValueError(f"no ungated activation {act!r}")
    return _cuda().linear_relu2(x, w) if _use_cuda(x) else ref.relu2(ref.linear(x, w))


def linear_fp32(x, w):
    """``x @ w.T`` with fp32 results (router logits): products of 16-bit operands are exact in the fp32 accumulator."""
    return _cuda().linear_fp32(x, w) if _use_cuda(x) else ref.linear(x.float(), w.float())


def embed_rows(tokens, w, norm_w=None, width=0, groups=1, eps=0.0, scale=1.0):
    """Embedded tokens as the fp32 residual stream and its copy in the weights' type: normed in groups with ``norm_w``, or times
    ``scale`` without."""
    return (_cuda() if _use_cuda(w) else ref).embed_rows(tokens, w, norm_w, width, groups, eps, scale)


def norm_add(res, y, w, width, groups, eps, next_w=None, experts=None):
    """Output norm in groups + add to the fp32 residual stream (in place) + the next sublayer's input, one kernel.
    ``experts``: ``(rows, plan)`` of :func:`moe_experts`, whose weighted sum joins ``y`` in the same pass."""
    return (_cuda() if _use_cuda(res) else ref).norm_add(res, y, w, width, groups, eps, next_w, experts)


def sum_norm(res, y, w, b, width, alpha, eps, nxt=None, scale=1.0, experts=None):
    """``res <- norm(alpha res + y)`` in place (fp32), a layer norm with weight and bias (RMS when ``b`` is None), and the next
    sublayer's input, one kernel; ``nxt``: ``(weight, bias)`` of the model's last norm, which then gives the result, times ``scale``.
    ``experts``: as for :func:`norm_add`."""
    return (_cuda() if _use_cuda(res) else ref).sum_norm(res, y, w, b, width, alpha, eps, nxt, scale, experts)


def rope_table(positions, offset, inv_freq):
    """cos / sin of every row's angles, computed once per forward for all layers that turn alike."""
    return (_cuda() if _use_cuda(positions) else ref).rope_table(positions, offset, inv_freq)


def attention_inputs(qkv, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps, k_pool, v_pool, slots):
    """Rotation and weightless norm of queries and keys, and the write of keys and values into their pages, one kernel."""
    return (_cuda() if _use_cuda(qkv) else ref).attention_inputs(qkv, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps, k_pool, v_pool, slots)


def projection_inputs(qkv, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, halves, eps, k_pool, v_pool, slots):
    """The same with weighted RMS norms over ALL query columns and over all key columns (``eps`` <= 0: none), then the rotation, of
    neighbours or (``halves``) of features ``rot_dims / 2`` apart."""
    return (_cuda() if _use_cuda(qkv) else ref).projection_inputs(qkv, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, halves, eps, k_pool,
                                                                  v_pool, slots)


def conv_inputs(qkv, bias, taps, state, batch, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps, k_pool, v_pool):
    """The same with biases, a causal convolution over time on every channel (its last rows carried in ``state`` by slot), and weighted
    norms head by head (``eps`` <= 0: none) before neighbours turn."""
    return (_cuda() if _use_cuda(qkv) else ref).conv_inputs(qkv, bias, taps, state, batch, q_w, k_w, table, heads, kv_heads, dim, vdim, dp, rot_dims, eps,
                                                            k_pool, v_pool)


def paged_attention(q, k_pool, v_pool, batch, block_size, scale, sink, out_width, window=0, gate=None, keep=0, chunk=0, softcap=0.0, talk=None):
    """Grouped-query attention over paged keys and values for every segment of a
    :class:`relax_b200.rollout.composed.SegmentBatch`, with an optional sink logit per head, an optional ``window`` (positions a
    row sees, its own included; 0 = all) that leaves the first ``keep`` positions visible, or chunks of ``chunk`` positions, optionally capped
    scores, an optional ``gate`` per output feature (``[T, heads * out_width]``, its sigmoid counts), and optionally heads whose weights
    are mixed by ``talk[H, H]`` before they meet the values."""
    if _use_cuda(q):
        return _cuda().paged_attention(q, k_pool, v_pool, batch, block_size, scale, sink, out_width, window, gate, keep, chunk, softcap, talk)
    return ref.paged_attention(q, k_pool, v_pool, batch.block_tables, block_size, batch.ctx, batch.cu, scale, sink, out_width, window, gate, keep, chunk,
                               softcap, talk)


def route_counters(layers: int, experts: int, device):
    """Zeroed counters for ``layers`` calls of :func:`moe_route` with up to ``experts`` experts (one memset per forward)."""
    on_gpu = torch.device(device).type == "cuda" and not _force_ref()
    return _cuda().route_counters(layers, experts, device) if on_gpu else [None] * layers


def moe_route(logits, spec, dtype, count=None, correction=None):
    """Expert choice of every row (:class:`relax_b200.models.config.MoESpec`) from fp32 logits; ``dtype``: of the experts' operands;
    ``count``: an unused row of :func:`route_counters`; ``correction``: offsets of the scores for the choice."""
    if _use_cuda(logits):
        return _cuda().moe_route(logits, spec, 64 if dtype == torch.float32 else 128, count, correction)      # rows per tile of the grouped GEMM
    return ref.moe_route(logits, spec, correction)


GLU_RUN = 32      # rows of one half that lie side by side in a gated expert's up-projection


def glu_rows(gate, up):
    """Rows ``[..., F, K]`` of the two halves of gated experts in the order of the grouped GEMM's epilogue: runs of :data:`GLU_RUN`
    gate rows, each followed by the up rows of the same features (``F`` is a multiple of it)."""
    s = (*gate.shape[:-2], gate.shape[-2] // GLU_RUN, GLU_RUN, gate.shape[-1])
    return torch.stack([gate.reshape(s), up.reshape(s)], -3).reshape(*gate.shape[:-2], 2 * gate.shape[-2], gate.shape[-1])


def moe_experts(h, plan, up, down, act, limit=0.0):
    """The chosen experts' outputs, unweighted, in an order :func:`norm_add` understands.  ``act`` ``clamped_swish``: ``up`` is made by
    :func:`glu_rows`, and ``limit`` bounds both halves."""
    return (_cuda() if _use_cuda(h) else ref).moe_experts(h, plan, up, down, act, limit)


def hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, eps, spans=None):
    """HGRN2 token mixing (gates, recurrence, per-head norm) on packed rows with the state carried in slots.  ``spans``:
    ``(row ranges [n, 2], first span of every segment [S + 1])`` lets long segments run in parts side by side."""
    if _use_cuda(qfv):
        return _cuda().hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, eps, spans)
    return ref.hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, eps)


def mingru(zxg, z_b, x_b, state, batch, width):
    """Gated running means per channel, read out through ``silu`` gates, with the state carried in slots."""
    return (_cuda() if _use_cuda(zxg) else ref).mingru(zxg, z_b, x_b, state, batch, width)


def gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, gate_col, eps, root, spans=None):
    """Linear attention whose state rows decay by gates of their own (recurrence, per-head norm, output gates), with the state carried in
    slots; ``spans`` as for :func:`hgrn2`."""
    if _use_cuda(rows):
        return _cuda().gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, gate_col, eps, root, spans)
    return ref.gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, heads, dim, vdim, gate_col, eps, root)


def stream_step(res, width, eps, y=None, norm_w=None, experts=None, norms=(), shift=None):
    """One pass over the fp32 stream ``res``: adds the mean of the rows in ``y`` (a list of one or two; with ``norm_w`` each is RMS-normed with
    its weight first) and the weighted expert rows ``experts``, in place; returns a list with the stream's layer norm for every weight in
    ``norms``, or with its copy in the weights' type.  ``shift``: ``(weights mu, state, batch)`` - the first norm's rows ``n`` become
    ``n + (before - n) mu`` with ``before`` the row in front in the same sequence, from ``state`` (by slot) for a segment's first row."""
    return (_cuda() if _use_cuda(res) else ref).stream_step(res, width, eps, y, norm_w, experts, norms, shift)


def side_gate(z, embed, tokens, first, dim):
    """``gelu_tanh(z)`` times a layer's own features of the tokens in a second embedding table."""
    return (_cuda() if _use_cuda(z) else ref).side_gate(z, embed, tokens, first, dim)


def softcap(z, cap):
    """``cap * tanh(z / cap)`` of fp32 logits (in place on the GPU)."""
    return (_cuda() if _use_cuda(z) else ref).softcap(z, cap)


def latent_write(raw, w, rank, eps, pool, slots, turned=None):
    """Norm of the latent projection + write of the new rows into the paged latent cache.  ``turned``: ``(q, k_rot, table, part, rot,
    dim)`` - the rotated key part ``k_rot`` goes to the rows' columns ``part ..``, and features ``dim .. dim + rot`` of every query head
    ``q[T, H, dk]`` turn in place (both pair by pair of neighbours)."""
    (_cuda() if _use_cuda(raw) else ref).latent_write(raw, w, rank, eps, pool, slots, turned)


def head_linear(x, w, transposed, gate=None):
    """One small linear map per head (folds a latent up-projection into the queries / applies it to attended latents), every output
    feature scaled by ``sigmoid(gate)`` when given (``[T, heads * out]``)."""
    return (_cuda() if _use_cuda(x) else ref).head_linear(x, w, transposed, gate)


def latent_columns(row: int, rank: int) -> int:
    """Columns per group that :func:`relax_b200.rollout.composed.attention_items` makes for latent rows of this size."""
    return _cuda().latent_columns(row, rank) or 64


def latent_attention(q, pool, batch, block_size, scale, gate, rank=None):
    """Attention of absorbed queries over paged latent rows for the short segments of a
    :class:`relax_b200.rollout.composed.SegmentBatch`; the first ``rank`` features of a row (all of them) are also the values.  Head outputs are
    scaled by ``sigmoid(gate)`` (``[T, H]``) when given."""
    if _use_cuda(q):
        return _cuda().latent_attention(q, pool, batch, block_size, scale, gate, rank)
    n = batch.long_segs
    cu = batch.short_cu if n else batch.cu
    return ref.latent_attention(q, pool, batch.block_tables[n:], block_size, batch.ctx[n:], cu, scale, gate, rank)


def dense_flash_serves(dtype, dk: int, dv: int) -> bool:
    """Whether :func:`dense_flash` takes heads of ``dk`` query / key and ``dv`` value features."""
    return not _force_ref() and dtype == torch.bfloat16 and dk <= 192 and dv <= 128


def dense_flash(q, k, v, first, blocks, scale, gate=None, features=False):
    """Causal attention on per-head keys and values ``[rows, H, dk / dv]`` (multiples of 8 that may differ), those of segment ``s`` from row
    ``first[s]`` on; ``blocks``: query tiles of up to 128 rows.  Every head's output (``features``: every output feature) is scaled by
    ``sigmoid(gate)``.  Returns ``[T, H * dv]``."""
    return _cuda().dense_flash(q, k, v, first, blocks, scale, gate, features)


def linear(x, w, bias=None):
    return _cuda().linear(x, w, bias) if _use_cuda(x) else ref.linear(x, w, bias)


def rope_cos_sin(positions, head_dim, theta, mrope_section=None):
    return ref.rope_cos_sin(positions, head_dim, theta, mrope_section)


_WARNED: set = set()


def _statement_on_gpu(what: str):
    """A shape no sm_100a kernel of this package covers runs as its PyTorch statement on the GPU; said once."""
    if what not in _WARNED:
        _WARNED.add(what)
        import warnings

        warnings.warn(f"relax_b200: {what}: no sm_100a kernel for this shape, running the PyTorch statement", stacklevel=3)


def apply_rope(x, cos, sin):
    if _use_cuda(x):
        if (x.shape[-1] // 2) % (16 // x.element_size()) == 0:
            return _cuda().apply_rope(x, cos, sin)
        _statement_on_gpu(f"rotary width {x.shape[-1]}")
    return ref.apply_rope(x, cos, sin)


def attention_varlen(q, k, v, cu_seqlens, causal=True, scale=None, cu_seqlens_k=None, max_seqlen=None):
    """Packed varlen attention.  On a GPU the tcgen05 kernels take bf16 with head_dim 128; narrower heads
    (64 / 80 / 96 - ViT towers, small models) are zero-padded to 128, which leaves q k^T and the first ``D`` output
    columns unchanged (the softmax scale stays 1 / sqrt(D))."""
    if _use_cuda(q):
        D = q.shape[-1]
        if q.dtype == torch.bfloat16 and D == v.shape[-1] and D <= 128 and D % 8 == 0:
            if D == 128:
                return _cuda().attention_varlen(q, k, v, cu_seqlens, causal, scale, cu_seqlens_k, max_seqlen)
            pad = (0, 128 - D)
            F = torch.nn.functional
            scale = scale if scale is not None else D ** -0.5
            o = _cuda().attention_varlen(F.pad(q, pad), F.pad(k, pad), F.pad(v, pad), cu_seqlens, causal, scale,
                                         cu_seqlens_k, max_seqlen)
            return o[..., :D]
        _statement_on_gpu(f"attention with {q.dtype}, head_dim {D} / {v.shape[-1]}")
    return ref.attention_varlen(q, k, v, cu_seqlens, causal, scale, cu_seqlens_k)


def paged_decode_attention(q, k_cache, v_cache, block_tables, context_lens, scale=None):
    if _use_cuda(q):
        if q.dtype == torch.bfloat16 and q.shape[-1] == 128:
            return _cuda().paged_decode_attention(q, k_cache, v_cache, block_tables, context_lens, scale)
        _statement_on_gpu(f"paged decode attention with {q.dtype}, head_dim {q.shape[-1]}")
    return ref.paged_decode_attention(q, k_cache, v_cache, block_tables, context_lens, scale)


def sample(logits, temperature, top_k, top_p, uniform):
    if _use_cuda(logits):
        return _cuda().sample(logits, temperature, top_k, top_p, uniform)
    return ref.sample(logits, temperature, top_k, top_p, uniform)


def grouped_linear(x, w, tile_expert, expert_rows):
    """Per-expert linear over an expert-sorted token buffer whose expert groups start at multiples of 128 rows
    (see :func:`relax_b200.models.moe.padded_expert_layout`); ``w`` is ``[E, N, K]``."""
    if _use_cuda(x):
        return _cuda().grouped_linear(x, w, tile_expert, expert_rows)
    return ref.grouped_linear(x, w, tile_expert, expert_rows)


def decode_advance(tok_new, lp_new, state, block_size):
    """In-place advance of the rollout engine's device-resident batch state after one decode step."""
    if _use_cuda(tok_new):
        return _cuda().decode_advance(tok_new, lp_new, state, block_size)
    return ref.decode_advance(tok_new, lp_new, state, block_size)


def topk_router(logits, top_k, norm_topk_prob=True):
    if _use_cuda(logits):
        return _cuda().topk_router(logits, top_k, norm_topk_prob)
    return ref.topk_router(logits, top_k, norm_topk_prob)


def fused_lm_head_logprob(hidden, weight, targets, tp_group=None, vocab_start=0, with_entropy=True,
                          temperature=1.0, chunk_size=4096):
    """LM-head GEMM fused with online-softmax log-prob / entropy; ``[T, V]`` is never stored."""
    if _use_cuda(hidden):
        return _cuda().fused_lm_head_logprob(hidden, weight, targets, tp_group, vocab_start, with_entropy, temperature)
    from ..algo.logprob import chunked_log_probs_and_entropy

    return chunked_log_probs_and_entropy(hidden, weight, targets, tp_group, vocab_start, with_entropy,
                                         temperature, chunk_size)


def fake_int4_quant(x, block_m, block_n, sym=True):
    if _use_cuda(x):
        return _cuda().fake_int4_quant(x, block_m, block_n, sym)
    return ref.fake_int4_quant(x, block_m, block_n, sym)


def blockwise_cast_to_fp8(w, block=128, ue8m0=False):
    if _use_cuda(w):
        return _cuda().blockwise_cast_to_fp8(w, block, ue8m0)
    return ref.blockwise_cast_to_fp8(w, block, ue8m0)


def blockwise_dequant_fp8(q, scale_inv, block=128, dtype=None):
    import torch

    dtype = dtype or torch.bfloat16
    if _use_cuda(q):
        return _cuda().blockwise_dequant_fp8(q, scale_inv, block, dtype)
    return ref.blockwise_dequant_fp8(q, scale_inv, block, dtype)


def kv_cache_write(k, v, k_cache, v_cache, slots):
    """Scatter new K/V rows ``[T, Hkv, D]`` into a paged cache ``[blocks, block_size, Hkv, D]``
    at flat slot indices ``slots[T]`` (``block * block_size + offset``)."""
    if _use_cuda(k):
        return _cuda().kv_scatter(k, v, k_cache, v_cache, slots)
    kc = k_cache.view(-1, k.shape[1], k.shape[2])
    vc = v_cache.view(-1, v.shape[1], v.shape[2])
    kc[slots] = k
    vc[slots] = v


def qkv_post(qkv, nq, nkv, q_norm_w, k_norm_w, cos, sin, eps, k_cache=None, v_cache=None, slots=None, dense_kv=True):
    """Inference-side glue after the fused QKV projection: optional per-head RMSNorm of q and k, rotary
    embedding, and the write of the new K/V rows into the paged cache.  One kernel on CUDA (bf16,
    head_dim 128); the statement below elsewhere.  Returns ``(q, k, v)`` with ``k``/``v`` None when
    ``dense_kv`` is False (decode: attention reads the cache)."""
    hd = qkv.shape[1] // (nq + 2 * nkv)
    if (_use_cuda(qkv) and hd == 128 and qkv.dtype == torch.bfloat16 and not torch.is_grad_enabled()
            and cos.shape[-1] == 64):
        return _cuda().qkv_post(qkv, nq, nkv, q_norm_w, k_norm_w, cos, sin, eps, k_cache, v_cache, slots, dense_kv)
    T = qkv.shape[0]
    q = qkv[:, : nq * hd].reshape(T, nq, hd)
    k = qkv[:, nq * hd:(nq + nkv) * hd].reshape(T, nkv, hd)
    v = qkv[:, (nq + nkv) * hd:].reshape(T, nkv, hd)
    if q_norm_w is not None:
        q, k = rmsnorm(q, q_norm_w, eps), rmsnorm(k, k_norm_w, eps)
    rot = 2 * cos.shape[-1]
    if rot < hd:      # partial rotary (GLM-4, Qwen3.5): only the first ``rot`` dims of every head turn
        q = torch.cat([apply_rope(q[..., :rot].contiguous(), cos, sin), q[..., rot:]], -1)
        k = torch.cat([apply_rope(k[..., :rot].contiguous(), cos, sin), k[..., rot:]], -1)
    else:
        q, k = apply_rope(q, cos, sin), apply_rope(k, cos, sin)
    if slots is not None:
        kv_cache_write(k, v, k_cache, v_cache, slots)
    return (q, k, v.contiguous()) if dense_kv else (q, None, None)


def linear_swiglu(x, w):
    """``swiglu(x @ w.T)`` with ``w`` = [gate; up]; fused split-K reduction + activation for decode shapes."""
    if _use_cuda(x) and x.shape[0] <= 256 and not torch.is_grad_enabled() and x.dim() == 2:
        return _cuda().linear_swiglu_skinny(x, w)
    return swiglu(linear(x, w))


def fp8_linear(x, w_q, w_scale_inv, block: int = 128):
    """``x @ dequant(w_q, w_scale_inv)^T`` with block-scaled e4m3 operands (weights: one scale per ``block x block``
    tile; activations quantised per row and ``block`` columns on the fly).  tcgen05 ``kind::f8f6f4`` on CUDA;
    elsewhere the dequantised product."""
    if _use_cuda(x) and block == 128:
        return _cuda().fp8_linear(x, w_q, w_scale_inv)
    w = blockwise_dequant_fp8(w_q, w_scale_inv, block, torch.float32)
    return (x.float() @ w.float().t()).to(torch.bfloat16)


def dgrad(dy, w):
    """dy[M,N] @ w[N,K] (input gradient of ``linear``)."""
    if _use_cuda(dy):
        return _cuda().matmul_nn(dy.contiguous(), w)
    return dy @ w


def wgrad(dy, x, w=None):
    """dy[M,N]^T @ x[M,K] (weight gradient of ``linear``).  When ``w`` carries an fp32
    ``main_grad`` buffer the CUDA path accumulates into it and returns ``None``."""
    if _use_cuda(dy):
        c = _cuda()
        mg = getattr(w, "main_grad", None) if w is not None else None
        import torch

        if mg is not None and mg.dtype == torch.float32 and mg.shape == w.shape:
            c.matmul_tn(dy.contiguous(), x.contiguous(), out=mg, accumulate=True)
            return None
        return c.matmul_tn(dy.contiguous(), x.contiguous())
    return dy.t() @ x
