"""Plain-PyTorch statements of every hot operator.

These are (1) the CPU path, (2) the fp32 oracle every CUDA kernel is tested
against and (3) the unfused library baseline the fused kernels are timed
against.  They run through autograd, so they need no hand-written backward.
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F

# --------------------------------------------------------------------------- norms / activations


def rmsnorm(x, w, eps: float = 1e-6):
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (y * w.float()).to(x.dtype)


def add_rmsnorm(x, residual, w, eps: float = 1e-6):
    """``r = x + residual; y = rmsnorm(r)``; returns ``(y, r)``."""
    r = (x.float() + residual.float()).to(x.dtype)
    return rmsnorm(r, w, eps), r


def swiglu(gate_up):
    g, u = gate_up.chunk(2, dim=-1)
    return (F.silu(g.float()) * u.float()).to(gate_up.dtype)


def glu(gate_up, act: str = "silu"):
    """``act(gate) * up`` for ``gate_up = [gate | up]``; ``act``: ``silu`` or ``gelu_tanh``."""
    g, u = gate_up.chunk(2, dim=-1)
    g = g.float()
    a = F.silu(g) if act == "silu" else F.gelu(g, approximate="tanh")
    return (a * u.float()).to(gate_up.dtype)


def linear(x, w, bias=None):
    return F.linear(x, w, bias)


# --------------------------------------------------------------------------- composed stacks (fp32 residual, grouped output norms)


def group_rms(x, w, width: int, groups: int, eps: float):
    """RMS norm over each of ``groups`` equal parts of the first ``width`` columns; the columns behind them are padding
    and come out zero (their weights are).  fp32 in, fp32 out."""
    y = torch.zeros_like(x, dtype=torch.float32)
    p = x[:, :width].float().reshape(x.shape[0], groups, width // groups)
    p = p / torch.sqrt(p.pow(2).mean(-1, keepdim=True) + eps)
    y[:, :width] = p.reshape(x.shape[0], width) * w[:width].float()
    return y


def embed_rows(tokens, w, norm_w=None, width: int = 0, groups: int = 1, eps: float = 0.0, scale: float = 1.0):
    """``(fp32 residual stream, its copy in the weights' type)`` of embedded tokens, group-normed when ``norm_w`` is given, else times
    ``scale``."""
    h = w[tokens]
    if norm_w is None:
        res = h.float() * scale
        return res, res.to(w.dtype, copy=True)
    res = group_rms(h.float(), norm_w, width, groups, eps)
    return res, res.to(w.dtype)


def norm_add(res, y, w, width: int, groups: int, eps: float, next_w=None, experts=None):
    """``res += group_rms(y) * w`` in place (fp32); returns the next sublayer's input in ``w``'s type: the new stream
    itself, or its own group norm with ``next_w`` when given.  ``experts = (rows, plan)``: the weighted rows of
    :func:`moe_experts` join ``y`` (which may be None) first."""
    if experts is not None:
        z = expert_sum(res, experts)
        y = z if y is None else y.float() + z
    res += group_rms(y, w, width, groups, eps)
    return (res if next_w is None else group_rms(res, next_w, width, groups, eps)).to(w.dtype)


def expert_sum(res, experts):
    """Weighted sum over a token's experts; identity experts (choices behind the last expert) give back the stream itself."""
    rows, plan = experts
    z = (rows.float() * plan.weight[..., None]).sum(1)
    return z + res * (plan.weight * (plan.index >= plan.experts)).sum(1, keepdim=True)


def sum_norm(res, y, w, b, width: int, alpha: float, eps: float, nxt=None, scale: float = 1.0, experts=None):
    """``res <- norm(alpha res + y + experts)`` over the first ``width`` columns, in place (fp32): a layer norm with weight ``w`` and bias
    ``b``, RMS when ``b`` is None.  Returns the new stream in ``w``'s type, or its norm with ``nxt = (weight, bias)`` times ``scale``."""
    def norm(x, w, b):
        if b is not None:
            x = x - x.mean(-1, keepdim=True)
        x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w[:width].float()
        return x if b is None else x + b[:width].float()

    x = alpha * res[:, :width]
    if y is not None:
        x = x + y[:, :width].float()
    if experts is not None:
        x = x + expert_sum(res, experts)[:, :width]
    res[:, :width] = norm(x, w, b)
    h = torch.zeros(res.shape, dtype=w.dtype, device=res.device)
    h[:, :width] = res[:, :width] if nxt is None else norm(res[:, :width], *nxt) * scale
    return h


def hgrn2(qfv, f_bias, lower, norm_w, state, state_slot, ctx_lens, cu, heads: int, dim: int, vdim: int, eps: float):
    """HGRN2 recurrence on packed rows ``[q | f | v]`` (raw projections), state carried in ``state[slot, h, dim, >= vdim]``.
    Segment ``s`` owns rows ``cu[s]:cu[s+1]`` (``cu`` None: one row each), the last of them at position ``ctx_lens[s] - 1``;
    a segment that starts at position 0 starts from a zero state whatever its slot holds.

    ``g = lower + (1 - lower) sigmoid(f + bias)``;  ``S <- diag(g) S + (1 - g) v^T``;  ``o = S^T silu(q)``, RMS-normed."""
    T, qd = qfv.shape[0], heads * dim
    q = F.silu(qfv[:, :qd].float()).view(T, heads, dim)
    lo = lower.float()
    g = (lo + (1 - lo) * torch.sigmoid(qfv[:, qd:2 * qd].float() + f_bias.float())).view(T, heads, dim)
    v = qfv[:, 2 * qd:2 * qd + heads * vdim].float().reshape(T, heads, vdim)
    o = torch.zeros(T, (heads * vdim + 7) // 8 * 8, dtype=torch.float32, device=qfv.device)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for s, (a, b) in enumerate(zip(bounds, bounds[1:])):
        S = state[int(state_slot[s])][:, :, :vdim]
        cur = torch.zeros_like(S) if int(ctx_lens[s]) - (b - a) == 0 else S.clone()
        for t in range(a, b):
            cur = cur * g[t][:, :, None] + (1 - g[t])[:, :, None] * v[t][:, None, :]
            r = (cur * q[t][:, :, None]).sum(1)
            r = r / torch.sqrt(r.pow(2).mean(-1, keepdim=True) + eps) * norm_w[:vdim].float()
            o[t, : heads * vdim] = r.reshape(-1)
        S.copy_(cur)
    return o.to(qfv.dtype)


def turn_neighbours(x, table):
    """Pairs of neighbouring features ``x[T, ..., 2 n]`` turned by ``table[T, n, 2]`` (cos, sin)."""
    c, s = (table[..., k].view(table.shape[0], *[1] * (x.dim() - 2), -1) for k in (0, 1))
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def latent_write(raw, w, rank: int, eps: float, pool, slots, turned=None):
    """RMS-normed latent rows -> ``pool[slots]`` (columns behind ``rank`` zero, but for the rotated key part of ``turned``, whose query
    features turn in place)."""
    c = torch.zeros(raw.shape[0], pool.shape[1], dtype=torch.float32, device=raw.device)
    x = raw[:, :rank].float()
    c[:, :rank] = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w[:rank].float()
    if turned is not None:
        q, k_rot, table, part, rot, dim = turned
        c[:, part:part + rot] = turn_neighbours(k_rot[:, :rot].float(), table)
        q[..., dim:dim + rot] = turn_neighbours(q[..., dim:dim + rot].float(), table).to(q.dtype)
    pool[slots] = c.to(pool.dtype)


def head_linear(x, w, transposed: bool, gate=None):
    """Per-head product ``x[T, H, a] -> [T, H, b]`` with ``w[H, a, b]`` (``transposed``: ``w[H, b, a]``), times ``sigmoid(gate[T, H * b])``
    when given."""
    y = torch.einsum("tha,hba->thb" if transposed else "tha,hab->thb", x.float(), w.float())
    if gate is not None:
        y = y * torch.sigmoid(gate[:, : y.shape[1] * y.shape[2]].float()).view(y.shape)
    return y.to(w.dtype)


def latent_attention(q, pool, block_tables, block_size: int, ctx_lens, cu, scale: float, gate=None, rank: Optional[int] = None):
    """Softmax attention of absorbed queries ``q[T, H, R]`` over the paged latent rows of their sequence (each row is key, and its
    first ``rank`` features are the value, of every head); row ``i`` of a segment of ``n`` rows sees the first ``ctx - n + i + 1`` of
    them.  ``gate[T, H]``: every head's output is multiplied by its sigmoid."""
    T, H, R = q.shape
    rank = rank or R
    out = torch.zeros(T, H, rank, dtype=torch.float32, device=q.device)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for s, (a, b) in enumerate(zip(bounds, bounds[1:])):
        L = int(ctx_lens[s])
        pos = torch.arange(L, device=q.device)
        c = pool[block_tables[s].long()[pos // block_size] * block_size + pos % block_size].float()
        sc = torch.einsum("thr,lr->thl", q[a:b].float(), c) * scale
        lim = L - (b - a) + torch.arange(b - a, device=q.device)
        sc = sc.masked_fill(pos[None, None, :] > lim[:, None, None], float("-inf"))
        out[a:b] = torch.einsum("thl,lr->thr", torch.softmax(sc, -1), c[:, :rank])
    if gate is not None:
        out = out * torch.sigmoid(gate.float())[..., None]
    return out.to(q.dtype)


def rope_table(positions, offset: int, inv_freq):
    """cos / sin ``[T, pairs, 2]`` (fp32) of the angles ``(position + offset) * inv_freq`` (fp64, so that late positions keep
    their low bits)."""
    a = (positions.double() + offset)[:, None] * inv_freq[None, :]
    return torch.stack([torch.cos(a), torch.sin(a)], -1).float()


def attention_inputs(qkv, table, heads: int, kv_heads: int, dim: int, vdim: int, dp: int, rot_dims: int, eps: float, k_pool, v_pool, slots):
    """Raw projections ``[q heads | k heads | v heads]`` -> queries ``[T, heads, dp]`` and rows of the paged key / value pools
    ``[rows, kv_heads, >= dim]``; ``k_pool`` None: the rows hold queries only.  The first ``rot_dims`` features of queries and
    keys turn in neighbouring pairs; ``eps`` > 0: they are then divided by their root mean square."""
    def head(x, norm_and_turn=True):
        x = x.float()
        if norm_and_turn:
            if rot_dims:
                c, s = table[:, None, :, 0], table[:, None, :, 1]
                u, v = x[..., 0:rot_dims:2], x[..., 1:rot_dims:2]
                x = torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., rot_dims:]], -1)
            if eps > 0:
                x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
        return x

    T, qd, kd = qkv.shape[0], heads * dim, kv_heads * dim
    q = torch.zeros(T, heads, dp, dtype=qkv.dtype, device=qkv.device)
    q[..., :dim] = head(qkv[:, :qd].view(T, heads, dim)).to(qkv.dtype)
    if k_pool is not None:
        k_pool[slots, :, :dim] = head(qkv[:, qd:qd + kd].view(T, kv_heads, dim)).to(k_pool.dtype)
        v_pool[slots, :, :vdim] = qkv[:, qd + kd:qd + kd + kv_heads * vdim].view(T, kv_heads, vdim).to(v_pool.dtype)
    return q


def projection_inputs(qkv, q_w, k_w, table, heads: int, kv_heads: int, dim: int, vdim: int, dp: int, rot_dims: int, halves: bool, eps: float, k_pool,
                      v_pool, slots):
    """Like :func:`attention_inputs` with RMS norms (weights ``q_w``, ``k_w``) over all query columns and over all key columns, before
    heads and rotation; ``halves``: features ``i`` and ``i + rot_dims / 2`` turn together."""
    def heads_of(x, w, n):
        x = x.float()
        if eps > 0:
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
            if w is not None:
                x = x * w.float()
        x = x.view(x.shape[0], n, dim)
        if not rot_dims:
            return x
        r, half = x[..., :rot_dims], rot_dims // 2
        if halves:
            c, s = table[:, None, :, 0], table[:, None, :, 1]
            u, v = r[..., :half], r[..., half:]
            r = torch.cat([u * c - v * s, v * c + u * s], -1)
        else:
            r = turn_neighbours(r, table)
        return torch.cat([r, x[..., rot_dims:]], -1)

    T, qd, kd = qkv.shape[0], heads * dim, kv_heads * dim
    q = torch.zeros(T, heads, dp, dtype=qkv.dtype, device=qkv.device)
    q[..., :dim] = heads_of(qkv[:, :qd], q_w, heads).to(qkv.dtype)
    if k_pool is not None:
        k_pool[slots, :, :dim] = heads_of(qkv[:, qd:qd + kd], k_w, kv_heads).to(k_pool.dtype)
        v_pool[slots, :, :vdim] = qkv[:, qd + kd:qd + kd + kv_heads * vdim].view(T, kv_heads, vdim).to(v_pool.dtype)
    return q


def paged_attention(q, k_pool, v_pool, block_tables, block_size: int, ctx_lens, cu, scale: float, sink, out_width: int, window: int = 0, gate=None,
                    keep: int = 0, chunk: int = 0, softcap: float = 0.0, talk=None):
    """Softmax attention of ``q[T, H, dp]`` over paged keys and values ``[rows, kv_heads, ...]`` of their sequence; row ``i`` of
    a segment of ``n`` rows sees the first ``ctx - n + i + 1`` positions, with a ``window`` only the last ``window`` of those and the first
    ``keep`` of the sequence, with a ``chunk`` only those of its own chunk.  ``softcap``: scores ``s`` become ``softcap tanh(s / softcap)``.
    ``sink[H]``: a logit per head that only joins the denominator.  ``talk[H, H]``: mixes the heads' weights before they meet the values.
    ``gate[T, H * out_width]``: its sigmoid multiplies the outputs.  Returns ``[T, H * out_width]``."""
    T, H, _ = q.shape
    G, rep = k_pool.shape[1], H // k_pool.shape[1]
    out = torch.zeros(T, H, out_width, dtype=torch.float32, device=q.device)
    w = min(out_width, v_pool.shape[2])
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for s, (a, b) in enumerate(zip(bounds, bounds[1:])):
        L = int(ctx_lens[s])
        pos = torch.arange(L, device=q.device)
        rows = block_tables[s].long()[pos // block_size] * block_size + pos % block_size
        k, v = k_pool[rows].float(), v_pool[rows].float()[..., :w]
        sc = torch.einsum("tgrd,lgd->tgrl", q[a:b].float().view(b - a, G, rep, -1), k).reshape(b - a, H, L) * scale
        if softcap:
            sc = softcap * torch.tanh(sc / softcap)
        lim = (L - (b - a) + torch.arange(b - a, device=q.device))[:, None, None]
        sc = sc.masked_fill(pos > lim, float("-inf"))
        if window:
            sc = sc.masked_fill((pos <= lim - window) & (pos >= keep), float("-inf"))
        if chunk:
            sc = sc.masked_fill(pos < lim // chunk * chunk, float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.float()[None, :, None].expand(b - a, H, 1)], -1)
        p = torch.softmax(sc, -1)[..., :L]
        if talk is not None:
            p = torch.einsum("hg,tgl->thl", talk.float(), p)
        p = p.reshape(b - a, G, rep, L)
        out[a:b, :, :w] = torch.einsum("tgrl,lgd->tgrd", p, v).reshape(b - a, H, w)
    out = out.reshape(T, H * out_width)
    return (out if gate is None else out * torch.sigmoid(gate[:, : H * out_width].float())).to(q.dtype)


class ExpertPlan:
    """Which experts every row takes, ``index [T, top]`` (from ``experts`` on: identity experts), and with which ``weight [T, top]``."""

    def __init__(self, index, weight, experts: int):
        self.index, self.weight, self.experts = index, weight, experts


def moe_route(logits, spec, correction=None):
    """Sigmoid or softmax scores; with ``correction`` added, the ``spec.keep`` groups with the largest sums of their ``spec.group_best``
    best scores stay, and of their outputs the ``spec.top`` best are taken."""
    z = logits[:, : spec.outputs].float()
    s = torch.softmax(z, -1) if spec.score == "softmax" else torch.sigmoid(z)
    choice = s if correction is None else s + correction[: spec.outputs].float()
    T, n = s.shape[0], spec.outputs // spec.groups
    best = choice.view(T, spec.groups, n).topk(min(spec.group_best, n), -1).values.sum(-1)
    open_ = torch.zeros(T, spec.groups, dtype=torch.bool, device=s.device).scatter_(1, best.topk(spec.keep, -1).indices, True)
    idx = choice.masked_fill(~open_.repeat_interleave(n, 1), float("-inf")).topk(spec.top, -1).indices
    w = s.gather(-1, idx)
    if spec.renormalize:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ExpertPlan(idx, w * spec.weight_scale, spec.experts)


def relu2(x):
    return torch.relu(x.float()).pow(2).to(x.dtype)


def clamped_swish(gate_up, limit: float):
    """``g sigmoid(1.702 g) (u + 1)`` of bounded halves; columns alternate between 32 gates and the 32 units they belong to."""
    g, u = gate_up.float().view(gate_up.shape[0], -1, 2, 32).unbind(2)
    g, u = g.clamp(max=limit), u.clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).flatten(1).to(gate_up.dtype)


def swiglu_runs(gate_up):
    """``silu(g) u`` of halves in alternating runs of 32 columns."""
    g, u = gate_up.float().view(gate_up.shape[0], -1, 2, 32).unbind(2)
    return (F.silu(g) * u).flatten(1).to(gate_up.dtype)


def moe_experts(h, plan, up, down, act: str, limit: float = 0.0):
    """Outputs ``down_e act(up_e h)`` of every row's experts, unweighted: ``[T, top, W]`` (zero for identity experts)."""
    T, k = plan.index.shape
    out = torch.zeros(T, k, down.shape[1], dtype=h.dtype, device=h.device)
    for e in plan.index.unique().tolist():
        if e >= plan.experts:
            continue
        t, j = (plan.index == e).nonzero(as_tuple=True)
        y = F.linear(h[t], up[e])
        out[t, j] = F.linear(relu2(y) if act == "relu2" else swiglu_runs(y) if act == "swiglu" else clamped_swish(y, limit), down[e])
    return out


def _segments(b, T: int) -> list:
    """``(first row, last row + 1, position of the first row, state slot)`` of a batch's segments."""
    bounds = list(range(T + 1)) if b.cu is None else b.cu.tolist()
    return [(a, e, int(n) - (e - a), int(s)) for a, e, n, s in zip(bounds, bounds[1:], b.ctx.tolist(), b.state_slot.tolist())]


def conv_inputs(qkv, bias, taps, state, b, q_w, k_w, table, heads: int, kv_heads: int, dim: int, vdim: int, dp: int, rot_dims: int, eps: float, k_pool,
                v_pool):
    """Like :func:`attention_inputs` with biases ``bias[channels]``, then a causal convolution over a sequence's rows (``taps[channels, n]``,
    the last tap on the row itself; ``state[slot, n - 1, channels]``: the rows before a segment, without biases, replaced by its last
    ones), then RMS norms head by head with weights (``eps`` > 0), then the rotation of neighbours."""
    T, C = qkv.shape[0], heads * dim + (kv_heads * (dim + vdim) if k_pool is not None else 0)
    add = 0.0 if bias is None else bias[:C].float()
    y = torch.empty(T, C, dtype=torch.float32, device=qkv.device)
    n = 1 if taps is None else taps.shape[1]
    for lo, hi, pos, slot in _segments(b, T):
        u = qkv[lo:hi, :C]
        if n == 1:
            y[lo:hi] = (u.float() + add) * (1.0 if taps is None else taps[:, 0].float())
            continue
        before = state[slot] if pos else torch.zeros_like(state[slot])
        rows = torch.cat([before, u.to(state.dtype)])
        x = rows.float() + add
        x[: max(0, n - 1 - pos)] = 0.0               # rows before the sequence's start have no bias either
        y[lo:hi] = sum(taps[:, j].float() * x[j:j + hi - lo] for j in range(n))
        state[slot] = rows[hi - lo:]

    def head(x, w):
        if eps > 0:
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        return torch.cat([turn_neighbours(x[..., :rot_dims], table), x[..., rot_dims:]], -1) if rot_dims else x

    qd, kd = heads * dim, kv_heads * dim
    q = torch.zeros(T, heads, dp, dtype=qkv.dtype, device=qkv.device)
    q[..., :dim] = head(y[:, :qd].view(T, heads, dim), q_w).to(qkv.dtype)
    if k_pool is not None:
        k_pool[b.slots, :, :dim] = head(y[:, qd:qd + kd].view(T, kv_heads, dim), k_w).to(k_pool.dtype)
        v_pool[b.slots, :, :vdim] = y[:, qd + kd:].view(T, kv_heads, vdim).to(v_pool.dtype)
    return q


def mingru(zxg, z_b, x_b, state, b, width: int):
    """Gated running means ``S <- (1 - z) S + z c`` per channel, ``z = sigmoid(z_t + z_b)`` and ``c`` = ``u + 1/2`` or (``u`` < 0)
    ``sigmoid(u)`` of ``u = x_t + x_b``; rows ``[z | x | g]`` whose parts are padded to 8 columns.  Returns ``S silu(g)``, padded alike."""
    T, n = zxg.shape[0], (width + 7) // 8 * 8
    z, u, g = (zxg[:, k * n:k * n + width].float() for k in range(3))
    z, u = torch.sigmoid(z + z_b[:width].float()), u + x_b[:width].float()
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = torch.zeros(T, n, dtype=torch.float32, device=zxg.device)
    for lo, hi, pos, slot in _segments(b, T):
        S = state[slot].view(-1)[:width]
        S = S.clone() if pos else torch.zeros_like(S)
        for t in range(lo, hi):
            S = (1 - z[t]) * S + z[t] * c[t]
            out[t, :width] = S * F.silu(g[t])
        state[slot].view(-1)[:width] = S
    return out.to(zxg.dtype)


def gla(rows, z, a2_b, norm_w, state, state_slot, ctx_lens, cu, heads: int, dim: int, vdim: int, gate_col: int, eps: float, root: float):
    """Linear attention ``S <- diag(alpha) S + k v^T``, read-outs ``S^T q dim^-1/2``, with ``alpha = sigmoid(z + a2_b) ** (1 / root)`` per key
    channel; read-outs normed head by head, times ``silu`` of the gates.  Rows ``[q | k | v | .. gate_col: g]``."""
    T, qd, vd = rows.shape[0], heads * dim, heads * vdim
    q, k, v = rows[:, : 2 * qd + vd].float().split([qd, qd, vd], 1)
    q, k, v = q.view(T, heads, dim) * dim ** -0.5, k.view(T, heads, dim), v.view(T, heads, vdim)
    alpha = torch.exp(F.logsigmoid(z[:, :qd].float() + a2_b.float()) / root).view(T, heads, dim)
    o = torch.zeros(T, heads, vdim, dtype=torch.float32, device=rows.device)
    bounds = list(range(T + 1)) if cu is None else cu.tolist()
    for s, (a, b) in enumerate(zip(bounds, bounds[1:])):
        S = state[state_slot[s], :, :, :vdim]
        cur = torch.zeros_like(S) if int(ctx_lens[s]) == b - a else S.clone()
        for t in range(a, b):
            cur = alpha[t][..., None] * cur + k[t][..., None] * v[t][:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", cur, q[t])
        S.copy_(cur)
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
    out = torch.zeros(T, (vd + 7) // 8 * 8, dtype=torch.float32, device=rows.device)
    out[:, :vd] = o.reshape(T, vd) * F.silu(rows[:, gate_col:gate_col + vd].float())
    return out.to(rows.dtype)


def stream_step(res, width: int, eps: float, y=None, norm_w=None, experts=None, norms=(), shift=None):
    """``res += ...`` (see :func:`relax_b200.ops.stream_step`)."""
    dt = norms[0].dtype if norms else y[0].dtype
    x = res[:, :width]
    if y is not None:
        parts = [a[:, :width].float() for a in y]
        if norm_w is not None:
            parts = [a / torch.sqrt(a.pow(2).mean(-1, keepdim=True) + eps) * w[:width].float() for a, w in zip(parts, norm_w)]
        x += sum(parts) / len(parts)
    if experts is not None:
        rows, plan = experts
        x += (rows[..., :width].float() * plan.weight[..., None]).sum(1)
    out = []
    for w in norms or (None,):
        h = torch.zeros(res.shape, dtype=torch.float32, device=res.device)
        d = x - x.mean(-1, keepdim=True)
        h[:, :width] = x if w is None else d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w[:width].float()
        out.append(h.to(dt))
    if shift is not None:
        mu, state, b = shift
        n, mixed = out[0], torch.empty_like(out[0])
        for lo, hi, pos, slot in _segments(b, n.shape[0]):
            first = state[slot] if pos else torch.zeros_like(state[slot])
            before = torch.cat([first[None], n[lo:hi - 1]]).float()
            mixed[lo:hi] = (n[lo:hi].float() + (before - n[lo:hi].float()) * mu.float()).to(dt)
            state[slot] = n[hi - 1]
        out[0] = mixed
    return out


def side_gate(z, embed, tokens, first: int, dim: int):
    """``gelu_tanh(z) * e`` of the tokens' features ``first .. first + dim`` in a second embedding, padded to 8 columns."""
    out = torch.zeros(z.shape[0], (dim + 7) // 8 * 8, dtype=torch.float32, device=z.device)
    out[:, :dim] = F.gelu(z[:, :dim].float(), approximate="tanh") * embed[tokens, first:first + dim].float()
    return out.to(z.dtype)


def softcap(z, cap: float):
    return cap * torch.tanh(z.float() / cap)


# --------------------------------------------------------------------------- rotary embedding


def rope_cos_sin(positions, head_dim: int, theta: float, mrope_section=None):
    """cos/sin tables ``[T, head_dim/2]`` (fp32).  ``positions`` is ``[T]`` or,
    for multimodal M-RoPE, ``[3, T]`` (temporal, height, width) with
    ``mrope_section`` giving how many of the ``head_dim/2`` frequencies follow
    each of the three position streams."""
    half = head_dim // 2
    inv = 1.0 / (theta ** (torch.arange(0, half, device=positions.device, dtype=torch.float32) / half))
    if positions.dim() == 1:
        ang = positions.float()[:, None] * inv[None, :]
    else:
        assert mrope_section is not None and sum(mrope_section) == half
        ang3 = positions.float()[:, :, None] * inv[None, None, :]  # [3, T, half]
        parts, s = [], 0
        for i, n in enumerate(mrope_section):
            parts.append(ang3[i, :, s : s + n])
            s += n
        ang = torch.cat(parts, -1)
    return ang.cos(), ang.sin()


def apply_rope(x, cos, sin):
    """Rotate-half (NeoX) convention on ``x[T, H, D]``."""
    d = x.shape[-1] // 2
    xf = x.float()
    x1, x2 = xf[..., :d], xf[..., d:]
    c, s = cos[:, None, :], sin[:, None, :]
    return torch.cat([x1 * c - x2 * s, x2 * c + x1 * s], -1).to(x.dtype)


# --------------------------------------------------------------------------- attention


def attention_varlen(q, k, v, cu_seqlens, causal: bool = True, scale: Optional[float] = None,
                     cu_seqlens_k=None, return_lse: bool = False):
    """Packed variable-length attention.  q ``[Tq, Hq, D]``, k/v ``[Tk, Hkv, D]``;
    sequence ``i`` owns rows ``cu[i]:cu[i+1]``.  With ``causal`` the last query
    of a sequence is aligned with its last key (bottom-right alignment), so a
    shorter query block attends to a longer key prefix correctly."""
    Hq, Hkv, D = q.shape[1], k.shape[1], q.shape[2]
    g = Hq // Hkv
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    cu_q = cu_seqlens.tolist()
    cu_k = (cu_seqlens_k if cu_seqlens_k is not None else cu_seqlens).tolist()
    outs, lses = [], []
    for i in range(len(cu_q) - 1):
        qs = q[cu_q[i] : cu_q[i + 1]].float().transpose(0, 1)  # [Hq, Lq, D]
        ks = k[cu_k[i] : cu_k[i + 1]].float().transpose(0, 1).repeat_interleave(g, 0)
        vs = v[cu_k[i] : cu_k[i + 1]].float().transpose(0, 1).repeat_interleave(g, 0)
        s = torch.einsum("hqd,hkd->hqk", qs, ks) * scale
        if causal:
            Lq, Lk = qs.shape[1], ks.shape[1]
            qi = torch.arange(Lq, device=q.device)[:, None] + (Lk - Lq)
            ki = torch.arange(Lk, device=q.device)[None, :]
            s = s.masked_fill(ki > qi, float("-inf"))
        lse = torch.logsumexp(s, -1)
        p = torch.exp(s - lse[..., None])
        outs.append(torch.einsum("hqk,hkd->hqd", p, vs).transpose(0, 1))
        lses.append(lse.transpose(0, 1))
    o = torch.cat(outs, 0).to(q.dtype)
    if return_lse:
        return o, torch.cat(lses, 0)
    return o


def paged_decode_attention(q, k_cache, v_cache, block_tables, context_lens, scale: Optional[float] = None):
    """One query token per sequence against a paged KV cache.

    q ``[B, Hq, D]``; caches ``[num_blocks, block_size, Hkv, D]``;
    ``block_tables [B, max_blocks]`` int32; ``context_lens [B]`` (including the
    current token, whose K/V must already be in the cache)."""
    B, Hq, D = q.shape
    bs, Hkv = k_cache.shape[1], k_cache.shape[2]
    g = Hq // Hkv
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    out = torch.empty_like(q)
    for b in range(B):
        L = int(context_lens[b])
        nb = (L + bs - 1) // bs
        blocks = block_tables[b, :nb].long()
        ks = k_cache[blocks].reshape(-1, Hkv, D)[:L].float()
        vs = v_cache[blocks].reshape(-1, Hkv, D)[:L].float()
        qq = q[b].float().view(Hkv, g, D)
        s = torch.einsum("hgd,lhd->hgl", qq, ks) * scale
        p = torch.softmax(s, -1)
        out[b] = torch.einsum("hgl,lhd->hgd", p, vs).reshape(Hq, D).to(q.dtype)
    return out


# --------------------------------------------------------------------------- sampling / routing


def sample(logits, temperature, top_k, top_p, uniform):
    """Sample one token per row.  ``temperature/top_k/top_p`` are per-row tensors
    (top_k <= 0 disables, top_p >= 1 disables); ``uniform [B]`` are U(0,1)
    draws supplied by the caller so the op is deterministic.  Returns
    ``(token[B], log_prob[B])`` where the log-prob is that of the *unfiltered*
    temperature-scaled distribution (what the trainer recomputes)."""
    z = logits.float() / temperature.float().clamp_min(1e-6)[:, None]
    logp_full = torch.log_softmax(z, -1)
    greedy = temperature <= 0
    V = z.shape[-1]
    # kept set: the k largest, then the shortest prefix (descending order) of those whose
    # renormalised mass reaches top_p
    sorted_z, idx = torch.sort(z, -1, descending=True)
    ranks = torch.arange(V, device=z.device)[None, :]
    k = torch.where(top_k > 0, top_k, torch.full_like(top_k, V))
    keep = ranks < k[:, None]
    probs = torch.softmax(sorted_z.masked_fill(~keep, float("-inf")), -1)
    csum = torch.cumsum(probs, -1)
    keep &= (csum - probs) < top_p.float()[:, None]
    mask = torch.zeros_like(keep).scatter(-1, idx, keep)
    # inverse CDF in vocabulary order over the kept entries
    e = torch.exp(z - z.max(-1, keepdim=True).values) * mask
    c = torch.cumsum(e.double(), -1)
    target = uniform.double()[:, None] * c[:, -1:]
    pick = (c <= target).sum(-1).clamp_max(V - 1)
    # rounding at the end of the CDF must not select a filtered slot
    last_kept = (mask * torch.arange(V, device=z.device)[None, :]).amax(-1)
    tok = torch.minimum(pick, last_kept)
    tok = torch.where(greedy, z.argmax(-1), tok)
    return tok, logp_full.gather(-1, tok[:, None])[:, 0]


def grouped_linear(x, w, tile_expert, expert_rows):
    """``y[row] = x[row] @ w[e].T`` for the rows of expert ``e`` (``expert_rows[e] : expert_rows[e + 1]`` of the padded,
    expert-sorted buffer); rows outside every expert's range stay zero."""
    y = x.new_zeros(x.shape[0], w.shape[1])
    bounds = expert_rows.tolist()
    parts = []
    for e in range(w.shape[0]):
        a, b = bounds[e], bounds[e + 1]
        parts.append(x[a:b] @ w[e].t().to(x.dtype))
    tail = x.new_zeros(x.shape[0] - bounds[w.shape[0]], w.shape[1]) + 0.0 * w.sum().to(x.dtype)
    return torch.cat(parts + [tail]) if parts else y


def decode_advance(tok_new, lp_new, st, block_size: int):
    """Turn the tokens sampled by one decode step into the next step's inputs, in place, without the host.

    ``st`` holds the batch state, one entry per row: ``tok`` (next input token), ``pos`` (its position), ``ctx``
    (context length including it), ``slots`` (its KV-cache row), ``bt`` (block table ``[B, max_blocks]``), ``active``
    (0 once the row stopped), ``remain`` (tokens it may still emit), ``eos`` (-1: none), ``stop`` (``[B, n]`` extra
    stop ids, -1 padding); the window ring ``out_tok`` / ``out_lp`` ``[W, B]`` with its write index ``counter``; the
    uniform draws of the whole window ``u_all [W, B]`` and of the coming step ``u [B]``.  Rows that already stopped
    append -1 and change nothing."""
    c = int(st["counter"][0])
    W = st["out_tok"].shape[0]
    if c >= W:
        return
    act = st["active"] != 0
    st["out_tok"][c] = torch.where(act, tok_new, torch.full_like(tok_new, -1))
    st["out_lp"][c] = torch.where(act, lp_new, torch.zeros_like(lp_new))
    left = st["remain"] - act.to(st["remain"].dtype)
    stop = (st["eos"] >= 0) & (tok_new == st["eos"])
    if st["stop"].shape[1]:
        stop = stop | ((st["stop"] >= 0) & (st["stop"] == tok_new[:, None])).any(-1)
    p = st["pos"] + 1
    blk = p // block_size
    fits = blk < st["bt"].shape[1]
    go = act & ~stop & (left > 0) & fits
    new_slot = st["bt"].gather(1, blk.clamp_max(st["bt"].shape[1] - 1)[:, None].long())[:, 0].long() * block_size + p % block_size
    st["tok"].copy_(torch.where(go, tok_new, st["tok"]))
    st["pos"].copy_(torch.where(go, p, st["pos"]))
    st["ctx"].copy_(torch.where(go, (p + 1).to(st["ctx"].dtype), st["ctx"]))
    st["slots"].copy_(torch.where(go, new_slot, st["slots"]))
    st["active"].copy_((go).to(st["active"].dtype))
    st["remain"].copy_(left)
    if c + 1 < W:
        st["u"].copy_(st["u_all"][c + 1])
    st["counter"] += 1


def topk_router(logits, top_k: int, norm_topk_prob: bool = True):
    """fp32 softmax over experts then top-k; returns ``(weights[T,k], idx[T,k], probs[T,E])``."""
    p = torch.softmax(logits.float(), -1)
    w, idx = torch.topk(p, top_k, dim=-1)
    if norm_topk_prob:
        w = w / w.sum(-1, keepdim=True)
    return w, idx, p


# --------------------------------------------------------------------------- optimizer


def adam_step(p32, g, m, v, step: int, lr: float, beta1: float, beta2: float, eps: float, weight_decay: float,
              grad_scale: float = 1.0):
    """AdamW on fp32 master weights (decoupled decay, bias correction)."""
    gf = g.float() * grad_scale
    m.mul_(beta1).add_(gf, alpha=1 - beta1)
    v.mul_(beta2).addcmul_(gf, gf, value=1 - beta2)
    bc1 = 1 - beta1**step
    bc2 = 1 - beta2**step
    denom = (v / bc2).sqrt_().add_(eps)
    p32.mul_(1 - lr * weight_decay).addcdiv_(m / bc1, denom, value=-lr)
    return p32


# --------------------------------------------------------------------------- quantisers


def fake_int4_quant(x, block_m: int, block_n: int, sym: bool = True):
    """Group-wise int4 fake quantisation.  Groups are ``block_m x block_n`` tiles
    of the 2-D input.  Symmetric: ``scale = absmax/7``, q in [-8, 7] (round to
    nearest even); asymmetric: ``scale = (max-min)/15`` with an integer
    zero-point, q in [0, 15].  Returns ``(dequantised, scale, zero)`` in the
    input dtype; scale/zero have one entry per group."""
    M, N = x.shape
    gm, gn = (M + block_m - 1) // block_m, (N + block_n - 1) // block_n
    xp = x.float()
    if M % block_m or N % block_n:
        xp = F.pad(xp, (0, gn * block_n - N, 0, gm * block_m - M))
    t = xp.view(gm, block_m, gn, block_n).permute(0, 2, 1, 3).reshape(gm, gn, -1)
    valid = torch.ones(gm * block_m, gn * block_n, dtype=torch.bool, device=x.device)
    valid[M:, :] = False
    valid[:, N:] = False
    vm = valid.view(gm, block_m, gn, block_n).permute(0, 2, 1, 3).reshape(gm, gn, -1)
    if sym:
        amax = torch.where(vm, t.abs(), torch.zeros_like(t)).amax(-1)
        scale = (amax / 7.0).clamp_min(1e-5)
        q = torch.round(t / scale[..., None]).clamp(-8, 7)
        dq = q * scale[..., None]
        zero = torch.zeros_like(scale)
    else:
        tmax = torch.where(vm, t, torch.full_like(t, -float("inf"))).amax(-1)
        tmin = torch.where(vm, t, torch.full_like(t, float("inf"))).amin(-1)
        scale = ((tmax - tmin) / 15.0).clamp_min(1e-5)
        zero = torch.round(-tmin / scale).clamp(0, 15)
        q = (torch.round(t / scale[..., None]) + zero[..., None]).clamp(0, 15)
        dq = (q - zero[..., None]) * scale[..., None]
    out = dq.view(gm, gn, block_m, block_n).permute(0, 2, 1, 3).reshape(gm * block_m, gn * block_n)[:M, :N]
    return out.to(x.dtype), scale.to(x.dtype), zero.to(x.dtype)


FP8_E4M3_MAX = 448.0


def blockwise_cast_to_fp8(w, block: int = 128, ue8m0: bool = False):
    """Per ``block x block`` absmax scaling to e4m3.  Returns ``(w_fp8, scale_inv)``
    with ``w ~= w_fp8 * scale_inv[block]``; ``ue8m0`` rounds the scale up to a
    power of two (the MX-style exponent-only scale format)."""
    M, N = w.shape
    gm, gn = (M + block - 1) // block, (N + block - 1) // block
    wp = F.pad(w.float(), (0, gn * block - N, 0, gm * block - M))
    t = wp.view(gm, block, gn, block)
    amax = t.abs().amax(dim=(1, 3)).clamp_min(1e-12)
    scale = amax / FP8_E4M3_MAX
    if ue8m0:
        scale = torch.exp2(torch.ceil(torch.log2(scale)))
    q = (t / scale[:, None, :, None]).clamp(-FP8_E4M3_MAX, FP8_E4M3_MAX)
    q = q.reshape(gm * block, gn * block)[:M, :N].to(torch.float8_e4m3fn)
    return q, scale


def blockwise_dequant_fp8(q, scale_inv, block: int = 128, dtype=torch.bfloat16):
    M, N = q.shape
    s = scale_inv.repeat_interleave(block, 0)[:M].repeat_interleave(block, 1)[:, :N]
    return (q.float() * s).to(dtype)
