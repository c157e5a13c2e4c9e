"""Composed stacks in the rollout engine: cache, batch description, forward and scheduling.

A composed stack (``ModelConfig.layer_specs``) mixes layers whose memory of the past differs in kind:

* recurrent layers keep one fp32 matrix per head and sequence (running means: one row), in a STATE SLOT of a fixed pool
  (:class:`StackCache.state`);
* short convolutions and shifted tokens keep the last rows they have read in the same slots (:class:`StackCache.conv`, ``shift``);
* latent-attention layers keep one row per token in PAGES of the engine's block manager (:class:`StackCache.latent`): the latent
  features and, where positions are rotated in, one rotated key part behind them;
* attention layers keep a key and a value row per token and key / value head in the same pages (:class:`StackCache.kv`), unless
  they read the rows of an earlier layer.

One forward (:meth:`ComposedForward.forward_segments`) runs a batch of SEGMENTS - the next ``n >= 1`` tokens of several
sequences, prompt portions beside single decoded tokens - from what earlier forwards left in slots and pages.  The engine's
scheduler cuts prompts into portions with it; pure decode batches take the same layers through the engine's captured
windows (:meth:`ComposedForward.forward_step`).
"""
from __future__ import annotations

import math
from collections import deque
from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from .. import ops
from ..models.config import ModelConfig
from ..models.native import pad_to

LONG_PORTION = 192     # portions of at least this many rows attend through projected keys / values (flash attention)


def head_pitch(n: int) -> int:
    """Columns a head of ``n`` features takes in the key / value pools and in the queries: the widths of the tensor-core kernels,
    beyond them 16-byte rows.  Padding stays zero."""
    return 64 if n <= 64 else (128 if n <= 128 else pad_to(n, 8))


def latent_row(spec) -> int:
    """Columns of a cached latent row: latent features, then the rotated key part, each in whole 64-column chunks."""
    return pad_to(spec.kv_rank, 64) + pad_to(spec.rot_dims, 64)


def projected(spec) -> int:
    """Columns of an attention layer's query, key and value projections."""
    return spec.heads * spec.dim + (spec.kv_heads * (spec.dim + spec.vdim) if spec.own_kv else 0)


class SlotManager:
    """Fixed pool of state slots, one per live sequence."""

    def __init__(self, n: int):
        self.n, self.free, self.used = n, deque(range(n)), set()

    @property
    def num_free(self) -> int:
        return len(self.free)

    def alloc(self) -> int:
        if not self.free:
            raise RuntimeError("no state slot is free")
        s = self.free.popleft()
        self.used.add(s)
        return s

    def release(self, s: int):
        if s not in self.used:
            raise RuntimeError(f"state slot {s} released twice")
        self.used.remove(s)
        self.free.append(s)


class StackCache:
    """The pools of a composed stack, by mixer (:meth:`ModelConfig.mixers`).  ``latent[key]``: ``[blocks * block_size, latent_row]`` rows in
    the model's type; ``kv[key]``: keys and values ``[blocks * block_size, kv heads, padded width]``, one pair for the layer that computes
    them and all that read them; ``state[key]``: ``[slots, heads, dim, padded vdim]`` fp32; ``conv[key]``: the last ``taps - 1`` projected
    rows ``[slots, taps - 1, channels]``; ``shift[layer]``: the mixer's last input row ``[slots, width]``.  All of it lives in ONE buffer."""

    def __init__(self, cfg: ModelConfig, num_blocks: int, block_size: int, num_slots: int, dtype, device, memory_saver: bool):
        self.block_size = block_size
        views, n = [], 0
        es = torch.empty(0, dtype=dtype).element_size()
        rows = num_blocks * block_size

        def room(key, kind, shape, dt, size):
            nonlocal n
            views.append((key, kind, shape, dt, n))
            n += pad_to(math.prod(shape) * size, 1024)

        for key, s in cfg.mixers():
            if s.mixer in ("hgrn2", "gla", "mingru"):
                room(key, "state", (num_slots, s.heads, s.dim, pad_to(s.vdim, 4)), torch.float32, 4)
            elif s.mixer == "latent_attention":
                room(key, "latent", (rows, latent_row(s)), dtype, es)
            else:
                if s.own_kv:
                    for k, d in (("k", s.dim), ("v", s.vdim)):
                        room(key, k, (rows, s.kv_heads, head_pitch(d)), dtype, es)
                if s.conv > 1:
                    room(key, "conv", (num_slots, s.conv - 1, projected(s)), dtype, es)
        if cfg.token_shift:
            for i in range(cfg.num_layers):
                room(i, "shift", (num_slots, pad_to(cfg.hidden_size, 64)), dtype, es)
        self.nbytes = n
        self.buf = None
        if memory_saver:
            from ..utils.memory_saver import PausableBuffer

            self.buf = PausableBuffer(n, device)
            make = lambda shape, dt, off: self.buf.tensor(shape, dt, off)
        else:
            flat = torch.zeros(max(n, 1), dtype=torch.uint8, device=device)
            make = lambda shape, dt, off: flat[off:off + math.prod(shape) * torch.empty(0, dtype=dt).element_size()].view(dt).view(shape)
        made = {k: {} for k in ("latent", "state", "k", "v", "conv", "shift")}
        for key, kind, shape, dt, off in views:
            made[kind][key] = make(shape, dt, off)
        self.latent, self.state, self.conv, self.shift = (made[k] for k in ("latent", "state", "conv", "shift"))
        self.kv = {key: (made["k"][key], made["v"][key]) for key in made["k"]}
        for key, s in cfg.mixers():
            if s.kv_from >= 0:
                self.kv[key] = self.kv[s.kv_from]
        self.paged = [p for k in ("latent", "k", "v") for p in made[k].values()]
        self.slotted = [p for k in ("state", "conv", "shift") for p in made[k].values()]

    def copy_sequence(self, src_blocks: Sequence[int], dst_blocks: Sequence[int], src_slot: int, dst_slot: int):
        """Pages ``src -> dst`` pairwise and the whole state slot."""
        for pool in self.paged:
            v = pool.view(-1, self.block_size, *pool.shape[1:])
            for a, b in zip(src_blocks, dst_blocks):
                v[b] = v[a]
        for st in self.slotted:
            st[dst_slot] = st[src_slot]


@dataclass
class SegmentBatch:
    """Device description of a batch of segments; the first ``long_segs`` of them (``long_rows`` rows) are long portions, those
    from ``multi_segs`` (row ``multi_rows``) on have a single row.
    ``cu`` is None when every segment is a single row.  ``short_*`` describe the segments behind the long ones, with row
    numbers counted from ``long_rows``; ``items[heads]`` are their column groups of up to ``item_width[heads]`` (64)
    columns (see :func:`attention_items`)."""
    tokens: torch.Tensor
    slots: torch.Tensor                      # [T] row of the latent pools that each token's row goes to
    ctx: torch.Tensor                        # [S] int32: tokens of the sequence including this segment
    block_tables: torch.Tensor               # [S, max blocks] int32
    state_slot: torch.Tensor                 # [S] int32
    cu: Optional[torch.Tensor] = None        # [S + 1] int32
    long_segs: int = 0
    long_rows: int = 0
    long_first: Optional[torch.Tensor] = None   # [long] int32 first row of a long segment's context among ``ctx_slots``
    long_blocks: Optional[torch.Tensor] = None  # [n, 4] int32 query tiles of the long segments (see :func:`query_blocks`)
    ctx_slots: Optional[torch.Tensor] = None  # pool rows of the long segments' whole contexts
    short_cu: Optional[torch.Tensor] = None
    row_seg: Optional[torch.Tensor] = None   # [short rows] int32: segment (among the short ones) and last visible position
    row_pos: Optional[torch.Tensor] = None
    max_ctx: int = 0                         # host upper bound of the short segments' contexts
    items: Optional[dict] = None
    item_width: Optional[dict] = None
    spans: Optional[tuple] = None            # row ranges of recurrent spans and the first span of every segment
    # attention layers (and positions for all that rotate)
    multi_segs: int = 0
    multi_rows: int = 0
    max_ctx_one: int = 0                     # host upper bound of the single-row segments' contexts
    pos: Optional[torch.Tensor] = None       # [T] int32 position of every row; None: ctx - 1
    seg_of: Optional[torch.Tensor] = None    # [T] int32 segment of every row
    blocks: Optional[dict] = None            # tokens per query tile -> [n, 4] int32 (see :func:`query_blocks`)


def attention_items(lens: Sequence[int], ctx: Sequence[int], heads: int, width: int = 64) -> list:
    """Cut the (row, head) columns of consecutive segments into groups of at most ``width`` that never span two segments:
    ``[segment, first column, columns, base]``; the column ``c`` belongs to row ``c // heads`` and sees the first
    ``base + c // heads`` positions."""
    out, row0 = [], 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        step = width // heads * heads if heads <= width else width     # whole rows per group when a row fits
        for c in range(row0 * heads, (row0 + n) * heads, step):
            out.append([s, c, min(step, (row0 + n) * heads - c), L - n - row0 + 1])
        row0 += n
    return out


def query_blocks(lens: Sequence[int], ctx: Sequence[int], tokens: int) -> list:
    """Cut segments into query tiles of at most ``tokens`` rows: ``[segment, first row, rows, position of the first row]``, those
    that see the most positions first (the last tiles to start are then the short ones)."""
    out, row = [], 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        out += [[s, row + a, min(tokens, n - a), L - n + a] for a in range(0, n, tokens)]
        row += n
    return sorted(out, key=lambda b: -(b[2] + b[3]))


QUERY_ROWS = 128       # (token, head) rows of a query tile


def tile_tokens(spec) -> int:
    """Tokens of one query tile of an attention layer: the heads of a key / value head's group lie side by side."""
    return max(1, QUERY_ROWS // (spec.heads // spec.kv_heads))


def recurrent_spans(lens: Sequence[int], heads: int, ctas: int = 296, shortest: int = 128) -> Optional[tuple]:
    """Cut long segments into spans so that (spans x heads) fills the machine (``ctas`` at a time); spans are multiples of
    the kernel's 16-token chunks.  ``(row ranges, first span of every segment)``, None when no segment is worth cutting:
    a CTA alone takes 1.25 times the time per chunk that a full machine needs for one chunk per SM, and spans add 0.57 for the
    pass over their states (measured on a B200)."""
    chunks = [-(-n // 16) for n in lens]
    full = sum(chunks) * heads / 148
    if max(1.25 * max(chunks), full) <= 1.57 * full:
        return None
    size = max(shortest, pad_to(-(-sum(lens) * heads // ctas), 16))
    spans, first, row = [], [0], 0
    for n in lens:
        k = max(1, round(n / size))
        step = pad_to(-(-n // k), 16)
        spans += [[row + a, row + min(n, a + step)] for a in range(0, n, step)]
        first.append(len(spans))
        row += n
    return (spans, first) if len(spans) > len(lens) else None


class ComposedForward:
    """The forward of composed stacks (mixed into :class:`relax_b200.rollout.weights.RolloutWeights`).

    The residual stream is fp32.  A sublayer reads its copy in the model's type, and one kernel norms the sublayer's
    output, adds it and writes the next copy (or adds first and norms the sum); at the last sublayer that kernel also applies the
    final norm.  With norms in front of the sublayers, one kernel adds the outputs of both and of the second embedding and writes
    the norms that the next layer reads."""

    @staticmethod
    def latent_dims(s) -> tuple:
        """Padded ``(dim, vdim, rank)`` of a latent layer (16-byte rows per head, 64-column latent chunks); ``dim`` counts the
        unrotated and the rotated features of a head."""
        return pad_to(s.dim + s.rot_dims, 8), pad_to(s.vdim, 8), pad_to(s.kv_rank, 64)

    @staticmethod
    def gate_column(s) -> int:
        """First column of an attention layer's output gate behind its projections (16-byte aligned)."""
        return pad_to(projected(s), 8)

    @staticmethod
    def gla_columns(s) -> dict:
        """First columns of queries, keys, values, output gates and the decay's inner projection, and the number of columns."""
        qd, vd = s.heads * s.dim, s.heads * s.vdim
        g = pad_to(2 * qd + vd, 8)
        a1 = pad_to(g + vd, 8)
        return {"q": 0, "k": qd, "v": 2 * qd, "g": g, "a1": a1, "end": a1 + pad_to(s.decay_rank, 8)}

    @staticmethod
    def attention_dims(s) -> tuple:
        """Pitch of a head's queries and keys, of its values, and of its output in an attention layer."""
        return head_pitch(s.dim), head_pitch(s.vdim), pad_to(s.vdim, 8)

    def rope_frequencies(self, spec) -> torch.Tensor:
        """``rot_base ** (-2 i / rot_dims)`` in fp64, kept on the device; with ``rot_scaling`` frequencies whose wavelength exceeds
        ``original / low`` are divided by ``factor``, and those down to ``original / high`` partly."""
        made = self.__dict__.setdefault("_rope_freq", {})
        key = (spec.rot_base, spec.rot_dims, spec.rot_scaling)
        if key not in made:
            i = torch.arange(spec.rot_dims // 2, dtype=torch.float64)
            f = float(spec.rot_base) ** (-2.0 * i / spec.rot_dims)
            if spec.rot_scaling is not None:
                factor, low, high, original = spec.rot_scaling
                kept = ((original * f / (2 * math.pi) - low) / (high - low)).clamp(0.0, 1.0)      # share that stays as it is
                f = (1 - kept) * f / factor + kept * f
            made[key] = f.to(self.device)
        return made[key]

    INPUT = {"hgrn2": "rec_qfv", "attention": "attn_qkv", "latent_attention": "lat_qcg", "mingru": "gru_zxg", "gla": "gla_in"}

    @staticmethod
    def mixer_param_shapes(s, p: str, Wp: int) -> dict:
        shapes, H = {}, s.heads
        if s.mixer == "hgrn2":
            qd, vd = H * s.dim, H * s.vdim
            shapes[p + "rec_qfv"] = (pad_to(2 * qd + vd, 64), Wp)
            shapes[p + "rec_f_bias"], shapes[p + "rec_lower"], shapes[p + "rec_norm"] = (qd,), (qd,), (s.vdim,)
            shapes[p + "rec_o"] = (Wp, pad_to(vd, 8))
        elif s.mixer == "mingru":
            n = pad_to(s.vdim, 8)
            shapes[p + "gru_zxg"], shapes[p + "gru_o"] = (pad_to(3 * n, 64), Wp), (Wp, n)
            shapes[p + "gru_z_b"], shapes[p + "gru_x_b"] = (n,), (n,)
        elif s.mixer == "gla":
            qd, vd = H * s.dim, H * s.vdim
            shapes[p + "gla_in"] = (pad_to(ComposedForward.gla_columns(s)["end"], 64), Wp)
            shapes[p + "gla_a2"], shapes[p + "gla_a2_b"] = (pad_to(qd, 64), pad_to(s.decay_rank, 8)), (qd,)
            shapes[p + "gla_norm"], shapes[p + "gla_o"] = (s.vdim,), (Wp, pad_to(vd, 8))
        elif s.mixer == "attention":
            cols = ComposedForward.gate_column(s) + H * pad_to(s.vdim, 8) if s.out_gate else projected(s)
            shapes[p + "attn_qkv"] = (pad_to(cols, 64), Wp)
            if s.qkv_bias:
                shapes[p + "attn_qkv_b"] = (projected(s),)
            if s.conv:
                shapes[p + "attn_conv"] = (projected(s), s.conv)
            if s.proj_norm or s.head_norm:
                shapes[p + "attn_q_norm"] = (H * s.dim if s.proj_norm else s.dim,)
                if s.own_kv:
                    shapes[p + "attn_k_norm"] = (s.kv_heads * s.dim if s.proj_norm else s.dim,)
            if s.sink or s.unit_sink:      # (a unit sink's logits stay zero)
                shapes[p + "attn_sink"] = (H,)
            if s.talk:
                shapes[p + "attn_talk"] = (H, H)
            shapes[p + "attn_o"] = (Wp, H * pad_to(s.vdim, 8))
        else:
            # rows of lat_qcg: queries (a head's unrotated, then its rotated features), latent, rotated key part, gates.  lat_uk maps
            # a cached row to a head's key; its rows of rotated features are those of the identity (:meth:`pass_rotated_keys`)
            dp, vp, Rp = pad_to(s.dim + s.rot_dims, 8), pad_to(s.vdim, 8), pad_to(s.kv_rank, 64)
            shapes[p + "lat_qcg"] = (pad_to(H * dp + Rp + pad_to(s.rot_dims, 8) + (H * vp if s.out_gate else H), 64), Wp)
            shapes[p + "lat_norm"] = (Rp,)
            shapes[p + "lat_uk"], shapes[p + "lat_uv"] = (H * dp, latent_row(s)), (H * vp, Rp)
            shapes[p + "lat_o"] = (Wp, H * vp)
        return shapes

    @staticmethod
    def composed_param_shapes(cfg: ModelConfig) -> dict:
        """Every projection's output features are padded to 64 and its input features to the pitch of the rows it reads;
        padding is zero and stays zero through every layer."""
        Wp, Vp = pad_to(cfg.hidden_size, 64), pad_to(cfg.vocab_size, 64)
        shapes = {"embed": (Vp, Wp)}
        if cfg.side_dim:
            shapes["side_embed"] = (Vp, pad_to(cfg.num_layers * cfg.side_dim, 8))
        for i, s in enumerate(cfg.layer_specs):
            p = f"layers.{i}."
            if s.pair is None:
                shapes.update(ComposedForward.mixer_param_shapes(s, p, Wp))
            else:      # the input projections of both lie one behind the other (:meth:`pair_views`)
                rows = 0
                for k, m in enumerate(s.pair):
                    own = ComposedForward.mixer_param_shapes(m, f"{p}{k}.", Wp)
                    rows += own.pop(f"{p}{k}.{ComposedForward.INPUT[m.mixer]}")[0]
                    shapes.update({**own, f"{p}{k}.out_norm": (Wp,)})
                shapes[p + "pair_in"] = (rows, Wp)
            if cfg.pre_norm:
                norms = ["norm1"] + (["norm2"] if s.has_ff else []) + (["shift"] if cfg.token_shift else [])
            else:
                norms = ["post_attn_norm"] + (["post_mlp_norm"] if s.has_ff else [])
            for norm in norms:
                shapes[p + norm] = (Wp,)
                if cfg.norm_sum:
                    shapes[p + norm + "_b"] = (Wp,)
            if cfg.side_dim:
                shapes[p + "side_gate"], shapes[p + "side_proj"] = (pad_to(cfg.side_dim, 64), Wp), (Wp, pad_to(cfg.side_dim, 8))
                shapes[p + "side_norm"] = (Wp,)
            if s.ff:
                Fp = pad_to(s.ff, 64)
                shapes[p + "gate_up"], shapes[p + "down"] = (2 * Fp, Wp), (Wp, Fp)
            if s.moe is not None:
                E, Fp, Fs = s.moe.experts, pad_to(s.moe.ff, 64), pad_to(s.moe.shared_ff, 64)
                shapes[p + "moe_router"] = (pad_to(s.moe.outputs, 64), Wp)
                if s.moe.correction:
                    shapes[p + "moe_correction"] = (s.moe.outputs,)
                shapes[p + "moe_up"], shapes[p + "moe_down"] = (E, 2 * Fp if s.moe.gated else Fp, Wp), (E, Wp, Fp)
                if Fs:
                    shapes[p + "shared_up"], shapes[p + "shared_down"] = (Fs, Wp), (Wp, Fs)
        shapes["final_norm"] = (Wp,)
        if cfg.norm_sum:
            shapes["final_norm_b"] = (Wp,)
        if cfg.embed_norm:
            shapes["embed_norm"] = (Wp,)
        if not cfg.tie_word_embeddings:
            shapes["lm_head"] = (Vp, Wp)
        return shapes

    @staticmethod
    def pair_views(cfg: ModelConfig, params: dict) -> dict:
        """The input projections of a pair's mixers as parameters of their own."""
        out = {}
        for i, s in enumerate(cfg.layer_specs):
            at = 0
            for k, m in enumerate(s.pair or ()):
                name, w = f"layers.{i}.{k}.{ComposedForward.INPUT[m.mixer]}", params[f"layers.{i}.pair_in"]
                n = ComposedForward.mixer_param_shapes(m, f"layers.{i}.{k}.", w.shape[1])[name][0]
                out[name] = w[at:at + n]
                at += n
        return out

    def pass_rotated_keys(self, i: int) -> None:
        """Let the key map of latent layer ``i`` hand the rotated part of a cached row on to every head's key unchanged (a reader calls
        this after it has filled the map's other rows)."""
        s = self.cfg.layer_specs[i]
        uk = self.p[f"layers.{i}.lat_uk"].view(s.heads, -1, latent_row(s))
        k = torch.arange(s.rot_dims, device=uk.device)
        uk[:, s.dim + k, pad_to(s.kv_rank, 64) + k] = 1.0

    # ------------------------------------------------------------------ mixers
    # every mixer: (cache key, spec, prefix of its parameters, rows of its input projection, batch, cache, angle tables) -> output rows
    def _hgrn2(self, key, s, pre, qfv, b: SegmentBatch, cache: StackCache, tables: dict):
        p = self.p
        o = ops.hgrn2(qfv, p[pre + "rec_f_bias"], p[pre + "rec_lower"], p[pre + "rec_norm"], cache.state[key], b.state_slot,
                      b.ctx, b.cu, s.heads, s.dim, s.vdim, self.cfg.rms_norm_eps, b.spans)
        return ops.linear(o, p[pre + "rec_o"])

    def _mingru(self, key, s, pre, zxg, b: SegmentBatch, cache: StackCache, tables: dict):
        p = self.p
        return ops.linear(ops.mingru(zxg, p[pre + "gru_z_b"], p[pre + "gru_x_b"], cache.state[key], b, s.vdim), p[pre + "gru_o"])

    def _gla(self, key, s, pre, rows, b: SegmentBatch, cache: StackCache, tables: dict):
        p, at = self.p, self.gla_columns(s)
        z = ops.linear_fp32(rows[:, at["a1"]:at["end"]], p[pre + "gla_a2"])
        o = ops.gla(rows, z, p[pre + "gla_a2_b"], p[pre + "gla_norm"], cache.state[key], b.state_slot, b.ctx, b.cu, s.heads, s.dim, s.vdim, at["g"],
                    self.cfg.rms_norm_eps, s.decay_root, b.spans)
        return ops.linear(o, p[pre + "gla_o"])

    def _latent(self, key, s, pre, qcg, b: SegmentBatch, cache: StackCache, tables: dict):
        """Keys and values are products of the cached latent row ``c``: ``q . (W_uk c) = (W_uk^T q) . c`` and
        ``sum p (W_uv c) = W_uv (sum p c)``.  Single tokens and short portions therefore attend to the latent rows in
        place, with the up-projections folded around the attention; long portions project keys and values of their whole
        context once and run the flash kernel on them.  A rotated key part in the row passes both ways unchanged
        (:meth:`pass_rotated_keys`)."""
        p = self.p
        H, (dp, vp, Rp), row, pool = s.heads, self.latent_dims(s), latent_row(s), cache.latent[key]
        T, rp = qcg.shape[0], pad_to(s.rot_dims, 8)
        q, c, k_rot, gate = qcg[:, : H * dp + Rp + rp + H * (vp if s.out_gate else 1)].split([H * dp, Rp, rp, H * (vp if s.out_gate else 1)], 1)
        q = q.view(T, H, dp)
        turned = (q, k_rot, self._rope_table(s, b, tables), Rp, s.rot_dims, s.dim) if s.rot_dims else None
        ops.latent_write(c, p[pre + "lat_norm"], s.kv_rank, self.cfg.rms_norm_eps, pool, b.slots, turned)
        uk, uv = p[pre + "lat_uk"], p[pre + "lat_uv"]
        n = b.long_rows
        parts = []
        if n:
            c = pool[b.ctx_slots]
            k, v = ops.linear(c, uk).view(-1, H, dp), ops.linear(c[:, :Rp], uv).view(-1, H, vp)
            parts.append(ops.dense_flash(q[:n], k, v, b.long_first, b.long_blocks, s.scale, gate[:n], s.out_gate))
        if n < T:
            ql = ops.head_linear(q[n:], uk.view(H, dp, row), False)
            o = ops.latent_attention(ql, pool, b, cache.block_size, s.scale, None if s.out_gate else gate[n:], Rp)
            parts.append(ops.head_linear(o, uv.view(H, vp, Rp), True, gate[n:] if s.out_gate else None).reshape(T - n, H * vp))
        return ops.linear(parts[0] if len(parts) == 1 else torch.cat(parts), p[pre + "lat_o"])

    def _attention(self, key, s, pre, qkv, b: SegmentBatch, cache: StackCache, tables: dict):
        p = self.p
        dp, _, vo = self.attention_dims(s)
        k_pool, v_pool = cache.kv[key]
        table, eps, pools = self._rope_table(s, b, tables), self.cfg.rms_norm_eps, (k_pool, v_pool) if s.own_kv else (None, None)
        if s.conv or s.qkv_bias or s.head_norm:
            q = ops.conv_inputs(qkv, p.get(pre + "attn_qkv_b"), p.get(pre + "attn_conv"), cache.conv.get(key), b, p.get(pre + "attn_q_norm"),
                                p.get(pre + "attn_k_norm"), table, s.heads, s.kv_heads, s.dim, s.vdim, dp, s.rot_dims, eps if s.head_norm else 0.0, *pools)
        elif s.proj_norm or s.rot_halves:
            q = ops.projection_inputs(qkv, p.get(pre + "attn_q_norm"), p.get(pre + "attn_k_norm"), table, s.heads, s.kv_heads, s.dim, s.vdim, dp, s.rot_dims,
                                      s.rot_halves, eps if s.proj_norm else 0.0, *pools, b.slots)
        else:
            q = ops.attention_inputs(qkv, table, s.heads, s.kv_heads, s.dim, s.vdim, dp, s.rot_dims, eps if s.qk_norm else 0.0, *pools, b.slots)
        g = self.gate_column(s)
        o = ops.paged_attention(q, k_pool, v_pool, b, cache.block_size, s.scale, p.get(pre + "attn_sink"), vo, s.window,
                                qkv[:, g:g + s.heads * vo] if s.out_gate else None, s.keep_first, s.chunk, s.softcap, p.get(pre + "attn_talk"))
        return ops.linear(o, p[pre + "attn_o"])

    def _mix(self, i, h, b: SegmentBatch, cache: StackCache, tables: dict) -> list:
        """Outputs of layer ``i``'s mixer, or of the two of a pair, on rows ``h``."""
        s, pre = self.cfg.layer_specs[i], f"layers.{i}."
        run = lambda key, m, at, x: getattr(self, "_latent" if m.mixer == "latent_attention" else "_" + m.mixer)(key, m, at, x, b, cache, tables)
        if s.pair is None:
            return [run(i, s, pre, ops.linear(h, self.p[pre + self.INPUT[s.mixer]]))]
        rows, at, out = ops.linear(h, self.p[pre + "pair_in"]), 0, []
        for k, m in enumerate(s.pair):
            n = self.p[f"{pre}{k}.{self.INPUT[m.mixer]}"].shape[0]
            out.append(run((i, k), m, f"{pre}{k}.", rows[:, at:at + n]))
            at += n
        return out

    def _rope_table(self, s, b: SegmentBatch, tables: dict):
        if not s.rot_dims:
            return None
        key = (s.rot_base, s.rot_dims, s.rot_scaling)
        if key not in tables:
            tables[key] = ops.rope_table(b.ctx if b.pos is None else b.pos, -1 if b.pos is None else 0, self.rope_frequencies(s))
        return tables[key]

    # ------------------------------------------------------------------ feed-forwards
    def _feed_forward(self, i, h, count):
        """``(output rows or None, (expert rows, plan) or None)`` of layer ``i``'s feed-forward; ``count``: the router's counters."""
        s, p, pre = self.cfg.layer_specs[i], self.p, f"layers.{i}."
        if s.moe is None:
            return ops.linear(ops.linear_glu(h, p[pre + "gate_up"], s.act), p[pre + "down"]), None
        plan = ops.moe_route(ops.linear_fp32(h, p[pre + "moe_router"]), s.moe, h.dtype, count, p.get(pre + "moe_correction"))
        rows = ops.moe_experts(h, plan, p[pre + "moe_up"], p[pre + "moe_down"], s.moe.act, s.moe.limit)
        shared = ops.linear(ops.linear_act(h, p[pre + "shared_up"], s.moe.act), p[pre + "shared_down"]) if s.moe.shared_ff else None
        return shared, (rows, plan)

    # ------------------------------------------------------------------ trunk
    def _route_counts(self, device) -> dict:
        """Counters of every routed layer's :func:`ops.moe_route`, zeroed at once."""
        specs = self.cfg.layer_specs
        routed = [i for i, s in enumerate(specs) if s.moe is not None]
        return dict(zip(routed, ops.route_counters(len(routed), max(specs[i].moe.experts for i in routed), device))) if routed else {}

    def _run_composed(self, b: SegmentBatch, cache: StackCache, taps: Optional[list] = None):
        """Final-norm output of every row.  ``taps``: a list that receives the fp32 residual stream after every layer."""
        cfg, p = self.cfg, self.p
        W, G, eps = cfg.hidden_size, cfg.norm_groups, cfg.rms_norm_eps
        if cfg.pre_norm:
            return self._run_pre_norm(b, cache, taps)
        res, h = ops.embed_rows(b.tokens, p["embed"], p.get("embed_norm"), W, G, eps, cfg.embed_scale)

        def join(y, norm, last, experts=None):
            """The sublayer's output meets the stream; returns the next sublayer's input."""
            if not cfg.norm_sum:
                return ops.norm_add(res, y, p[norm], W, G, eps, p["final_norm"] if last else None, experts)
            nxt = (p["final_norm"], p["final_norm_b"]) if last else None
            return ops.sum_norm(res, y, p[norm], p[norm + "_b"], W, cfg.sum_alpha, eps, nxt, cfg.logit_scale if last else 1.0, experts)

        tables: dict = {}
        counts = self._route_counts(res.device)
        for i, s in enumerate(cfg.layer_specs):
            pre = f"layers.{i}."
            final = i + 1 == cfg.num_layers
            h = join(self._mix(i, h, b, cache, tables)[0], pre + "post_attn_norm", final and not s.has_ff)
            if s.has_ff:
                m, experts = self._feed_forward(i, h, counts.get(i))
                h = join(m, pre + "post_mlp_norm", final, experts)
            if taps is not None:
                taps.append(res[:, :W].clone())
        return h

    def _run_pre_norm(self, b: SegmentBatch, cache: StackCache, taps: Optional[list] = None):
        """The same for sublayers that read norms of the stream: ``x <- x + mixer(norm1 x) + ff(norm2 x)``, then the second
        embedding's part."""
        cfg, p = self.cfg, self.p
        W, eps = cfg.hidden_size, cfg.rms_norm_eps

        def reads(i):
            """``(norms of the stream that layer i reads, what shifts the first of them)``; behind the last layer: the final norm."""
            if i == cfg.num_layers:
                return (p["final_norm"],), None
            pre = f"layers.{i}."
            norms = (p[pre + "norm1"],) + ((p[pre + "norm2"],) if cfg.layer_specs[i].has_ff else ())
            return norms, (p[pre + "shift"], cache.shift[i], b) if cfg.token_shift else None

        tables: dict = {}
        counts = self._route_counts(b.tokens.device)
        res, _ = ops.embed_rows(b.tokens, p["embed"])
        h = ops.stream_step(res, W, eps, norms=reads(0)[0], shift=reads(0)[1])
        for i, s in enumerate(cfg.layer_specs):
            pre = f"layers.{i}."
            y = self._mix(i, h[0], b, cache, tables)
            pair = (p[pre + "0.out_norm"], p[pre + "1.out_norm"]) if s.pair is not None else None
            experts = self._feed_forward(i, h[1], counts.get(i))[1] if s.has_ff else None
            norms, shift = reads(i + 1)
            if cfg.side_dim:
                x, = ops.stream_step(res, W, eps, y, pair, experts)
                g = ops.side_gate(ops.linear(x, p[pre + "side_gate"]), p["side_embed"], b.tokens, i * cfg.side_dim, cfg.side_dim)
                h = ops.stream_step(res, W, eps, [ops.linear(g, p[pre + "side_proj"])], (p[pre + "side_norm"],), norms=norms, shift=shift)
            else:
                h = ops.stream_step(res, W, eps, y, pair, experts, norms, shift)
            if taps is not None:
                taps.append(res[:, :W].clone())
        return h[0]

    def forward_segments(self, b: SegmentBatch, cache: StackCache, rows: Optional[torch.Tensor], tp, taps: Optional[list] = None):
        """Logits of the given rows (None: no row is asked for, only slots and pages are advanced)."""
        h = self._run_composed(b, cache, taps)
        return None if rows is None else self._logits(h[rows], tp)

    def forward_step(self, tokens, block_tables, context_lens, slots, state_slot, cache: StackCache, tp):
        """One decoded token per sequence (the captured step): everything is read from device arrays."""
        b = SegmentBatch(tokens, slots, context_lens, block_tables, state_slot,
                         max_ctx=block_tables.shape[1] * cache.block_size, max_ctx_one=block_tables.shape[1] * cache.block_size)
        return self._logits(self._run_composed(b, cache), tp)


class ComposedScheduler:
    """Scheduling of composed stacks (mixed into :class:`relax_b200.rollout.engine.RolloutEngine`).

    Every running request has ``fed`` tokens in its pages and state slot.  A step feeds the newest token of the requests
    that decode and, within ``max_prefill_tokens``, the next portions of the prompts, all in one batch; a request whose
    last known token has been fed is sampled.  When only decoding is left the engine's windowed loop takes over."""

    def _release_request(self, r):
        self.bm.release(r.blocks)
        r.blocks = []
        if r.state_slot is not None:
            self.sm.release(r.state_slot)
            r.state_slot = None

    # ------------------------------------------------------------------ the step function
    def run_segments(self, parts: Sequence[tuple], want: Sequence[Sequence[int]], taps: Optional[list] = None):
        """One batch: ``parts[j] = (request, n)`` feeds the request's tokens ``fed .. fed + n``; ``want[j]`` are the places
        among them whose logits are returned, ``[sum(len(w)), vocab]`` in the order of ``parts`` (None when nothing is
        wanted).  Pages are taken as needed."""
        if not parts or any(n < 1 for _, n in parts):
            raise ValueError("a batch is made of segments of at least one token")
        bs = self.block_size
        for r, n in parts:
            if r.state_slot is None:
                r.state_slot = self.sm.alloc()
            need = self.bm.blocks_for(r.fed + n)
            while len(r.blocks) < need:
                r.blocks.append(self.bm.alloc())
                r._reserve = max(0, getattr(r, "_reserve", 0) - 1)
        long_ok = self._long_portions
        kind = lambda n: 0 if long_ok and n >= LONG_PORTION else (1 if n > 1 else 2)      # long portions, short ones, single rows
        order = sorted(range(len(parts)), key=lambda j: kind(parts[j][1]))                # (stable)
        n_long = sum(1 for r, n in parts if kind(n) == 0)
        n_multi = sum(1 for r, n in parts if n > 1)
        toks, slots, cu, ctx, sslot, bt, rows_of = [], [], [0], [], [], [], {}
        for j in order:
            r, n = parts[j]
            seq = r.prompt + r.output
            toks += seq[r.fed:r.fed + n]
            slots += self._slots(r, r.fed, r.fed + n)
            rows_of[j] = cu[-1]
            cu.append(cu[-1] + n)
            ctx.append(r.fed + n)
            sslot.append(r.state_slot)
        maxb = pad_to(max(len(parts[j][0].blocks) for j in order), 8)
        bt = [parts[j][0].blocks + [0] * (maxb - len(parts[j][0].blocks)) for j in order]
        rows = [rows_of[j] + w for j in range(len(parts)) for w in want[j]]
        single = all(n == 1 for _, n in parts)
        i32, i64 = torch.int32, torch.int64
        arrays = {"tokens": (toks, i64), "slots": (slots, i64), "ctx": (ctx, i32), "block_tables": (bt, i32), "state_slot": (sslot, i32)}
        host = {"long_segs": n_long, "long_rows": cu[n_long], "max_ctx": max(ctx[n_long:], default=0),
                "multi_segs": n_multi, "multi_rows": cu[n_multi], "max_ctx_one": max(ctx[n_multi:], default=0)}
        widths, tiles = {}, []
        if not single:
            arrays["cu"] = (cu, i32)
            lens = [b - a for a, b in zip(cu, cu[1:])]
            sl, sc = lens[n_long:], ctx[n_long:]
            attn = self.cfg.specs_with("attention")
            if attn or self.cfg.token_shift or any(s.rot_dims for _, s in self.cfg.mixers()):
                arrays["pos"] = ([c - n + k for n, c in zip(lens, ctx) for k in range(n)], i32)
            if attn or self.cfg.token_shift:
                arrays["seg_of"] = ([s for s, n in enumerate(lens) for _ in range(n)], i32)
            if attn:
                tiles = sorted({tile_tokens(s) for s in attn})
                for t in tiles:
                    arrays[f"blocks{t}"] = (query_blocks(lens[:n_multi], ctx, t), i32)
            if n_long:
                arrays["long_first"] = ([sum(ctx[:s]) for s in range(n_long)], i32)
                arrays["long_blocks"] = (query_blocks(lens[:n_long], ctx, QUERY_ROWS), i32)
                arrays["ctx_slots"] = ([x for j in order[:n_long] for x in self._slots(parts[j][0], 0, parts[j][0].fed + parts[j][1])], i64)
            rec = [s.heads for s in self.cfg.specs_with("hgrn2", "gla")]
            cuts = recurrent_spans(lens, max(rec)) if rec and self.device.type == "cuda" else None
            if cuts is not None:
                arrays["spans"], arrays["span_first"] = (cuts[0], i32), (cuts[1], i32)
            specs = self.cfg.specs_with("latent_attention")
            if sl and specs:
                arrays["short_cu"] = ([c - cu[n_long] for c in cu[n_long:]], i32)
                arrays["row_seg"] = ([s for s, n in enumerate(sl) for _ in range(n)], i32)
                arrays["row_pos"] = ([c - n + k for n, c in zip(sl, sc) for k in range(n)], i32)
                for s in specs:
                    widths[s.heads] = min(widths.get(s.heads, 64), ops.latent_columns(latent_row(s), pad_to(s.kv_rank, 64)))
                for H, width in widths.items():
                    arrays[f"items{H}"] = (attention_items(sl, sc, H, width), i32)
        if rows:
            arrays["rows"] = (rows, i64)
        dev = dict(zip(arrays, self._stage(list(arrays.values()))))
        want_t = dev.pop("rows", None)
        spans = (dev.pop("spans"), dev.pop("span_first")) if "spans" in dev else None
        items = {H: dev.pop(f"items{H}") for H in widths}
        blocks = {t: dev.pop(f"blocks{t}") for t in tiles}
        batch = SegmentBatch(**dev, **host, items=items or None, item_width=widths or None, spans=spans, blocks=blocks or None)
        logits = self.weights.forward_segments(batch, self.kv, want_t, self.tp, taps)
        for r, n in parts:
            r.fed += n
        return logits

    # ------------------------------------------------------------------ sequences driven from outside (trace replay)
    def open_sequence(self):
        """A sequence whose tokens are given step by step (:meth:`feed`) instead of being sampled."""
        from .engine import Request, SamplingParams

        r = Request(self._next_rid, [], SamplingParams())
        self._next_rid += 1
        r.status = "running"
        return r

    @torch.no_grad()
    def feed(self, entries: Sequence[tuple]):
        """``entries[j] = (sequence, its next tokens, wanted places)``; returns the wanted rows of logits (or None)."""
        for r, tokens, _ in entries:
            bad = [t for t in tokens if not 0 <= t < self.cfg.vocab_size]
            if bad:
                raise ValueError(f"token {bad[0]} is outside the vocabulary of {self.cfg.vocab_size}")
            r.prompt.extend(tokens)
        z = self.run_segments([(r, len(t)) for r, t, _ in entries], [w for _, _, w in entries])
        return None if z is None else z[:, : self.cfg.vocab_size]

    def close_sequence(self, r):
        self._release_request(r)
        r.status = "finished"

    # ------------------------------------------------------------------ generation
    def _step_composed(self):
        for r in self._admit():
            r.state_slot = self.sm.alloc()
            self.running.append(r)
        live = [r for r in self.running if r._lead is None or r.fed > 0]      # followers wait for their leader's prompt
        if not live:
            return
        if all(r.num_tokens - r.fed == 1 and r.output for r in self.running):
            if self.windowed_decode and self._decode_window():
                for r in self.running:
                    if r.status == "running":
                        r.fed = r.num_tokens - 1
                return
        budget = self.max_prefill_tokens
        parts = []
        for r in live:      # decoding requests first, then prompt portions in order of arrival
            if r.num_tokens - r.fed == 1:
                parts.append((r, 1))
                budget -= 1
        budget = max(budget, self.block_size)      # prompts advance however many requests decode
        for r in live:
            left = r.num_tokens - r.fed
            if left > 1 and budget > 0:
                n = min(left, budget)
                parts.append((r, n))
                budget -= n
        done = [(r, n) for r, n in parts if r.fed + n == r.num_tokens]
        want = [[n - 1] if r.fed + n == r.num_tokens else [] for r, n in parts]
        first = {id(r) for r, _ in done if not r.output}
        logits = self.run_segments(parts, want)
        self.stats["prefill_tokens"] += sum(n for r, n in parts if not (r.output and n == 1))
        self.stats["decode_tokens"] += sum(1 for r, n in parts if r.output and n == 1)
        if not done:
            return
        reqs, pick = [r for r, _ in done], list(range(len(done)))
        for k, (r, _) in enumerate(done):
            for f in [f for f in self.running if f._lead is r and f.fed == 0]:
                # same prompt: same latent rows (full pages are shared already) and same states; sampled from the same row
                shared = f.cached_tokens // self.block_size
                self.kv.copy_sequence(r.blocks[shared:len(f.blocks)], f.blocks[shared:], r.state_slot, f.state_slot)
                f.fed = r.fed
                self.stats["cached_tokens"] += len(f.prompt)
                first.add(id(f))
                reqs.append(f)
                pick.append(k)
        if len(pick) > len(done):
            logits = logits[torch.tensor(pick, device=self.device)]
        import time

        now = time.perf_counter()
        for r in reqs:
            if id(r) in first:
                r.t_first = now
        self._sample_and_append(reqs, logits)
