"""Zoguzen: reader of the design's ``config.json`` and of its tensors.

A Zoguzen model is a composed stack (:class:`relax_b200.models.config.LayerSpec`) whose sublayers read layer norms of the stream and
join it together.  Mixers read shifted tokens and are of three kinds: attention inside chunks (projections with biases and short
convolutions, norms head by head, capped scores, a unit sink, mixed heads, keys and values of a layer's own or of an earlier one);
a gated running mean (minGRU); and a pair of sliding-window attention (kept first tokens, stretched rotation, gated outputs) and
linear attention with decaying rows.  Feed-forwards are routed over gated experts; a second embedding joins after every layer; the
embedding table gives the logits, which are capped.  This module only translates names and layouts; the layers are computed by
:mod:`relax_b200.rollout.composed`.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import glu_rows
from .config import LayerSpec, ModelConfig, MoESpec, composed_config
from .native import check_tensors, pad_to, put, save_folder

ARCHITECTURE = "Zoguzen"


def _feed_forward(i: int, mlp) -> dict:
    if mlp is None:
        return {}
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    r = mlp["router"]
    return {"moe": MoESpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), act="swiglu", score="softmax", renormalize=True)}


def _attention(m: dict) -> dict:
    return dict(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), conv=int(m.get("conv") or 0))


def _left(m: dict) -> LayerSpec:
    rot, mask = m.get("rot") or {"dims": 0, "base": 0.0}, m.get("mask") or {"size": 0}
    sc = rot.get("scaling")
    return LayerSpec("attention", rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), window=int(mask["size"]), keep_first=int(mask.get("keep_first") or 0),
                     rot_scaling=None if sc is None else tuple(float(sc[k]) for k in ("factor", "low", "high", "original")), out_gate=True, **_attention(m))


def _right(i: int, m: dict, shapes: Optional[dict]) -> LayerSpec:
    a1 = f"l{i}.mix.right.a1"
    if shapes is None or a1 not in shapes:
        raise ValueError(f"layer {i}: the rank of the decay is the height of tensor {a1}, which is missing")
    return LayerSpec("gla", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), decay_root=float(m["tau"]), decay_rank=int(shapes[a1][0]))


def config_from_dict(d: dict, name: str = "zoguzen", dtype: str = "bf16", shapes: Optional[dict] = None) -> ModelConfig:
    """``shapes``: tensor name -> shape of the checkpoint (the rank of a decay's projection stands nowhere else)."""
    layers = []
    for i, entry in enumerate(d["layers"]):
        kind, m, ff = entry["type"], entry["mixer"], _feed_forward(i, entry.get("mlp"))
        if kind == "attention":
            src, mask = m.get("kv_from"), m.get("mask") or {"size": 0}
            layers.append(LayerSpec("attention", chunk=int(mask["size"]), softcap=float(m.get("softcap") or 0.0), unit_sink=True, talk=True, qkv_bias=True,
                                    head_norm=True, kv_from=-1 if src is None else int(src), **_attention(m), **ff))
        elif kind == "mingru":
            layers.append(LayerSpec("mingru", vdim=int(m["width"]), **ff))
        elif kind == "parallel":
            layers.append(LayerSpec("pair", pair=(_left(m["left"]), _right(i, m["right"], shapes)), **ff))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
    return composed_config(name, layers, hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), eps=float(d["norm"]["eps"]), pre_norm=True,
                           token_shift=True, side_dim=int((d.get("token_side") or {"dim": 0})["dim"]), logit_softcap=float(d.get("logit_softcap") or 0.0),
                           tie_word_embeddings=True, dtype=dtype)


def config_to_dict(cfg: ModelConfig) -> dict:
    def attention(s: LayerSpec) -> dict:
        return {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale, "conv": s.conv}

    layers = []
    for s in cfg.layer_specs:
        if s.mixer == "attention":
            m = {**attention(s), "mask": {"size": s.chunk}, "softcap": s.softcap}
            if s.kv_from >= 0:
                m["kv_from"] = s.kv_from
        elif s.mixer == "mingru":
            m = {"width": s.vdim}
        else:
            a, g = s.pair
            rot = {"dims": a.rot_dims, "base": a.rot_base}
            if a.rot_scaling is not None:
                rot["scaling"] = dict(zip(("factor", "low", "high", "original"), a.rot_scaling))
            m = {"left": {**attention(a), "mask": {"size": a.window, "keep_first": a.keep_first}, "rot": rot},
                 "right": {"heads": g.heads, "dim": g.dim, "vdim": g.vdim, "tau": g.decay_root}}
        e = s.moe
        mlp = None if e is None else {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top}}
        layers.append({"type": "parallel" if s.mixer == "pair" else s.mixer, "mixer": m, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "layers": layers, "norm": {"eps": cfg.rms_norm_eps}, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
            "token_side": {"dim": cfg.side_dim}, "logit_softcap": cfg.logit_softcap}


def _mixer_shapes(s: LayerSpec, m: str, W: int) -> dict:
    out = {m + "o": (W, s.heads * s.vdim)}
    if s.mixer == "mingru":
        return {**out, m + "z": (s.vdim, W), m + "z.b": (s.vdim,), m + "x": (s.vdim, W), m + "x.b": (s.vdim,), m + "g": (s.vdim, W)}
    if s.mixer == "gla":
        qd, vd = s.heads * s.dim, s.heads * s.vdim
        return {**out, m + "q": (qd, W), m + "k": (qd, W), m + "v": (vd, W), m + "g": (vd, W), m + "norm": (s.vdim,), m + "a1": (s.decay_rank, W),
                m + "a2": (qd, s.decay_rank), m + "a2.b": (qd,)}
    for k, n in (("q", s.heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim))[:3 if s.own_kv else 1]:
        out[m + k] = (n, W)
        if s.conv:
            out[m + k + ".conv"] = (n, s.conv)
        if s.qkv_bias:
            out[m + k + ".b"] = (n,)
        if s.head_norm and k != "v":
            out[m + k + ".norm"] = (s.dim,)
    if s.talk:
        out[m + "talk"] = (s.heads, s.heads)
    if s.out_gate:
        out[m + "g"] = (s.heads * s.vdim, W)
    return out


def tensor_shapes(cfg: ModelConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are ``[out, in]``)."""
    W, S = cfg.hidden_size, cfg.side_dim
    out = {"embed": (cfg.vocab_size, W), "final.norm": (W,)}
    if S:
        out["side.embed"] = (cfg.vocab_size, cfg.num_layers * S)
    for i, s in enumerate(cfg.layer_specs):
        p, m, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
        out.update({p + "norm1": (W,), p + "shift": (W,)})
        if s.pair is None:
            out.update(_mixer_shapes(s, m, W))
        else:
            for side, x in zip(("left.", "right."), s.pair):
                out.update({**_mixer_shapes(x, m + side, W), m + side + "out": (W,)})
        if s.moe is not None:
            out.update({p + "norm2": (W,), f + "router": (s.moe.experts, W)})
            for e in range(s.moe.experts):
                out.update({f"{f}e{e}.gate": (s.moe.ff, W), f"{f}e{e}.up": (s.moe.ff, W), f"{f}e{e}.down": (W, s.moe.ff)})
        if S:
            out.update({p + "side.gate": (S, W), p + "side.proj": (W, S), p + "side.norm": (W,)})
    return out


def _load_mixer(weights, s: LayerSpec, t: dict, m: str, o: str) -> None:
    """Tensors ``m...`` of one mixer into the parameters ``o...``."""
    p = weights.p

    def put_heads(dst, src, heads):
        """Rows of ``heads`` heads into rows of wider heads."""
        put(dst.view(heads, -1, *dst.shape[1:]), src.view(heads, -1, *src.shape[1:]))

    def out_heads(dst, vp):
        W = t[m + "o"].shape[0]
        put(dst[:, : s.heads * vp].view(-1, s.heads, vp), t[m + "o"].view(W, s.heads, s.vdim))

    if s.mixer == "mingru":
        n = pad_to(s.vdim, 8)
        for k, x in enumerate("zxg"):
            put(p[o + "gru_zxg"][k * n:], t[m + x])
        put(p[o + "gru_z_b"], t[m + "z.b"])
        put(p[o + "gru_x_b"], t[m + "x.b"])
        put(p[o + "gru_o"], t[m + "o"])
    elif s.mixer == "gla":
        at = weights.gla_columns(s)
        for x in ("q", "k", "v", "g", "a1"):
            put(p[o + "gla_in"][at[x]:], t[m + x])
        put(p[o + "gla_a2"], t[m + "a2"])
        put(p[o + "gla_a2_b"], t[m + "a2.b"])
        put(p[o + "gla_norm"], t[m + "norm"])
        put(p[o + "gla_o"], t[m + "o"])
    else:
        names = [k for k in "qkv" if m + k in t]
        rows = lambda suffix: torch.cat([t[m + k + suffix] for k in names])
        put(p[o + "attn_qkv"], rows(""))
        if s.conv:
            put(p[o + "attn_conv"], rows(".conv"))
        if s.qkv_bias:
            put(p[o + "attn_qkv_b"], rows(".b"))
        if s.head_norm:
            for k in names[:2]:
                put(p[f"{o}attn_{k}_norm"], t[f"{m}{k}.norm"])
        if s.talk:
            put(p[o + "attn_talk"], t[m + "talk"])
        vp = weights.attention_dims(s)[2]
        if s.out_gate:
            gate = weights.gate_column(s)
            put_heads(p[o + "attn_qkv"][gate: gate + s.heads * vp], t[m + "g"], s.heads)
        out_heads(p[o + "attn_o"], vp)


def load_tensors(cfg: ModelConfig, tensors: dict, weights) -> None:
    """Copy a checkpoint's tensors into a :class:`relax_b200.rollout.weights.RolloutWeights` buffer (zero-filled there, so
    every padded row and column stays zero).  Names and shapes must match exactly."""
    check_tensors(tensor_shapes(cfg), tensors)
    p = weights.p
    put(p["embed"], tensors["embed"])
    put(p["final_norm"], tensors["final.norm"])
    if cfg.side_dim:
        put(p["side_embed"], tensors["side.embed"])
    for i, s in enumerate(cfg.layer_specs):
        a, m, f, o = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", f"layers.{i}."
        put(p[o + "norm1"], tensors[a + "norm1"])
        put(p[o + "shift"], tensors[a + "shift"])
        if s.pair is None:
            _load_mixer(weights, s, tensors, m, o)
        else:
            for k, (side, x) in enumerate(zip(("left.", "right."), s.pair)):
                _load_mixer(weights, x, tensors, m + side, f"{o}{k}.")
                put(p[f"{o}{k}.out_norm"], tensors[m + side + "out"])
        if cfg.side_dim:
            for n in ("gate", "proj", "norm"):
                put(p[o + "side_" + n], tensors[a + "side." + n])
        if s.moe is not None:
            put(p[o + "norm2"], tensors[a + "norm2"])
            put(p[o + "moe_router"], tensors[f + "router"])
            up, down = p[o + "moe_up"], p[o + "moe_down"]
            for e in range(s.moe.experts):
                halves = torch.zeros(2, down.shape[2], up.shape[2], dtype=up.dtype, device=up.device)
                put(halves[0], tensors[f"{f}e{e}.gate"])
                put(halves[1], tensors[f"{f}e{e}.up"])
                up[e].copy_(glu_rows(*halves))
                put(down[e], tensors[f"{f}e{e}.down"])


def save(directory: str, cfg: ModelConfig, tensors: dict) -> None:
    save_folder(directory, config_to_dict(cfg), tensors)
