"""Zupupel: reader of the design's ``config.json`` and of its tensors.

A Zupupel model is a composed stack (:class:`relax_b200.models.config.LayerSpec`) of sliding-window attention layers (norms over the
whole query and key projections, halves of a head's leading features turned together, keys and values that a layer projects
itself or takes from an earlier layer's cache) and latent-attention layers with a rotated key part, each with a gate per output
feature; routed feed-forwards with identity experts, or none; layer norms after every sum; an embedding factor, a logit factor and
an output matrix of its own.  This module only translates names and layouts; the layers are computed by
:mod:`relax_b200.rollout.composed`.
"""
from __future__ import annotations

import torch

from ..ops import glu_rows
from .config import LayerSpec, ModelConfig, MoESpec, composed_config
from .native import check_tensors, put, save_folder

ARCHITECTURE = "Zupupel"


def _feed_forward(i: int, mlp) -> dict:
    if mlp is None:
        return {}
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    return {"moe": MoESpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), groups=int(g["count"]), keep=int(g["keep"]),
                           act="clamped_swish", limit=float(mlp["expert"]["limit"]), renormalize=True, score="softmax", correction=True,
                           identity=int(r.get("identity") or 0), group_best=1)}


def config_from_dict(d: dict, name: str = "zupupel", dtype: str = "bf16", shapes=None) -> ModelConfig:
    layers = []
    for i, entry in enumerate(d["layers"]):
        m = entry["mixer"]
        rot = m.get("rot") or {"dims": 0, "base": 0.0}
        common = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), rot_dims=int(rot["dims"]),
                      rot_base=float(rot["base"]), out_gate=True, **_feed_forward(i, entry.get("mlp")))
        if entry["type"] == "attention":
            src, mask = m.get("kv_from"), m.get("mask") or {"size": 0}
            layers.append(LayerSpec("attention", kv_heads=int(m["kv_heads"]), rot_halves=True, proj_norm=True, window=int(mask["size"]),
                                    kv_from=-1 if src is None else int(src), **common))
        elif entry["type"] == "latent_attention":
            if int(m["rot_dim"]) != int(rot["dims"]):
                raise ValueError(f"layer {i}: {rot['dims']} of {m['rot_dim']} features of the rotated part turn")
            layers.append(LayerSpec("latent_attention", kv_rank=int(m["kv_rank"]), **common))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
    return composed_config(name, layers, hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), eps=float(d["norm"]["eps"]), norm_sum=True,
                           sum_alpha=float(d["postln_alpha"]), embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]), dtype=dtype)


def config_to_dict(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale, "rot": {"dims": s.rot_dims, "base": s.rot_base}}
        if s.mixer == "attention":
            m["kv_heads"] = s.kv_heads
            if s.window:
                m["mask"] = {"size": s.window}
            if s.kv_from >= 0:
                m["kv_from"] = s.kv_from
        else:
            m.update(kv_rank=s.kv_rank, rot_dim=s.rot_dims)
        e = s.moe
        mlp = None if e is None else {"kind": "moe", "expert": {"ff": e.ff, "limit": e.limit},
                                      "router": {"experts": e.experts, "top": e.top, "identity": e.identity, "groups": {"count": e.groups, "keep": e.keep}}}
        layers.append({"type": s.mixer, "mixer": m, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "layers": layers, "norm": {"eps": cfg.rms_norm_eps}, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
            "embedding": {"scale": cfg.embed_scale}, "logit_scale": cfg.logit_scale, "postln_alpha": cfg.sum_alpha}


def tensor_shapes(cfg: ModelConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are ``[out, in]``)."""
    W = cfg.hidden_size
    norm = lambda n: {n: (W,), n + ".b": (W,)}
    out = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), **norm("final.norm")}
    for i, s in enumerate(cfg.layer_specs):
        p, m, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
        out.update({**norm(p + "norm1"), m + "g": (s.heads * s.vdim, W), m + "o": (W, s.heads * s.vdim)})
        if s.mixer == "attention":
            out.update({m + "q": (s.heads * s.dim, W), m + "q.norm": (s.heads * s.dim,)})
            if s.own_kv:
                out.update({m + "k": (s.kv_heads * s.dim, W), m + "k.norm": (s.kv_heads * s.dim,), m + "v": (s.kv_heads * s.vdim, W)})
        else:
            out.update({m + "q": (s.heads * (s.dim + s.rot_dims), W), m + "dkv": (s.kv_rank + s.rot_dims, W), m + "dkv.norm": (s.kv_rank,),
                        m + "uk": (s.heads * s.dim, s.kv_rank), m + "uv": (s.heads * s.vdim, s.kv_rank)})
        if s.moe is not None:
            out.update({**norm(p + "norm2"), f + "router": (s.moe.outputs, W), f + "correction": (s.moe.outputs,)})
            for e in range(s.moe.experts):
                out.update({f"{f}e{e}.gate": (s.moe.ff, W), f"{f}e{e}.up": (s.moe.ff, W), f"{f}e{e}.down": (W, s.moe.ff)})
    return out


def load_tensors(cfg: ModelConfig, tensors: dict, weights) -> None:
    """Copy a checkpoint's tensors into a :class:`relax_b200.rollout.weights.RolloutWeights` buffer (zero-filled there, so
    every padded row and column stays zero).  Names and shapes must match exactly."""
    check_tensors(tensor_shapes(cfg), tensors)
    p, W = weights.p, cfg.hidden_size

    def norm(dst, name):
        put(p[dst], tensors[name])
        put(p[dst + "_b"], tensors[name + ".b"])

    def put_heads(dst, src, heads):
        """Rows of ``heads`` heads into rows of wider heads."""
        put(dst.view(heads, -1, dst.shape[1]), src.view(heads, -1, src.shape[1]))

    put(p["embed"], tensors["embed"])
    put(p["lm_head"], tensors["head"])
    norm("final_norm", "final.norm")
    for i, s in enumerate(cfg.layer_specs):
        a, m, f, o = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", f"layers.{i}."
        H = s.heads
        norm(o + "post_attn_norm", a + "norm1")
        if s.mixer == "attention":
            w, vp = p[o + "attn_qkv"], weights.attention_dims(s)[2]
            put(w, torch.cat([tensors[m + k] for k in ("q", "k", "v") if m + k in tensors]))
            for k in ("q", "k") if s.own_kv else ("q",):
                put(p[f"{o}attn_{k}_norm"], tensors[f"{m}{k}.norm"])
            gate, out = weights.gate_column(s), p[o + "attn_o"]
        else:
            dp, vp, Rp = weights.latent_dims(s)
            w, dkv = p[o + "lat_qcg"], tensors[m + "dkv"]
            put_heads(w[: H * dp], tensors[m + "q"], H)
            put(w[H * dp:], dkv[: s.kv_rank])
            put(w[H * dp + Rp:], dkv[s.kv_rank:])
            put(p[o + "lat_norm"], tensors[m + "dkv.norm"])
            put_heads(p[o + "lat_uk"], tensors[m + "uk"], H)
            put_heads(p[o + "lat_uv"], tensors[m + "uv"], H)
            weights.pass_rotated_keys(i)
            gate, out = H * dp + Rp + (s.rot_dims + 7) // 8 * 8, p[o + "lat_o"]
        put_heads(w[gate: gate + H * vp], tensors[m + "g"], H)
        put(out.view(-1, H, vp), tensors[m + "o"].view(W, H, s.vdim))
        if s.moe is not None:
            norm(o + "post_mlp_norm", a + "norm2")
            put(p[o + "moe_router"], tensors[f + "router"])
            put(p[o + "moe_correction"], tensors[f + "correction"])
            up, down = p[o + "moe_up"], p[o + "moe_down"]
            for e in range(s.moe.experts):
                halves = torch.zeros(2, down.shape[2], up.shape[2], dtype=up.dtype, device=up.device)
                put(halves[0], tensors[f"{f}e{e}.gate"])
                put(halves[1], tensors[f"{f}e{e}.up"])
                up[e].copy_(glu_rows(*halves))
                put(down[e], tensors[f"{f}e{e}.down"])


def save(directory: str, cfg: ModelConfig, tensors: dict) -> None:
    save_folder(directory, config_to_dict(cfg), tensors)
