"""Ketolorn: reader of the design's ``config.json`` and of its tensors.

A Ketolorn model is a composed stack (:class:`relax_b200.models.config.LayerSpec`) of softmax-attention layers: rotated, then
normed queries and keys, one sink logit per head, keys and values that a layer projects itself or takes from an earlier layer's
cache; feed-forwards that are gated (silu), routed over grouped experts with a shared one, or absent; norms on the sublayers'
outputs, on the embedded tokens and before the logits, which the embedding table gives.  This module only translates names and
layouts; the layers are computed by :mod:`relax_b200.rollout.composed`.
"""
from __future__ import annotations

import torch

from .config import LayerSpec, ModelConfig, MoESpec, composed_config
from .native import check_tensors, put, save_folder

ARCHITECTURE = "Ketolorn"


def _feed_forward(i: int, mlp) -> dict:
    if mlp is None:
        return {}
    if mlp["kind"] == "dense":
        return {"ff": int(mlp["ff"])}
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    r = mlp["router"]
    g, shared = r.get("groups") or {"count": 1, "keep": 1}, mlp.get("shared")
    return {"moe": MoESpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), groups=int(g["count"]),
                           keep=int(g["keep"]), shared_ff=int(shared["ff"]) if shared else 0)}


def config_from_dict(d: dict, name: str = "ketolorn", dtype: str = "bf16", shapes=None) -> ModelConfig:
    layers = []
    for i, entry in enumerate(d["layers"]):
        m = entry["mixer"]
        if entry["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        rot, src = m.get("rot") or {"dims": 0, "base": 0.0}, m.get("kv_from")
        layers.append(LayerSpec("attention", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_heads=int(m["kv_heads"]),
                                scale=float(m["scale"]), rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), qk_norm=True, sink=True,
                                act="silu", kv_from=-1 if src is None else int(src), **_feed_forward(i, entry.get("mlp"))))
    return composed_config(name, layers, hidden_size=int(d["width"]), vocab_size=int(d["vocab"]), eps=float(d["norm"]["eps"]),
                           embed_norm=True, tie_word_embeddings=True, dtype=dtype)


def config_to_dict(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale,
             "rot": {"dims": s.rot_dims, "base": s.rot_base}}
        if s.kv_from >= 0:
            m["kv_from"] = s.kv_from
        mlp = {"kind": "dense", "ff": s.ff} if s.ff else None
        if s.moe is not None:
            e = s.moe
            mlp = {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top, "groups": {"count": e.groups, "keep": e.keep}}}
            if e.shared_ff:
                mlp["shared"] = {"ff": e.shared_ff}
        layers.append({"type": "attention", "mixer": m, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "layers": layers, "norm": {"eps": cfg.rms_norm_eps}, "vocab": cfg.vocab_size, "width": cfg.hidden_size}


def tensor_shapes(cfg: ModelConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are ``[out, in]``)."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "embed.norm": (W,), "final.norm": (W,)}
    for i, s in enumerate(cfg.layer_specs):
        p, m, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
        out[p + "norm1"] = (W,)
        out.update({m + "q": (s.heads * s.dim, W), m + "sink": (s.heads,), m + "o": (W, s.heads * s.vdim)})
        if s.own_kv:
            out.update({m + "k": (s.kv_heads * s.dim, W), m + "v": (s.kv_heads * s.vdim, W)})
        if s.has_ff:
            out[p + "norm2"] = (W,)
        if s.ff:
            out.update({f + "gate": (s.ff, W), f + "up": (s.ff, W), f + "down": (W, s.ff)})
        if s.moe is not None:
            out[f + "router"] = (s.moe.experts, W)
            for e in range(s.moe.experts):
                out.update({f"{f}e{e}.up": (s.moe.ff, W), f"{f}e{e}.down": (W, s.moe.ff)})
            if s.moe.shared_ff:
                out.update({f + "shared.up": (s.moe.shared_ff, W), f + "shared.down": (W, s.moe.shared_ff)})
    return out


def load_tensors(cfg: ModelConfig, tensors: dict, weights) -> None:
    """Copy a checkpoint's tensors into a :class:`relax_b200.rollout.weights.RolloutWeights` buffer (zero-filled there, so
    every padded row and column stays zero).  Names and shapes must match exactly."""
    check_tensors(tensor_shapes(cfg), tensors)
    p, W = weights.p, cfg.hidden_size
    put(p["embed"], tensors["embed"])
    put(p["embed_norm"], tensors["embed.norm"])
    put(p["final_norm"], tensors["final.norm"])
    for i, s in enumerate(cfg.layer_specs):
        a, m, f, o = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", f"layers.{i}."
        put(p[o + "post_attn_norm"], tensors[a + "norm1"])
        put(p[o + "attn_qkv"], torch.cat([tensors[m + k] for k in ("q", "k", "v") if m + k in tensors]))
        put(p[o + "attn_sink"], tensors[m + "sink"])
        put(p[o + "attn_o"].view(-1, s.heads, weights.attention_dims(s)[2]), tensors[m + "o"].view(W, s.heads, s.vdim))
        if s.has_ff:
            put(p[o + "post_mlp_norm"], tensors[a + "norm2"])
        if s.ff:
            put(p[o + "gate_up"], tensors[f + "gate"])
            put(p[o + "gate_up"][p[o + "gate_up"].shape[0] // 2:], tensors[f + "up"])
            put(p[o + "down"], tensors[f + "down"])
        if s.moe is not None:
            put(p[o + "moe_router"], tensors[f + "router"])
            for e in range(s.moe.experts):
                put(p[o + "moe_up"][e], tensors[f"{f}e{e}.up"])
                put(p[o + "moe_down"][e], tensors[f"{f}e{e}.down"])
            if s.moe.shared_ff:
                put(p[o + "shared_up"], tensors[f + "shared.up"])
                put(p[o + "shared_down"], tensors[f + "shared.down"])


def save(directory: str, cfg: ModelConfig, tensors: dict) -> None:
    save_folder(directory, config_to_dict(cfg), tensors)
