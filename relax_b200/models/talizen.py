"""Talizen: reader of the design's ``config.json`` and of its tensors.

A Talizen model is a composed stack (:class:`relax_b200.models.config.LayerSpec`): HGRN2 recurrent layers and latent-attention
layers in any order, each with its own sizes and with or without a gated feed-forward; output norms in groups; untied
embedding and head.  This module only translates names and layouts; the layers are computed by
:mod:`relax_b200.rollout.composed`.
"""
from __future__ import annotations

import torch

from .config import LayerSpec, ModelConfig, composed_config
from .native import check_tensors, put, save_folder

ARCHITECTURE = "Talizen"


def config_from_dict(d: dict, name: str = "talizen", dtype: str = "bf16", shapes=None) -> ModelConfig:
    layers = []
    for i, entry in enumerate(d["layers"]):
        kind, m, mlp = entry["type"], entry["mixer"], entry.get("mlp")
        if kind not in ("hgrn2", "latent_attention"):
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        ff = 0
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            ff = int(mlp["ff"])
        own = {"kv_rank": int(m["kv_rank"]), "scale": float(m["scale"])} if kind == "latent_attention" else {}
        layers.append(LayerSpec(kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), ff=ff, **own))
    return composed_config(name, layers, hidden_size=int(d["width"]), vocab_size=int(d["vocab"]),
                           norm_groups=int(d["norm"]["groups"]), eps=float(d["norm"]["eps"]), dtype=dtype)


def config_to_dict(cfg: ModelConfig) -> dict:
    layers = []
    for s in cfg.layer_specs:
        m = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim}
        if s.mixer == "latent_attention":
            m.update(kv_rank=s.kv_rank, scale=s.scale)
        layers.append({"type": s.mixer, "mixer": m, "mlp": {"kind": "dense", "ff": s.ff} if s.ff else None})
    return {"architecture": ARCHITECTURE, "layers": layers, "norm": {"eps": cfg.rms_norm_eps, "groups": cfg.norm_groups},
            "vocab": cfg.vocab_size, "width": cfg.hidden_size}


def tensor_shapes(cfg: ModelConfig) -> dict:
    """Checkpoint tensor name -> shape (linear weights are ``[out, in]``)."""
    W = cfg.hidden_size
    out = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), "final.norm": (W,)}
    for i, s in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", f"l{i}.mix."
        out[p + "norm1"] = (W,)
        qd, vd = s.heads * s.dim, s.heads * s.vdim
        if s.mixer == "hgrn2":
            out.update({m + "q": (qd, W), m + "f": (qd, W), m + "f.b": (qd,), m + "lower": (qd,), m + "v": (vd, W), m + "norm": (s.vdim,)})
        else:
            out.update({m + "q": (qd, W), m + "dkv": (s.kv_rank, W), m + "dkv.norm": (s.kv_rank,), m + "uk": (qd, s.kv_rank),
                        m + "uv": (vd, s.kv_rank), m + "g": (s.heads, W)})
        out[m + "o"] = (W, vd)
        if s.ff:
            out[p + "norm2"] = (W,)
            out.update({p + "mlp.gate": (s.ff, W), p + "mlp.up": (s.ff, W), p + "mlp.down": (W, s.ff)})
    return out


def load_tensors(cfg: ModelConfig, tensors: dict, weights) -> None:
    """Copy a checkpoint's tensors into a :class:`relax_b200.rollout.weights.RolloutWeights` buffer (zero-filled there, so
    every padded row and column stays zero).  Names and shapes must match exactly."""
    check_tensors(tensor_shapes(cfg), tensors)
    p, W = weights.p, cfg.hidden_size
    put(p["embed"], tensors["embed"])
    put(p["lm_head"], tensors["head"])
    put(p["final_norm"], tensors["final.norm"])
    for i, s in enumerate(cfg.layer_specs):
        a, m, o = f"l{i}.", f"l{i}.mix.", f"layers.{i}."
        H, qd, vd = s.heads, s.heads * s.dim, s.heads * s.vdim
        put(p[o + "post_attn_norm"], tensors[a + "norm1"])
        if s.mixer == "hgrn2":
            put(p[o + "rec_qfv"], torch.cat([tensors[m + "q"], tensors[m + "f"], tensors[m + "v"]]))
            put(p[o + "rec_f_bias"], tensors[m + "f.b"])
            put(p[o + "rec_lower"], tensors[m + "lower"])
            put(p[o + "rec_norm"], tensors[m + "norm"])
            put(p[o + "rec_o"], tensors[m + "o"])
        else:
            R, (dp, vp, Rp) = s.kv_rank, weights.latent_dims(s)
            w = p[o + "lat_qcg"]
            put(w[: H * dp].view(H, dp, -1), tensors[m + "q"].view(H, s.dim, W))
            put(w[H * dp:], tensors[m + "dkv"])
            put(w[H * dp + Rp:], tensors[m + "g"])
            put(p[o + "lat_norm"], tensors[m + "dkv.norm"])
            put(p[o + "lat_uk"].view(H, dp, Rp), tensors[m + "uk"].view(H, s.dim, R))
            put(p[o + "lat_uv"].view(H, vp, Rp), tensors[m + "uv"].view(H, s.vdim, R))
            put(p[o + "lat_o"][:, : H * vp].view(-1, H, vp), tensors[m + "o"].view(W, H, s.vdim))
        if s.ff:
            put(p[o + "post_mlp_norm"], tensors[a + "norm2"])
            Fp = p[o + "gate_up"].shape[0] // 2
            put(p[o + "gate_up"], tensors[a + "mlp.gate"])
            put(p[o + "gate_up"][Fp:], tensors[a + "mlp.up"])
            put(p[o + "down"], tensors[a + "mlp.down"])


def save(directory: str, cfg: ModelConfig, tensors: dict) -> None:
    save_folder(directory, config_to_dict(cfg), tensors)
