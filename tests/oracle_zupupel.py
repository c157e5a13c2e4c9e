"""Plain float64 statements of the layers of Zupupel stacks, written from their equations, one function per mechanism, and small
random models to run them on.  Nothing here is shared with the engine."""
import copy
import math

import torch

F64 = torch.float64


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def centred(x, w, b, eps):
    """Layer norm: deviations from the mean over the root of their mean square."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def _pair(u, v, position, i, dims, base):
    a = position * base ** (-2 * i / dims)
    return u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)


def turn_halves(x, positions, dims, base):
    """x [T, heads, d]: features i and i + dims / 2 turn together."""
    y = x.clone()
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            y[t, :, i], y[t, :, i + dims // 2] = _pair(x[t, :, i], x[t, :, i + dims // 2], p, i, dims, base)
    return y


def turn_neighbours(x, positions, dims, base):
    """x [T, heads, d]: features 2 i and 2 i + 1 turn together."""
    y = x.clone()
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            y[t, :, 2 * i], y[t, :, 2 * i + 1] = _pair(x[t, :, 2 * i], x[t, :, 2 * i + 1], p, i, dims, base)
    return y


def attend(q, k, v, first, scale, window=None):
    """q [n, H, d] at positions first .. first + n - 1 over k [L, G, d], v [L, G, dv]: every position sees itself and what is behind it,
    with a window only itself and the window - 1 positions before.  Returns [n, H, dv]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for i in range(n):
        end = first + i + 1
        lo = 0 if window is None else max(0, end - window)
        for h in range(H):
            s = k[lo:end, h // rep] @ q[i, h] * scale
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:end, h // rep]
    return out


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def latent_keys_values(c, turned, uk, uv, H):
    """Latent rows c [L, R] and shared turned parts [L, r] -> keys [L, H, d + r], values [L, H, dv]."""
    L = c.shape[0]
    k = (c @ uk.T).view(L, H, -1)
    return torch.cat([k, turned[:, None, :].expand(L, H, turned.shape[1])], -1), (c @ uv.T).view(L, H, -1)


def expert(h, gate, up, down, limit):
    g, u = (h @ gate.T).clamp(max=limit), (h @ up.T).clamp(min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def choose(choice, top, groups, keep):
    """Chosen outputs of one row by its choice scores, and how far the choice is from another one."""
    n = len(choice) // groups
    worth = [max(choice[g * n:(g + 1) * n]) for g in range(groups)]
    by_worth = sorted(range(groups), key=lambda g: -worth[g])
    kept, gap = by_worth[:keep], math.inf
    if keep < groups:
        gap = worth[kept[-1]] - worth[by_worth[keep]]
    allowed = sorted((e for e in range(len(choice)) if e // n in kept), key=lambda e: -choice[e])
    if top < len(allowed):
        gap = min(gap, choice[allowed[top - 1]] - choice[allowed[top]])
    return allowed[:top], gap


def weigh(z):
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def routed(h, w, mlp):
    """(output, gap of the closest choice per row)"""
    r, g, limit = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}, mlp["expert"]["limit"]
    out, gaps = torch.zeros_like(h), []
    s = weigh(h @ w["router"].T)
    for t in range(h.shape[0]):
        chosen, gap = choose((s[t] + w["correction"]).tolist(), r["top"], g["count"], g["keep"])
        gaps.append(gap)
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            y = h[t] if e >= r["experts"] else expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], limit)
            out[t] += s[t, e] / total * y
    return out, torch.tensor(gaps)


def mix_attention(x, t, m, eps, cached, i):
    T, H, G, d = x.shape[0], m["heads"], m["kv_heads"], m["dim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = turn_halves(rms(x @ t["q"].T, t["q.norm"], eps).view(T, H, d), range(T), rot["dims"], rot["base"])
    if "kv_from" in m:
        k, v = cached[m["kv_from"]]
    else:
        k = turn_halves(rms(x @ t["k"].T, t["k.norm"], eps).view(T, G, d), range(T), rot["dims"], rot["base"])
        v = (x @ t["v"].T).view(T, G, m["vdim"])
        cached[i] = (k, v)
    o = attend(q, k, v, 0, m["scale"], (m.get("mask") or {}).get("size"))
    return (o.reshape(T, -1) * sigmoid(x @ t["g"].T)) @ t["o"].T


def mix_latent(x, t, m, eps):
    T, H, d, r, R = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (x @ t["q"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], turn_neighbours(q[..., d:], range(T), r, base)], -1)
    row = x @ t["dkv"].T
    c, turned = rms(row[:, :R], t["dkv.norm"], eps), turn_neighbours(row[:, None, R:], range(T), r, base)[:, 0]
    k, v = latent_keys_values(c, turned, t["uk"], t["uv"], H)
    return (attend(q, k, v, 0, m["scale"]).reshape(T, -1) * sigmoid(x @ t["g"].T)) @ t["o"].T


def run(cfg, tensors, tokens):
    """(logits [T, vocab], gap of the closest expert choice of every row, streams after the layers)"""
    w = {k: v.to(F64) for k, v in tensors.items()}
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    eps, T, alpha = cfg["norm"]["eps"], len(tokens), cfg["postln_alpha"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    gaps, cached, streams = torch.full((T,), math.inf, dtype=F64), {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, t, m = f"l{i}.", sub(f"l{i}.mix."), layer["mixer"]
        y = mix_attention(x, t, m, eps, cached, i) if layer["type"] == "attention" else mix_latent(x, t, m, eps)
        x = centred(alpha * x + y, w[p + "norm1"], w[p + "norm1.b"], eps)
        if layer["mlp"] is not None:
            y, gap = routed(x, sub(p + "mlp."), layer["mlp"])
            gaps = torch.minimum(gaps, gap)
            x = centred(alpha * x + y, w[p + "norm2"], w[p + "norm2.b"], eps)
        streams.append(x)
    return centred(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T * cfg["logit_scale"], gaps, streams


def model(cfg, tensors, tokens):
    return run(cfg, tensors, tokens)[0]


# ---------------------------------------------------------------------------------------------------- random models


def moe(experts, top, ff, limit, identity=0, groups=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "identity": identity, "groups": {"count": groups, "keep": keep}}}


def att(heads, kv_heads, dim, vdim, scale, rot, base, window, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot, "base": base}, "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lat(heads, dim, rot, vdim, rank, scale, base, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                             "rot": {"dims": rot, "base": base}}}


def stack(width, vocab, eps, layers, alpha=1.7, embed=0.8, logit=0.6):
    return {"architecture": "Zupupel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed}, "logit_scale": logit,
            "postln_alpha": alpha, "layers": layers}


CONFIGS = {
    # every padding rule at once: nothing is a multiple of anything; readers with other windows than their source, above a latent layer
    "odd": stack(74, 131, 3e-5, [att(6, 2, 18, 13, 0.31, 10, 1e3, 21, moe(7, 2, 20, 0.7, 2, 3, 2)), lat(3, 10, 6, 7, 20, 0.4, 300.0, moe(5, 2, 9, 1.3, 1, 2, 1)),
                                 att(6, 2, 18, 13, 0.22, 10, 1e3, 9, moe(4, 3, 33, 0.5, 3), 0), att(5, 5, 7, 9, 0.9, 4, 50.0, 33),
                                 att(6, 2, 18, 13, 0.4, 10, 1e3, 40, moe(6, 1, 12, 2.0, 0, 2, 2), 0)]),
    # whole heads turn; wide groups, narrow keys beside wide values, a whole latent layer between
    "even": stack(128, 256, 1e-4, [lat(8, 56, 24, 64, 128, 0.12, 1e4, moe(12, 4, 64, 1.5, 4, 4, 2)), att(8, 1, 64, 128, 0.2, 64, 1e4, 48, moe(8, 2, 64, 1.0, 0, 4, 2)),
                                   att(4, 4, 128, 32, 0.11, 32, 1e5, 100, moe(14, 3, 128, 0.8, 2, 2, 1)), att(4, 4, 128, 32, 0.2, 32, 1e5, 64, None, 2),
                                   lat(16, 96, 32, 128, 192, 0.1, 1e5)], 2.5, 3.0, 1.4),
    # one head, one feature pair, a window of one token, experts of one per group
    "single": stack(64, 65, 1e-6, [att(1, 1, 16, 40, 0.7, 2, 10.0, 1, moe(3, 2, 8, 1.0, 1, 4, 3)), lat(1, 8, 2, 5, 12, 0.7, 10.0, moe(2, 1, 8, 0.4)),
                                   att(1, 1, 16, 40, 0.5, 2, 10.0, 500, None, 0)], 1.0, 1.0, 1.0),
    # more heads per group than the decode tile takes; heads and latent rows wider than the tensor-core kernels take
    "wide": stack(256, 320, 1e-5, [att(40, 2, 24, 16, 0.3, 8, 1e4, 17, moe(8, 3, 96, 1.0, 4, 2, 1)), att(3, 1, 144, 136, 0.1, 96, 1e6, 70),
                                   lat(6, 96, 64, 100, 576, 0.09, 1e4, moe(6, 2, 64, 3.0, 2, 2, 2)), lat(20, 24, 16, 24, 40, 0.3, 1e4)]),
}


def random_model(cfg, seed=0, sharp=1.0):
    """bf16-representable random tensors; ``sharp`` multiplies the attention scales of the configuration that comes back."""
    cfg = copy.deepcopy(cfg)
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    lin = lambda out, fan: n(out, fan, std=fan ** -0.5)
    t = {"embed": n(V, W), "head": n(V, W, std=W ** -0.5), "final.norm": 1 + n(W, std=0.2), "final.norm.b": n(W, std=0.2)}
    for i, layer in enumerate(cfg["layers"]):
        m, a, p, f, mlp = layer["mixer"], f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", layer["mlp"]
        m["scale"] *= sharp
        H, vd = m["heads"], m["heads"] * m["vdim"]
        t.update({a + "norm1": 1 + n(W, std=0.2), a + "norm1.b": n(W, std=0.2), p + "g": lin(vd, W), p + "o": lin(W, vd) * 2})
        if layer["type"] == "attention":
            qd, kd = H * m["dim"], m["kv_heads"] * m["dim"]
            t.update({p + "q": lin(qd, W), p + "q.norm": 1.2 + n(qd, std=0.3)})
            if "kv_from" not in m:
                t.update({p + "k": lin(kd, W), p + "k.norm": 1.2 + n(kd, std=0.3), p + "v": lin(m["kv_heads"] * m["vdim"], W)})
        else:
            R = m["kv_rank"]
            t.update({p + "q": lin(H * (m["dim"] + m["rot_dim"]), W) * 1.5, p + "dkv": lin(R + m["rot_dim"], W), p + "dkv.norm": 1 + n(R, std=0.2),
                      p + "uk": lin(H * m["dim"], R) * 1.5, p + "uv": lin(vd, R)})
        if mlp is None:
            continue
        r, ff = mlp["router"], mlp["expert"]["ff"]
        N = r["experts"] + r["identity"]
        t.update({a + "norm2": 1 + n(W, std=0.2), a + "norm2.b": n(W, std=0.2), f + "router": lin(N, W) * 1.5, f + "correction": n(N, std=0.3) - 0.4})
        for e in range(r["experts"]):
            t.update({f"{f}e{e}.gate": lin(ff, W) * 2, f"{f}e{e}.up": lin(ff, W) * 2, f"{f}e{e}.down": lin(W, ff)})
    return cfg, {k: v.to(torch.bfloat16) for k, v in t.items()}
