"""Plain float64 statements of the layers of Ketolorn stacks, written from their equations, one function per mechanism, and small
random models to run them on.  Nothing here is shared with the engine."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def turn(x, positions, dims, base):
    """x [T, heads, dim]: features 2i and 2i + 1 below ``dims`` turn by position * base^(-2i / dims)."""
    y = x.clone()
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = p * base ** (-2 * i / dims)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i] = u * math.cos(a) - v * math.sin(a)
            y[t, :, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return y


def attend(q, k, v, first, scale, sink=None):
    """q [n, H, d] at positions first .. first + n - 1 over k [L, G, d], v [L, G, dv]; returns [n, H, dv]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for i in range(n):
        L = first + i + 1
        for h in range(H):
            s = k[:L, h // rep] @ q[i, h] * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - top)
            den = p.sum() if sink is None else p.sum() + torch.exp(sink[h] - top)
            out[i, h] = p @ v[:L, h // rep] / den
    return out


def silu(x):
    return x / (1 + torch.exp(-x))


def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def expert(h, up, down):
    z = h @ up.T
    return torch.where(z > 0, z ** 2, torch.zeros_like(z)) @ down.T


def choose(scores, top, groups, keep):
    """Chosen experts of one row, and how far the choice is from another one."""
    n = len(scores) // groups
    worth = []
    for g in range(groups):
        best = sorted(scores[g * n:(g + 1) * n], reverse=True)
        worth.append(sum(best[:2]))
    by_worth = sorted(range(groups), key=lambda g: -worth[g])
    kept = by_worth[:keep]
    gap = worth[kept[-1]] - worth[by_worth[keep]] if keep < groups else math.inf
    allowed = sorted((e for e in range(len(scores)) if e // n in kept), key=lambda e: -scores[e])
    if top < len(allowed):
        gap = min(gap, scores[allowed[top - 1]] - scores[allowed[top]])
    return allowed[:top], gap


def routed(h, w, mlp):
    """(output, gap of the closest choice per row)"""
    r, g = mlp["router"], mlp["router"]["groups"]
    out, gaps = torch.zeros_like(h), []
    s = 1 / (1 + torch.exp(-(h @ w["router"].T)))
    for t in range(h.shape[0]):
        chosen, gap = choose(s[t].tolist(), r["top"], g["count"], g["keep"])
        gaps.append(gap)
        for e in chosen:
            out[t] += s[t, e] * expert(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if "shared" in mlp:
        out += expert(h, w["shared.up"], w["shared.down"])
    return out, torch.tensor(gaps)


def run(cfg, tensors, tokens):
    """(logits [T, vocab], gap of the closest expert choice of every row, streams after the layers)"""
    w = {k: v.to(F64) for k, v in tensors.items()}
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    eps, T = cfg["norm"]["eps"], len(tokens)
    x = rms(w["embed"][torch.tensor(tokens)], eps) * w["embed.norm"]
    gaps, cached, streams = torch.full((T,), math.inf, dtype=F64), {}, []
    for i, layer in enumerate(cfg["layers"]):
        m, t = layer["mixer"], sub(f"l{i}.mix.")
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        q = rms(turn((x @ t["q"].T).view(T, H, d), range(T), m["rot"]["dims"], m["rot"]["base"]), eps)
        if "kv_from" in m:
            k, v = cached[m["kv_from"]]
        else:
            k = rms(turn((x @ t["k"].T).view(T, G, d), range(T), m["rot"]["dims"], m["rot"]["base"]), eps)
            v = (x @ t["v"].T).view(T, G, m["vdim"])
            cached[i] = (k, v)
        y = attend(q, k, v, 0, m["scale"], t["sink"]).reshape(T, -1) @ t["o"].T
        x = x + rms(y, eps) * w[f"l{i}.norm1"]
        mlp = layer["mlp"]
        if mlp is not None:
            t = sub(f"l{i}.mlp.")
            if mlp["kind"] == "dense":
                y = gated(x, t["gate"], t["up"], t["down"])
            else:
                y, gap = routed(x, t, mlp)
                gaps = torch.minimum(gaps, gap)
            x = x + rms(y, eps) * w[f"l{i}.norm2"]
        streams.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T, gaps, streams


def model(cfg, tensors, tokens):
    return run(cfg, tensors, tokens)[0]


# ---------------------------------------------------------------------------------------------------- random models


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups, keep, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    return {**m, "shared": {"ff": shared}} if shared else m


def att(heads, kv_heads, dim, vdim, scale, rot, base, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def stack(width, vocab, eps, layers):
    return {"architecture": "Ketolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # every padding rule at once: nothing is a multiple of anything; a reader two layers up, two sources, three heads per group
    "odd": stack(74, 131, 3e-5, [att(6, 2, 18, 13, 0.31, 10, 1e3, moe(6, 2, 20, 3, 2, 12)), att(5, 5, 7, 9, 0.9, 4, 50.0),
                                 att(6, 2, 18, 13, 0.22, 10, 1e3, dense(50), 0), att(5, 5, 7, 9, 1.3, 4, 50.0, moe(9, 3, 30, 3, 2), 1),
                                 att(6, 2, 18, 13, 0.4, 10, 1e3, moe(5, 1, 33, 1, 1, 70), 0)]),
    # whole heads turn; eight heads per group, narrow keys beside wide values
    "even": stack(128, 256, 1e-4, [att(8, 1, 64, 128, 0.2, 64, 1e4, dense(192)), att(4, 4, 128, 32, 0.11, 32, 1e5, moe(16, 4, 64, 4, 2, 64)),
                                   att(8, 1, 64, 128, 0.3, 64, 1e4, moe(16, 4, 128, 2, 1, 128), 0), att(4, 4, 128, 32, 0.2, 32, 1e5, None, 1)]),
    # one head, one expert per group, no feed-forward after the last attention
    "single": stack(64, 65, 1e-6, [att(1, 1, 16, 40, 0.7, 2, 10.0, moe(4, 2, 8, 4, 3)), att(1, 1, 16, 40, 0.5, 2, 10.0, None, 0)]),
    # more heads per group than the decode tile takes; heads wider than the tensor-core kernels take
    "wide": stack(256, 320, 1e-5, [att(40, 2, 24, 16, 0.3, 8, 1e4, moe(12, 3, 96, 2, 1, 160)), att(3, 1, 144, 136, 0.1, 96, 1e6, dense(128)),
                                   att(24, 2, 96, 72, 0.15, 96, 1e4, None), att(24, 2, 96, 72, 0.2, 96, 1e4, dense(64), 2)]),
}


def random_model(cfg, seed=0, sharp=1.0):
    """bf16-representable random tensors.  ``sharp`` multiplies the attention scales of the configuration it returns with the
    tensors: queries and keys have unit size, so the scale decides whether single keys dominate."""
    import copy

    cfg = copy.deepcopy(cfg)
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    t = {"embed": n(V, W), "embed.norm": 1 + n(W, std=0.2), "final.norm": (1 + n(W, std=0.2)) * W ** -0.5}
    for i, layer in enumerate(cfg["layers"]):
        m, p, f, mlp = layer["mixer"], f"l{i}.mix.", f"l{i}.mlp.", layer["mlp"]
        m["scale"] *= sharp
        qd, vd = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        t[f"l{i}.norm1"] = 0.6 + n(W, std=0.2)
        t.update({p + "q": n(qd, W, std=W ** -0.5), p + "o": n(W, vd, std=vd ** -0.5), p + "sink": 1.5 + n(m["heads"])})
        if "kv_from" not in m:
            t.update({p + "k": n(m["kv_heads"] * m["dim"], W, std=W ** -0.5), p + "v": n(m["kv_heads"] * m["vdim"], W, std=W ** -0.5)})
        if mlp is None:
            continue
        t[f"l{i}.norm2"] = 0.6 + n(W, std=0.2)
        if mlp["kind"] == "dense":
            ff = mlp["ff"]
            t.update({f + "gate": n(ff, W, std=W ** -0.5), f + "up": n(ff, W, std=W ** -0.5), f + "down": n(W, ff, std=ff ** -0.5)})
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        t[f + "router"] = n(E, W, std=W ** -0.5)
        for e in range(E):
            t.update({f"{f}e{e}.up": n(ff, W, std=W ** -0.5), f"{f}e{e}.down": n(W, ff, std=ff ** -0.5)})
        if "shared" in mlp:
            s = mlp["shared"]["ff"]
            t.update({f + "shared.up": n(s, W, std=W ** -0.5), f + "shared.down": n(W, s, std=s ** -0.5)})
    return cfg, {k: v.to(torch.bfloat16) for k, v in t.items()}
