"""Plain float64 statements of the layers of Zoguzen stacks, written from their equations, one function per mechanism, and small
random models to run them on.  Nothing here is shared with the engine."""
import copy
import math

import torch

F64 = torch.float64


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def centred(x, w, eps):
    """Layer norm without a bias: deviations from the mean over the root of their mean square."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def shifted(h, mu):
    """Every row moves by ``mu`` towards the row before it (the first one towards zero)."""
    out = h.clone()
    for t in range(h.shape[0]):
        before = h[t - 1] if t else torch.zeros_like(h[0])
        out[t] = h[t] + (before - h[t]) * mu
    return out


def convolved(u, w):
    """u [T, channels] under causal taps w [channels, n], the last tap on the row itself."""
    T, n = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(n):
            if t - n + 1 + j >= 0:
                y[t] += w[:, j] * u[t - n + 1 + j]
    return y


def frequencies(rot):
    """Of every pair; long wavelengths are stretched, those between two bounds partly."""
    s, out = rot.get("scaling"), []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        if s:
            length = 2 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                part = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1 - part) * f / s["factor"] + part * f
        out.append(f)
    return out


def turned(x, positions, freqs):
    """x [T, heads, d]: features 2 i and 2 i + 1 turn together."""
    y = x.clone()
    for t, p in enumerate(positions):
        for i, f in enumerate(freqs):
            c, s, u, v = math.cos(p * f), math.sin(p * f), x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i], y[t, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def sees_window(size, keep):
    return lambda i, j: j <= i and (i - j < size or j < keep)


def sees_chunk(size):
    return lambda i, j: j <= i and i // size == j // size


def weights(q, k, first, scale, sees, softcap=None, one=False):
    """Attention weights [n, H, L] of q [n, H, d] at positions first .. over keys k [L, G, d]; ``one``: one more in the denominator."""
    n, H, _ = q.shape
    L, rep = k.shape[0], H // k.shape[1]
    out = torch.zeros(n, H, L, dtype=F64)
    for i in range(n):
        js = [j for j in range(L) if sees(first + i, j)]
        for h in range(H):
            s = torch.stack([k[j, h // rep] @ q[i, h] for j in js]) * scale
            if softcap is not None:
                s = softcap * torch.tanh(s / softcap)
            m = max(float(s.max()), 0.0)
            e = torch.exp(s - m)
            out[i, h, js] = e / (e.sum() + (math.exp(-m) if one else 0.0))
    return out


def talked(p, T):
    """The heads' weights [n, H, L] mixed: row h of T weighs the heads for head h."""
    out = torch.zeros_like(p)
    for h in range(p.shape[1]):
        for g in range(p.shape[1]):
            out[:, h] += T[h, g] * p[:, g]
    return out


def applied(p, v):
    """Weights [n, H, L] on the values v [L, G, dv] of every head's own group."""
    rep = p.shape[1] // v.shape[1]
    return torch.stack([p[:, h] @ v[:, h // rep] for h in range(p.shape[1])], 1)


def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def mingru(z, u, state=None):
    """Gates z and candidates' inputs u [T, width] -> states of every row."""
    S, out = torch.zeros_like(z[0]) if state is None else state, []
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * candidate(u[t])
        out.append(S)
    return torch.stack(out)


def linear_attention(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, d], v [T, H, dv]: states decay row by row.  Returns (read-outs [T, H, dv], state [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] = torch.diag(alpha[t, h]) @ S[h] + torch.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def routed(h, w, mlp):
    """(output, gap of the closest choice per row)"""
    top, n = mlp["router"]["top"], mlp["router"]["experts"]
    out, gaps, z = torch.zeros_like(h), [], h @ w["router"].T
    for t in range(h.shape[0]):
        order = sorted(range(n), key=lambda e: -z[t, e].item())
        gaps.append((z[t, order[top - 1]] - z[t, order[top]]).item() if top < n else math.inf)
        e = torch.exp(z[t, order[:top]] - z[t, order[0]])
        for p, k in zip(e / e.sum(), order):
            out[t] += p * expert(h[t], w[f"e{k}.gate"], w[f"e{k}.up"], w[f"e{k}.down"])
    return out, torch.tensor(gaps)


def mix_attention(x, t, m, eps, cached, i):
    T, H, G = x.shape[0], m["heads"], m["kv_heads"]
    q = rms(convolved(x @ t["q"].T + t["q.b"], t["q.conv"]).view(T, H, -1), t["q.norm"], eps)
    if "kv_from" in m:
        k, v = cached[m["kv_from"]]
    else:
        k = rms(convolved(x @ t["k"].T + t["k.b"], t["k.conv"]).view(T, G, -1), t["k.norm"], eps)
        v = convolved(x @ t["v"].T + t["v.b"], t["v.conv"]).view(T, G, -1)
        cached[i] = (k, v)
    p = weights(q, k, 0, m["scale"], sees_chunk(m["mask"]["size"]), m["softcap"], True)
    return applied(talked(p, t["talk"]), v).reshape(T, -1) @ t["o"].T


def mix_left(x, t, m):
    T, H, G, r = x.shape[0], m["heads"], m["kv_heads"], m["rot"]
    f = frequencies(r)
    q = turned(convolved(x @ t["q"].T, t["q.conv"]).view(T, H, -1), range(T), f)
    k = turned(convolved(x @ t["k"].T, t["k.conv"]).view(T, G, -1), range(T), f)
    v = convolved(x @ t["v"].T, t["v.conv"]).view(T, G, -1)
    p = weights(q, k, 0, m["scale"], sees_window(m["mask"]["size"], m["mask"]["keep_first"]))
    return (applied(p, v).reshape(T, -1) * sigmoid(x @ t["g"].T)) @ t["o"].T


def mix_right(x, t, m, eps):
    T, H = x.shape[0], m["heads"]
    heads = lambda y: y.view(T, H, -1)
    alpha = sigmoid((x @ t["a1"].T) @ t["a2"].T + t["a2.b"]) ** (1 / m["tau"])
    o, _ = linear_attention(heads(x @ t["q"].T) * m["dim"] ** -0.5, heads(x @ t["k"].T), heads(x @ t["v"].T), heads(alpha))
    return (rms(o, t["norm"], eps).reshape(T, -1) * silu(x @ t["g"].T)) @ t["o"].T


def mix_mingru(x, t):
    S = mingru(sigmoid(x @ t["z"].T + t["z.b"]), x @ t["x"].T + t["x.b"])
    return (S * silu(x @ t["g"].T)) @ t["o"].T


def run(cfg, tensors, tokens):
    """(logits [T, vocab], gap of the closest expert choice of every row, streams after the layers)"""
    w = {k: v.to(F64) for k, v in tensors.items()}
    part = lambda d, p: {k[len(p):]: v for k, v in d.items() if k.startswith(p)}
    eps, T, S = cfg["norm"]["eps"], len(tokens), cfg["token_side"]["dim"]
    ids = torch.tensor(tokens)
    x = w["embed"][ids]
    gaps, cached, streams = torch.full((T,), math.inf, dtype=F64), {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, t, m = f"l{i}.", part(w, f"l{i}.mix."), layer["mixer"]
        h = shifted(centred(x, w[p + "norm1"], eps), w[p + "shift"])
        if layer["type"] == "attention":
            y = mix_attention(h, t, m, eps, cached, i)
        elif layer["type"] == "mingru":
            y = mix_mingru(h, t)
        else:
            left, right = part(t, "left."), part(t, "right.")
            y = 0.5 * (rms(mix_left(h, left, m["left"]), left["out"], eps) + rms(mix_right(h, right, m["right"], eps), right["out"], eps))
        if layer["mlp"] is not None:
            f, gap = routed(centred(x, w[p + "norm2"], eps), part(w, p + "mlp."), layer["mlp"])
            gaps, y = torch.minimum(gaps, gap), y + f
        x = x + y
        side = gelu(x @ w[p + "side.gate"].T) * w["side.embed"][ids][:, i * S:(i + 1) * S]
        x = x + rms(side @ w[p + "side.proj"].T, w[p + "side.norm"], eps)
        streams.append(x)
    z = centred(x, w["final.norm"], eps) @ w["embed"].T
    c = cfg["logit_softcap"]
    return c * torch.tanh(z / c), gaps, streams


def model(cfg, tensors, tokens):
    return run(cfg, tensors, tokens)[0]


# ---------------------------------------------------------------------------------------------------- random models


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def att(heads, kv_heads, dim, vdim, scale, chunk, cap, conv, mlp=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}, "softcap": cap, "conv": conv}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gru(width, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, scale, window, keep, conv, rot, base, scaling=None):
    r = {"dims": rot, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window, "keep_first": keep}, "conv": conv, "rot": r}


def right(heads, dim, vdim, tau, rank):
    """(the rank is no key of a configuration: :func:`random_model` takes it out)"""
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def pair(a, b, mlp=None):
    return {"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": mlp}


def stack(width, vocab, eps, layers, side, cap):
    return {"architecture": "Zoguzen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "token_side": {"dim": side}, "logit_softcap": cap, "layers": layers}


CONFIGS = {
    # every padding rule at once: nothing is a multiple of anything; readers with chunks and caps other than their source's
    "odd": stack(74, 131, 3e-5, [att(6, 2, 18, 13, 0.31, 21, 5.0, 3, moe(7, 2, 20)), gru(37, moe(5, 1, 9)), att(6, 2, 18, 13, 0.22, 9, 3.0, 4, moe(4, 3, 33), 0),
                                 pair(left(4, 2, 10, 7, 0.5, 12, 5, 2, 6, 300.0, (3.0, 1.0, 3.0, 60.0)), right(3, 6, 5, 3.0, 3), moe(6, 3, 12)),
                                 att(5, 5, 7, 9, 0.9, 33, 2.0, 5), pair(left(3, 3, 8, 11, 0.6, 20, 2, 3, 8, 50.0), right(2, 9, 12, 5.0, 20))], 5, 7.0),
    # whole heads turn; wide groups, narrow keys beside wide values, more groups than two
    "even": stack(128, 256, 1e-4, [pair(left(8, 2, 64, 64, 0.15, 48, 16, 4, 64, 1e4, (8.0, 1.0, 4.0, 64.0)), right(4, 32, 64, 12.0, 8), moe(8, 2, 64)),
                                   att(8, 1, 64, 128, 0.2, 40, 15.0, 4, moe(6, 3, 64)), gru(192, moe(8, 2, 32)), att(16, 4, 128, 32, 0.11, 64, 25.0, 2, moe(14, 4, 128)),
                                   att(16, 4, 128, 32, 0.2, 100, 10.0, 4, None, 3), pair(left(4, 4, 128, 40, 0.1, 33, 70, 4, 32, 1e5), right(3, 64, 32, 16.0, 24))], 16, 20.0),
    # one head, one feature pair, one tap, a window of one token without kept ones, chunks of one token, all experts taken
    "single": stack(64, 65, 1e-3, [att(1, 1, 16, 40, 0.7, 1, 4.0, 1, moe(2, 2, 8)), gru(8, moe(3, 1, 8)),
                                   pair(left(1, 1, 16, 8, 0.7, 1, 0, 1, 2, 10.0), right(1, 8, 8, 1.0, 1)), att(1, 1, 16, 40, 0.5, 500, 9.0, 6, None, 0)], 1, 3.0),
    # more heads per group than the decode tile takes; heads wider than the tensor-core kernels take; a decay of odd shape
    "wide": stack(256, 320, 1e-5, [att(40, 2, 24, 16, 0.3, 17, 8.0, 4, moe(8, 3, 96)), pair(left(20, 1, 24, 16, 0.4, 19, 3, 4, 8, 1e4), right(2, 128, 96, 20.0, 40)),
                                   att(3, 1, 144, 136, 0.1, 70, 12.0, 3, moe(6, 2, 64)), gru(300, moe(9, 5, 40)),
                                   pair(left(2, 2, 144, 136, 0.1, 30, 9, 2, 96, 1e6, (2.0, 0.5, 5.0, 100.0)), right(5, 20, 28, 2.0, 6))], 40, 12.0),
}


def random_model(cfg, seed=0, sharp=1.0):
    """bf16-representable random tensors; ``sharp`` multiplies the attention scales of the configuration that comes back."""
    cfg = copy.deepcopy(cfg)
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    lin = lambda out, fan: n(out, fan, std=fan ** -0.5)
    t = {"embed": n(V, W, std=0.4), "side.embed": n(V, S * len(cfg["layers"])), "final.norm": 1 + n(W, std=0.2)}

    def attention(m, p, extras):
        m["scale"] *= sharp
        for k, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"]))[:1 if "kv_from" in m else 3]:
            t.update({p + k: lin(rows, W), p + k + ".conv": n(rows, m["conv"], std=m["conv"] ** -0.5)})
            if extras:
                t[p + k + ".b"] = n(rows, std=0.3)
                if k != "v":
                    t[p + k + ".norm"] = 1.2 + n(m["dim"], std=0.3)
        t[p + "o"] = lin(W, m["heads"] * m["vdim"])

    for i, layer in enumerate(cfg["layers"]):
        m, a, p, f, mlp = layer["mixer"], f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", layer["mlp"]
        t.update({a + "norm1": 1 + n(W, std=0.2), a + "shift": torch.rand(W, generator=g), a + "side.gate": lin(S, W) * 0.7, a + "side.proj": lin(W, S),
                  a + "side.norm": 0.5 + n(W, std=0.2)})
        if layer["type"] == "attention":
            attention(m, p, True)
            t[p + "talk"] = torch.eye(m["heads"]) + n(m["heads"], m["heads"], std=0.4)
        elif layer["type"] == "mingru":
            w = m["width"]
            t.update({p + "z": lin(w, W), p + "z.b": n(w) - 1, p + "x": lin(w, W), p + "x.b": n(w, std=0.5), p + "g": lin(w, W), p + "o": lin(W, w) * 2})
        else:
            r = m["right"]
            rank, qd, vd = r.pop("rank"), r["heads"] * r["dim"], r["heads"] * r["vdim"]
            attention(m["left"], p + "left.", False)
            q = p + "right."
            t.update({p + "left.g": lin(m["left"]["heads"] * m["left"]["vdim"], W), p + "left.out": 1 + n(W, std=0.2), q + "out": 1 + n(W, std=0.2),
                      q + "q": lin(qd, W), q + "k": lin(qd, W), q + "v": lin(vd, W), q + "g": lin(vd, W), q + "o": lin(W, vd), q + "norm": 1 + n(r["vdim"], std=0.2),
                      q + "a1": lin(rank, W), q + "a2": lin(qd, rank) * 2, q + "a2.b": n(qd) + 1})
        if mlp is None:
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        t.update({a + "norm2": 1 + n(W, std=0.2), f + "router": lin(E, W) * 1.5})
        for e in range(E):
            t.update({f"{f}e{e}.gate": lin(ff, W) * 1.5, f"{f}e{e}.up": lin(ff, W), f"{f}e{e}.down": lin(W, ff) * 2})
    return cfg, {k: v.to(torch.bfloat16) for k, v in t.items()}
