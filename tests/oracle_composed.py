"""Plain float64 statements of the layers of composed stacks, written from their equations, one function per mechanism, and
small random models to run them on.  Nothing here is shared with the engine."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def norm_in_groups(x, w, groups, eps):
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * w


def forget_gate(raw, bias, lower):
    return lower + (1 - lower) / (1 + torch.exp(-(raw + bias)))


def hgrn2_token(state, gate, q, v):
    """state [heads, dim, vdim], gate and q [heads, dim], v [heads, vdim] -> (new state, read-out [heads, vdim])"""
    new = torch.empty_like(state)
    for h in range(state.shape[0]):
        new[h] = torch.diag(gate[h]) @ state[h] + torch.outer(1 - gate[h], v[h])
    return new, torch.stack([new[h].T @ q[h] for h in range(state.shape[0])])


def silu(x):
    return x / (1 + torch.exp(-x))


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def hgrn2_mixer(h, w, heads, dim, vdim, eps):
    T = h.shape[0]
    q = silu(h @ w["q"].T).view(T, heads, dim)
    g = forget_gate(h @ w["f"].T, w["f.b"], w["lower"]).view(T, heads, dim)
    v = (h @ w["v"].T).view(T, heads, vdim)
    S = torch.zeros(heads, dim, vdim, dtype=F64)
    out = []
    for t in range(T):
        S, o = hgrn2_token(S, g[t], q[t], v[t])
        out.append((rms(o, eps) * w["norm"]).reshape(-1))
    return torch.stack(out) @ w["o"].T


def latent_mixer(h, w, heads, dim, vdim, scale, eps):
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, heads, dim)
    c = rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    k, v = (c @ w["uk"].T).view(T, heads, dim), (c @ w["uv"].T).view(T, heads, vdim)
    gate = 1 / (1 + torch.exp(-(h @ w["g"].T)))
    out = torch.zeros(T, heads, vdim, dtype=F64)
    for i in range(T):
        for n in range(heads):
            s = (k[: i + 1, n] @ q[i, n]) * scale
            p = torch.exp(s - s.max())
            out[i, n] = gate[i, n] * ((p / p.sum()) @ v[: i + 1, n])
    return out.reshape(T, -1) @ w["o"].T


def feed_forward(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def model(cfg, tensors, tokens):
    """Logits ``[T, vocab]`` of a token list."""
    w = {k: v.to(F64) for k, v in tensors.items()}
    sub = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        if layer["type"] == "hgrn2":
            y = hgrn2_mixer(x, sub(f"l{i}.mix."), m["heads"], m["dim"], m["vdim"], eps)
        else:
            y = latent_mixer(x, sub(f"l{i}.mix."), m["heads"], m["dim"], m["vdim"], m["scale"], eps)
        x = x + norm_in_groups(y, w[f"l{i}.norm1"], groups, eps)
        if layer["mlp"] is not None:
            x = x + norm_in_groups(feed_forward(x, sub(f"l{i}.mlp.")), w[f"l{i}.norm2"], groups, eps)
    return norm_in_groups(x, w["final.norm"], groups, eps) @ w["head"].T


# ---------------------------------------------------------------------------------------------------- random models


def rec(heads, dim, vdim, ff=0):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def att(heads, dim, vdim, rank, scale, ff=0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


CONFIGS = {
    # every padding rule at once: nothing is a multiple of anything
    "odd": {"width": 90, "vocab": 131, "norm": {"eps": 3e-5, "groups": 3},
            "layers": [att(3, 20, 12, 36, 0.31, 50), rec(5, 12, 7), rec(1, 33, 18, 70), att(2, 9, 30, 100, 0.4), rec(2, 8, 8, 24)]},
    "even": {"width": 128, "vocab": 256, "norm": {"eps": 1e-4, "groups": 1},
              "layers": [rec(2, 64, 64, 192), att(4, 32, 32, 64, 0.2, 192), att(16, 16, 48, 192, 0.25, 64), rec(4, 32, 32)]},
    # sizes that often coincide differ; one head; one group per eight features
    "single": {"width": 64, "vocab": 65, "norm": {"eps": 1e-6, "groups": 8}, "layers": [rec(1, 16, 40), att(1, 24, 8, 16, 0.7, 8)]},
    "wide": {"width": 256, "vocab": 320, "norm": {"eps": 1e-5, "groups": 2},
             "layers": [rec(2, 128, 96, 320), att(40, 16, 16, 320, 0.3, 128), rec(3, 96, 128), att(70, 8, 8, 128, 0.5)]},
}


def random_model(cfg, seed=0, sharp=1.0):
    """bf16-representable random tensors.  ``sharp`` scales the queries of the attention layers: large values make single
    keys dominate, so that a wrong or missing key shows."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    n = lambda *s, std=1.0: torch.randn(*s, generator=g) * std
    t = {"embed": n(V, W), "head": n(V, W, std=W ** -0.5), "final.norm": 1 + n(W, std=0.2)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        qd, vd = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        t[f"l{i}.norm1"] = 0.6 + n(W, std=0.2)
        t[p + "o"] = n(W, vd, std=vd ** -0.5)
        if layer["type"] == "hgrn2":
            t.update({p + "q": n(qd, W, std=W ** -0.5), p + "f": n(qd, W, std=2 * W ** -0.5), p + "f.b": 1 + n(qd), p + "v": n(vd, W, std=W ** -0.5),
                      p + "lower": torch.rand(qd, generator=g) ** 2 * 0.98, p + "norm": 1 + n(m["vdim"], std=0.2)})
            t[p + "lower"][::3] = 0.0
        else:
            R = m["kv_rank"]
            t.update({p + "q": n(qd, W, std=sharp * W ** -0.5), p + "dkv": n(R, W, std=W ** -0.5), p + "dkv.norm": 1 + n(R, std=0.2),
                      p + "uk": n(qd, R, std=R ** -0.5), p + "uv": n(vd, R, std=R ** -0.5), p + "g": n(m["heads"], W, std=W ** -0.5)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            t[f"l{i}.norm2"] = 0.6 + n(W, std=0.2)
            t.update({f"l{i}.mlp.gate": n(ff, W, std=W ** -0.5), f"l{i}.mlp.up": n(ff, W, std=W ** -0.5), f"l{i}.mlp.down": n(W, ff, std=ff ** -0.5)})
    return {k: v.to(torch.bfloat16) for k, v in t.items()}


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def distances(got, want):
    """Per position the root-mean-square difference of logits (means removed), in units of their spread."""
    d = got.to(F64).cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return (d ** 2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()


def distance(got, want):
    return float(distances(got, want).max())
