"""Helpers of the composed-stack tests: engines on random models, and feeding sequences in portions."""
import torch

import oracle_composed
import oracle_ketolorn
import oracle_zoguzen
import oracle_zupupel


def oracle(cfg):
    return {"Ketolorn": oracle_ketolorn, "Zupupel": oracle_zupupel, "Zoguzen": oracle_zoguzen}.get(cfg.get("architecture"), oracle_composed)


def engine(cfg, tensors, device="cpu", dtype=torch.float32, blocks=64, block_size=16, **kw):
    from relax_b200.models.architectures import architecture_of
    from relax_b200.rollout.engine import RolloutEngine

    full = {"architecture": "Talizen", **cfg}
    design = architecture_of(full)
    mc = design.config_from_dict(full, dtype="fp32" if dtype == torch.float32 else "bf16", shapes={k: tuple(v.shape) for k, v in tensors.items()})
    eng = RolloutEngine(mc, device=device, dtype=dtype, num_kv_blocks=blocks, block_size=block_size, memory_saver=False,
                        **{"state_slots": 4, "use_cuda_graph": False, **kw})
    design.load_tensors(mc, tensors, eng.weights)
    return eng


def cut(n, sizes):
    """Portions of a sequence of ``n`` tokens with sizes taken in turn from ``sizes``."""
    out, k = [], 0
    while n > 0:
        out.append(min(n, sizes[k % len(sizes)]))
        n -= out[-1]
        k += 1
    return out


def feed_alone(eng, toks, sizes):
    """Logits of every position, fed in portions; gives pages and slot back."""
    r, at, out = eng.open_sequence(), 0, []
    for n in cut(len(toks), sizes):
        out.append(eng.feed([(r, toks[at:at + n], list(range(n)))]).float().cpu())
        at += n
    eng.close_sequence(r)
    return torch.cat(out)


def feed_mixed(eng, seqs, plans, starts):
    """Several sequences at once: sequence ``i`` joins at step ``starts[i]`` and takes its portions ``plans[i]`` in turn
    (0 = sits a step out).  Returns every sequence's logits; pages and slots go back as sequences end."""
    live, at, k, out, step = {}, [0] * len(seqs), [0] * len(seqs), [[] for _ in seqs], 0
    while any(at[i] < len(s) for i, s in enumerate(seqs)):
        entries, owner = [], []
        for i, s in enumerate(seqs):
            if step < starts[i] or at[i] >= len(s):
                continue
            n = min(plans[i][k[i] % len(plans[i])], len(s) - at[i])
            k[i] += 1
            if n == 0:
                continue
            if i not in live:
                live[i] = eng.open_sequence()
            entries.append((live[i], s[at[i]:at[i] + n], list(range(n))))
            owner.append((i, n))
            at[i] += n
        if entries:
            z = eng.feed(entries).float().cpu()
            o = 0
            for i, n in owner:
                out[i].append(z[o:o + n])
                o += n
                if at[i] == len(seqs[i]):
                    eng.close_sequence(live.pop(i))
        step += 1
    return [torch.cat(x) for x in out]


def all_free(eng):
    assert eng.bm.num_free == eng.bm.num_blocks and eng.sm.num_free == eng.sm.n - 1      # one slot is the padding rows' own


def greedy(cfg, tensors, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(oracle(cfg).model(cfg, tensors, seq)[-1].argmax()))
    return seq[len(prompt):]
