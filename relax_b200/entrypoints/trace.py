"""Trace replay: given token ids through the rollout engine's step function, logits to files (``bin/trace_run``)."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64           # tokens per page of the engine's block manager
MAX_LIVE = 4        # requests that may be live at once


def build_engine(model_dir: str, dtype, max_tokens: int, device="cuda"):
    """An engine whose page pool holds ``max_tokens`` tokens and whose state pool holds :data:`MAX_LIVE` sequences."""
    from ..checkpoint.hf import config_from_hf, load_hf_into_rollout
    from ..rollout.engine import RolloutEngine

    cfg = config_from_hf(model_dir)
    if not cfg.is_composed:
        raise SystemExit(f"trace replay drives composed stacks; {model_dir} holds a {cfg.name} of another kind")
    eng = RolloutEngine(cfg, device=device, dtype=dtype, num_kv_blocks=(max_tokens + PAGE - 1) // PAGE, block_size=PAGE,
                        state_slots=MAX_LIVE, use_cuda_graph=False, memory_saver=False)
    load_hf_into_rollout(model_dir, cfg, eng.weights)
    return eng


def replay(eng, lines, out_dir: str, report):
    """Run the steps of ``lines``; ``report(step)`` is called after each."""
    import numpy as np

    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if not e["tokens"]:
                continue
            if e["id"] not in live:
                live[e["id"]] = eng.open_sequence()
            entries.append((live[e["id"]], e["tokens"], e.get("want", [])))
        if entries:
            z = eng.feed(entries)
            if z is not None:
                path = os.path.join(out_dir, f"{step['step']}.f32")
                z.float().cpu().numpy().astype(np.dtype("<f4")).tofile(path)
        for i in step.get("end", []):
            if i in live:
                eng.close_sequence(live.pop(i))
        report(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens the live requests hold (each rounded up to 64)")
    a = ap.parse_args(argv)
    import torch

    if not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    from ..ops import build, cuda as C

    C._load(build.ensure_serving())
    eng = build_engine(a.model, getattr(torch, a.dtype), a.max_tokens)

    def report(step):
        C.check_error_flag()
        print(f"done {step}", flush=True)

    replay(eng, sys.stdin, a.out, report)
    return 0
