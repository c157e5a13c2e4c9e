"""What the readers of self-describing designs share (:mod:`relax_b200.models.architectures`): strict checks of a checkpoint's
names and shapes, and writing a model folder."""
from __future__ import annotations

import json
import os


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def check_tensors(want: dict, tensors: dict) -> None:
    """Names and shapes must match exactly."""
    extra, missing = sorted(set(tensors) - set(want)), sorted(set(want) - set(tensors))
    bad = [f"{k}: {tuple(tensors[k].shape)} instead of {want[k]}" for k in want if k in tensors and tuple(tensors[k].shape) != want[k]]
    if extra or missing or bad:
        raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:8]}, unknown {extra[:8]}, shapes {bad[:8]}")


def put(dst, src) -> None:
    """Copy ``src`` into the leading corner of ``dst`` (what lies behind it is padding and stays as it is)."""
    dst[tuple(slice(0, n) for n in src.shape)].copy_(src)


def save_folder(directory: str, config: dict, tensors: dict) -> None:
    from safetensors.torch import save_file

    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(directory, "model.safetensors"))
