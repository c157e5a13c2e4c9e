"""Model designs that name themselves with an ``architecture`` key in ``config.json`` and bring their own configuration keys and
tensor names: ``name -> module`` with ``config_from_dict(d, name, dtype, shapes)`` and ``load_tensors(cfg, tensors, rollout_weights)``
(``shapes``: tensor name -> shape of the checkpoint, for sizes that ``config.json`` leaves out).
Checkpoints without the key are read as Hugging Face layouts (:mod:`relax_b200.checkpoint.hf`)."""
from __future__ import annotations

from . import ketolorn, talizen, zoguzen, zupupel

ARCHITECTURES = {m.ARCHITECTURE: m for m in (talizen, ketolorn, zupupel, zoguzen)}


def architecture_of(config_json: dict):
    """The registered module of a ``config.json``, None for a Hugging Face layout."""
    name = config_json.get("architecture")
    if name is None:
        return None
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name]
