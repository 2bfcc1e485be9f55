"""Helpers of the model families that are described by a `config.json` and served from a checkpoint folder."""
from typing import Any, Dict, Mapping, Tuple

import torch

__all__ = ["take", "check_tensors"]


def take(d: Mapping[str, Any], where: str, required: Tuple[str, ...], optional: Tuple[str, ...] = ()) -> Dict[str, Any]:
    """The entries of a configuration object; an entry the design does not have is an error, not something to ignore (unless
    it is there only to say that something is absent)."""
    unknown = {k for k, v in d.items() if v is not None and v is not False} - set(required) - set(optional)
    missing = set(required) - set(d)
    if unknown or missing:
        raise ValueError(f"{where}: unknown entries {sorted(unknown)}, missing entries {sorted(missing)}")
    return {k: d.get(k) for k in (*required, *optional)}


def check_tensors(ckpt: Mapping[str, torch.Tensor], want: Mapping[str, Tuple[int, ...]]) -> None:
    """A checkpoint must hold exactly the tensors `want` (name -> shape)."""
    missing, extra = sorted(set(want) - set(ckpt)), sorted(set(ckpt) - set(want))
    if missing or extra:
        raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:8]}, unexpected {extra[:8]}")
    for k, shape in want.items():
        if tuple(ckpt[k].shape) != tuple(shape):
            raise ValueError(f"checkpoint tensor {k!r} has shape {tuple(ckpt[k].shape)}, expected {tuple(shape)}")
