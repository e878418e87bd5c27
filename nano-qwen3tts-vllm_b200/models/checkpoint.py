"""Filling a model's parameters from a checkpoint by a table of targets."""
from __future__ import annotations

import torch


def load_targets(targets: dict, state_dict: dict, strict: bool = True) -> set:
    """``targets``: checkpoint name -> (parameter, shard of a merged weight or None, transform of the stored tensor or None).
    Values are converted to the parameter's type (what the kernels keep in float is widened exactly); a stored tensor whose number of
    axes differs is reshaped ([heads * d, r] -> [heads, d, r]).  Returns the names seen; ``strict``: unexpected and missing tensors
    raise KeyError."""
    seen = set()
    for name, value in state_dict.items():
        if name not in targets:
            if strict:
                raise KeyError(f"unexpected tensor {name!r} in the checkpoint")
            continue
        param, shard, transform = targets[name]
        if transform is not None:
            value = transform(value)
        with torch.no_grad():
            if shard is not None:
                param.weight_loader(param, value.to(param.dtype), shard)
            else:
                if param.numel() != value.numel() or (param.dim() == value.dim() and tuple(param.shape) != tuple(value.shape)):
                    raise ValueError(f"{name}: shape {tuple(value.shape)} does not fit {tuple(param.shape)}")
                param.copy_(value.to(param.dtype).reshape(param.shape))
        seen.add(name)
    if strict:
        missing = sorted(set(targets) - seen)
        if missing:
            raise KeyError(f"missing tensors: {missing[:8]}{' ...' if len(missing) > 8 else ''}")
    return seen
