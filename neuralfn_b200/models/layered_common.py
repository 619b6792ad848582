"""Shared by the readers of layer-list models (``bulidra``, ``murilorn``): strict access to configuration dictionaries, padding of weight
rows, checks of tensor names and shapes."""
from __future__ import annotations

from typing import Any, Mapping

import torch

__all__ = ["ModelConfigError", "check_tensors", "known", "need", "pad_cols", "pad_rows", "positive_int", "up"]


class ModelConfigError(ValueError):
    pass


def need(d: Mapping, key: str, where: str) -> Any:
    if key not in d:
        raise ModelConfigError(f"{where}: {key} is missing")
    return d[key]


def positive_int(v: Any, where: str, low: int = 1) -> int:
    if isinstance(v, bool) or int(v) != v or int(v) < low:
        raise ModelConfigError(f"{where}: expected an integer >= {low}, got {v!r}")
    return int(v)


def known(d: Mapping, keys: set[str], where: str) -> None:
    extra = {k for k, v in d.items() if v is not None} - keys
    if extra:
        raise ModelConfigError(f"{where}: unknown settings {sorted(extra)}")


def up(v: int, m: int = 16) -> int:
    return (v + m - 1) // m * m


def pad_rows(t: torch.Tensor, groups: int, to: int) -> torch.Tensor:
    """[groups * n, ...] -> [groups * to, ...]: zero rows after each group."""
    n = t.shape[0] // groups
    if n == to:
        return t
    out = t.new_zeros(groups, to, *t.shape[1:])
    out[:, :n] = t.reshape(groups, n, *t.shape[1:])
    return out.reshape(groups * to, *t.shape[1:])


def pad_cols(t: torch.Tensor, groups: int, to: int) -> torch.Tensor:
    """The same on the columns of a matrix."""
    return t if t.shape[1] // groups == to else pad_rows(t.T, groups, to).T.contiguous()


def check_tensors(want: Mapping[str, tuple[int, ...]], tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The tensors named in ``want`` in bf16; anything missing, unexpected or of another shape is an error."""
    missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
    if missing or extra:
        raise ModelConfigError(f"tensors do not fit the configuration (missing {missing[:4]}, unexpected {extra[:4]})")
    for n, shape in want.items():
        if tuple(tensors[n].shape) != shape:
            raise ModelConfigError(f"{n}: shape {tuple(tensors[n].shape)} instead of {shape}")
    return {n: tensors[n].to(torch.bfloat16) for n in want}
