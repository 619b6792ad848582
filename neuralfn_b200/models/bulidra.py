"""Bulidra: a decoder whose attention and feed-forward read one norm in parallel, with short causal convolutions on q, k and v, linear
distance biases instead of rotation, a position-dependent query temperature, sliding windows, a sigmoid output gate, layers that reuse
an earlier layer's keys and values, and a per-layer token input after the feed-forward.

``BulidraConfig.from_dict`` reads the model's ``config.json``, ``pack_tensors`` turns its tensors into the fused, padded ones of the
layer-list engine (``serving.engine.LayeredEngineConfig``), ``engine_config`` describes the layers to it. All sizes and constants come
from the configuration; every layer has its own.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

import torch

from ..serving.engine import LayeredEngineConfig, LayerSpec

__all__ = ["BulidraConfig", "BulidraError", "engine_config", "expected_shapes", "pack_tensors", "random_tensors"]

_ALIBI = 8.0     # slope of head h (from 0): 2^(-8 (h + 1) / heads)


class BulidraError(ValueError):
    pass


def _need(d: Mapping, key: str, where: str):
    if key not in d:
        raise BulidraError(f"{where}: {key} is missing")
    return d[key]


def _int(v, where: str, low: int = 1) -> int:
    if isinstance(v, bool) or int(v) != v or int(v) < low:
        raise BulidraError(f"{where}: expected an integer >= {low}, got {v!r}")
    return int(v)


def _known(d: Mapping, keys: set[str], where: str) -> None:
    extra = set(d) - keys
    if extra:
        raise BulidraError(f"{where}: unknown settings {sorted(extra)}")


@dataclass(frozen=True)
class BulidraLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    window: int = 0
    q_temp_coef: float = 0.0
    q_temp_every: int = 0
    kv_from: int | None = None
    ff: int = 0


@dataclass(frozen=True)
class BulidraConfig:
    vocab: int
    width: int
    embed_scale: float
    norm_eps: float
    side_dim: int = 0
    layers: tuple[BulidraLayer, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "BulidraConfig":
        layers = []
        for i, entry in enumerate(_need(raw, "layers", "config")):
            where = f"layer {i}"
            if _need(entry, "type", where) != "attention":
                raise BulidraError(f"{where}: unknown layer type {entry['type']!r}")
            m, mlp = _need(entry, "mixer", where), entry.get("mlp")
            _known(m, {"heads", "kv_heads", "dim", "vdim", "conv", "scale", "mask", "q_temp", "kv_from"}, where)
            heads, kv_heads = _int(_need(m, "heads", where), where), _int(_need(m, "kv_heads", where), where)
            if heads % kv_heads:
                raise BulidraError(f"{where}: {heads} query heads do not divide into {kv_heads} key / value heads")
            mask, temp, kv_from = m.get("mask"), m.get("q_temp"), m.get("kv_from")
            if mask is not None:
                _known(mask, {"size"}, where)
            if temp is not None:
                _known(temp, {"coef", "every"}, where)
            if mlp is not None and _need(mlp, "kind", where) != "dense":
                raise BulidraError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
            if kv_from is not None:
                kv_from = _int(kv_from, where, 0)
                if kv_from >= i or layers[kv_from].kv_from is not None:
                    raise BulidraError(f"{where}: kv_from must name an earlier layer that has keys and values of its own")
            layers.append(BulidraLayer(
                heads, kv_heads, _int(_need(m, "dim", where), where), _int(_need(m, "vdim", where), where), _int(m.get("conv") or 0, where, 0),
                float(_need(m, "scale", where)), _int(_need(mask, "size", where), where) if mask is not None else 0,
                float(_need(temp, "coef", where)) if temp is not None else 0.0, _int(_need(temp, "every", where), where) if temp is not None else 0,
                kv_from, _int(_need(mlp, "ff", where), where) if mlp is not None else 0))
        if not layers:
            raise BulidraError("config: no layers")
        side = raw.get("token_side")
        return cls(_int(_need(raw, "vocab", "config"), "vocab"), _int(_need(raw, "width", "config"), "width"),
                   float(_need(_need(raw, "embedding", "config"), "scale", "embedding")), float(_need(_need(raw, "norm", "config"), "eps", "norm")),
                   _int(_need(side, "dim", "token_side"), "token_side") if side else 0, tuple(layers))

    def to_dict(self) -> dict:
        def layer(y: BulidraLayer) -> dict:
            m: dict[str, Any] = {"conv": y.conv, "dim": y.dim, "heads": y.heads, "kv_heads": y.kv_heads, "scale": y.scale, "vdim": y.vdim}
            if y.window:
                m["mask"] = {"size": y.window}
            if y.q_temp_every:
                m["q_temp"] = {"coef": y.q_temp_coef, "every": y.q_temp_every}
            if y.kv_from is not None:
                m["kv_from"] = y.kv_from
            return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": y.ff} if y.ff else None}

        out: dict[str, Any] = {"architecture": "Bulidra", "embedding": {"scale": self.embed_scale}, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                               "width": self.width, "layers": [layer(y) for y in self.layers]}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out


def expected_shapes(cfg: BulidraConfig) -> dict[str, tuple[int, ...]]:
    """Tensor names and shapes of a model of this configuration."""
    w, out = cfg.width, {"embed": (cfg.vocab, cfg.width), "final.norm": (cfg.width,)}
    if cfg.side_dim:
        out["side.embed"] = (cfg.vocab, len(cfg.layers) * cfg.side_dim)
    for i, y in enumerate(cfg.layers):
        p = f"l{i}."
        out[p + "norm1"] = (w,)
        rows = {"q": y.heads * y.dim}
        if y.kv_from is None:
            rows.update(k=y.kv_heads * y.dim, v=y.kv_heads * y.vdim)
        for n, r in rows.items():
            out[p + f"mix.{n}"] = (r, w)
            if y.conv:
                out[p + f"mix.{n}.conv"] = (r, y.conv)
        out[p + "mix.g"], out[p + "mix.o"] = (y.heads * y.vdim, w), (w, y.heads * y.vdim)
        if y.ff:
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = (y.ff, w), (y.ff, w), (w, y.ff)
        if cfg.side_dim:
            out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (cfg.side_dim, w), (w, cfg.side_dim), (w,)
    return out


def engine_config(cfg: BulidraConfig, **kw) -> LayeredEngineConfig:
    """``kw``: serving limits (``max_seq``, ``max_batch``, ``kv_tokens``, ``dtype``, ...)."""
    specs = tuple(LayerSpec(heads=y.heads, kv_heads=y.kv_heads, dim=y.dim, vdim=y.vdim, conv_taps=y.conv, window=y.window,
                            kv_from=-1 if y.kv_from is None else y.kv_from, scale=y.scale, alibi=_ALIBI, q_temp_coef=y.q_temp_coef,
                            q_temp_every=y.q_temp_every, out_gate=1, ff=y.ff, ff_act="relu") for y in cfg.layers)
    return LayeredEngineConfig(layers=specs, width=cfg.width, vocab=cfg.vocab, side_dim=cfg.side_dim, embed_scale=cfg.embed_scale,
                               norm_eps=cfg.norm_eps, **kw)


def _up(v: int, m: int = 16) -> int:
    return (v + m - 1) // m * m


def _pad_rows(t: torch.Tensor, groups: int, to: int) -> torch.Tensor:
    """[groups * n, ...] -> [groups * to, ...]: zero rows after each group."""
    n = t.shape[0] // groups
    if n == to:
        return t
    out = t.new_zeros(groups, to, *t.shape[1:])
    out[:, :n] = t.reshape(groups, n, *t.shape[1:])
    return out.reshape(groups * to, *t.shape[1:])


def pack_tensors(cfg: BulidraConfig, tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The model's tensors under the engine's names: one input product [q | k | v | g | gate | up] and one output product [o | down] per
    layer, heads and widths padded with zeros to multiples of 16."""
    want = expected_shapes(cfg)
    missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
    if missing or extra:
        raise BulidraError(f"tensors do not fit the configuration (missing {missing[:4]}, unexpected {extra[:4]})")
    for n, shape in want.items():
        if tuple(tensors[n].shape) != shape:
            raise BulidraError(f"{n}: shape {tuple(tensors[n].shape)} instead of {shape}")
    T = {n: tensors[n].to(torch.bfloat16) for n in want}
    wp = _up(cfg.width)

    def cols(t: torch.Tensor) -> torch.Tensor:                   # [rows, width] -> [rows, wp]
        return _pad_rows(t.T, 1, wp).T if t.shape[1] != wp else t

    def vec(n: str) -> torch.Tensor:
        return _pad_rows(T[n], 1, wp)

    out = {"embed": _pad_rows(cols(T["embed"]), 1, _up(cfg.vocab)), "final_norm": vec("final.norm")}
    sp = _up(cfg.side_dim) if cfg.side_dim else 0
    if sp:
        out["side_embed"] = _pad_rows(T["side.embed"].T, len(cfg.layers), sp).T.contiguous()
    for i, y in enumerate(cfg.layers):
        p, q = f"l{i}.", f"layers.{i}."
        dp, vp, fp = _up(y.dim), _up(y.vdim), _up(y.ff) if y.ff else 0
        heads = [("q", y.heads, dp)] + ([("k", y.kv_heads, dp), ("v", y.kv_heads, vp)] if y.kv_from is None else [])
        rows = [_pad_rows(cols(T[p + f"mix.{n}"]), g, to) for n, g, to in heads] + [_pad_rows(cols(T[p + "mix.g"]), y.heads, vp)]
        o = [_pad_rows(T[p + "mix.o"].T, y.heads, vp)]           # [heads * vp, width]
        if y.ff:
            rows += [_pad_rows(cols(T[p + "mlp.gate"]), 1, fp), _pad_rows(cols(T[p + "mlp.up"]), 1, fp)]
            o.append(_pad_rows(T[p + "mlp.down"].T, 1, fp))
        out[q + "norm1"] = vec(p + "norm1")
        out[q + "w_in"] = torch.cat(rows)
        if y.conv:
            out[q + "conv"] = torch.cat([_pad_rows(T[p + f"mix.{n}.conv"], g, to) for n, g, to in heads]).T.contiguous()
        out[q + "w_out"] = _pad_rows(torch.cat(o).T.contiguous(), 1, wp)
        if sp:
            out[q + "side_gate"] = _pad_rows(cols(T[p + "side.gate"]), 1, sp)
            out[q + "side_proj"] = _pad_rows(_pad_rows(T[p + "side.proj"].T, 1, sp).T.contiguous(), 1, wp)
            out[q + "side_norm"] = vec(p + "side.norm")
    return out


def random_tensors(cfg: BulidraConfig, seed: int = 0, device: str = "cpu") -> dict[str, torch.Tensor]:
    """Random bf16 weights with activations of order one (tests, throughput runs)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for n, shape in expected_shapes(cfg).items():
        if n.endswith("norm") or n.endswith("norm1"):
            t = 1 + 0.1 * torch.randn(shape, generator=g, device=device)
        else:
            t = torch.randn(shape, generator=g, device=device) / (1.0 if n == "side.embed" else shape[-1] ** 0.5)
        out[n] = t.to(torch.bfloat16)
    return out
