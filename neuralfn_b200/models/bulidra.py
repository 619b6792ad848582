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
from .layered_common import ModelConfigError, check_tensors, known, need, pad_cols, pad_rows, positive_int, up

__all__ = ["BulidraConfig", "BulidraError", "engine_config", "expected_shapes", "pack_tensors", "random_tensors"]

_ALIBI = 8.0     # slope of head h (from 0): 2^(-8 (h + 1) / heads)


BulidraError = ModelConfigError


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
        for i, entry in enumerate(need(raw, "layers", "config")):
            where = f"layer {i}"
            if need(entry, "type", where) != "attention":
                raise BulidraError(f"{where}: unknown layer type {entry['type']!r}")
            m, mlp = need(entry, "mixer", where), entry.get("mlp")
            known(m, {"heads", "kv_heads", "dim", "vdim", "conv", "scale", "mask", "q_temp", "kv_from"}, where)
            heads, kv_heads = positive_int(need(m, "heads", where), where), positive_int(need(m, "kv_heads", where), where)
            if heads % kv_heads:
                raise BulidraError(f"{where}: {heads} query heads do not divide into {kv_heads} key / value heads")
            mask, temp, kv_from = m.get("mask"), m.get("q_temp"), m.get("kv_from")
            if mask is not None:
                known(mask, {"size"}, where)
            if temp is not None:
                known(temp, {"coef", "every"}, where)
            if mlp is not None and need(mlp, "kind", where) != "dense":
                raise BulidraError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
            if kv_from is not None:
                kv_from = positive_int(kv_from, where, 0)
                if kv_from >= i or layers[kv_from].kv_from is not None:
                    raise BulidraError(f"{where}: kv_from must name an earlier layer that has keys and values of its own")
            layers.append(BulidraLayer(
                heads, kv_heads, positive_int(need(m, "dim", where), where), positive_int(need(m, "vdim", where), where), positive_int(m.get("conv") or 0, where, 0),
                float(need(m, "scale", where)), positive_int(need(mask, "size", where), where) if mask is not None else 0,
                float(need(temp, "coef", where)) if temp is not None else 0.0, positive_int(need(temp, "every", where), where) if temp is not None else 0,
                kv_from, positive_int(need(mlp, "ff", where), where) if mlp is not None else 0))
        if not layers:
            raise BulidraError("config: no layers")
        side = raw.get("token_side")
        return cls(positive_int(need(raw, "vocab", "config"), "vocab"), positive_int(need(raw, "width", "config"), "width"),
                   float(need(need(raw, "embedding", "config"), "scale", "embedding")), float(need(need(raw, "norm", "config"), "eps", "norm")),
                   positive_int(need(side, "dim", "token_side"), "token_side") if side else 0, tuple(layers))

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


def pack_tensors(cfg: BulidraConfig, tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The model's tensors under the engine's names: one input product [q | k | v | g | gate | up] and one output product [o | down] per
    layer, heads and widths padded with zeros to multiples of 16."""
    T = check_tensors(expected_shapes(cfg), tensors)
    wp = up(cfg.width)

    def cols(t: torch.Tensor) -> torch.Tensor:                   # [rows, width] -> [rows, wp]
        return pad_cols(t, 1, wp)

    def vec(n: str) -> torch.Tensor:
        return pad_rows(T[n], 1, wp)

    out = {"embed": pad_rows(cols(T["embed"]), 1, up(cfg.vocab)), "final_norm": vec("final.norm")}
    sp = up(cfg.side_dim) if cfg.side_dim else 0
    if sp:
        out["side_embed"] = pad_rows(T["side.embed"].T, len(cfg.layers), sp).T.contiguous()
    for i, y in enumerate(cfg.layers):
        p, q = f"l{i}.", f"layers.{i}."
        dp, vp, fp = up(y.dim), up(y.vdim), up(y.ff) if y.ff else 0
        heads = [("q", y.heads, dp)] + ([("k", y.kv_heads, dp), ("v", y.kv_heads, vp)] if y.kv_from is None else [])
        rows = [pad_rows(cols(T[p + f"mix.{n}"]), g, to) for n, g, to in heads] + [pad_rows(cols(T[p + "mix.g"]), y.heads, vp)]
        o = [pad_rows(T[p + "mix.o"].T, y.heads, vp)]           # [heads * vp, width]
        if y.ff:
            rows += [pad_rows(cols(T[p + "mlp.gate"]), 1, fp), pad_rows(cols(T[p + "mlp.up"]), 1, fp)]
            o.append(pad_rows(T[p + "mlp.down"].T, 1, fp))
        out[q + "norm1"] = vec(p + "norm1")
        out[q + "w_in"] = torch.cat(rows)
        if y.conv:
            out[q + "conv"] = torch.cat([pad_rows(T[p + f"mix.{n}.conv"], g, to) for n, g, to in heads]).T.contiguous()
        out[q + "w_out"] = pad_rows(torch.cat(o).T.contiguous(), 1, wp)
        if sp:
            out[q + "side_gate"] = pad_rows(cols(T[p + "side.gate"]), 1, sp)
            out[q + "side_proj"] = pad_rows(pad_rows(T[p + "side.proj"].T, 1, sp).T.contiguous(), 1, wp)
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
