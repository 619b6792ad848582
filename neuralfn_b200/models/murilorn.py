"""Murilorn: a decoder that alternates gated-delta-rule layers (a decay per key channel, short convolutions, a gated output norm) with
sliding-window attention (kept first tokens, score soft cap, a sink in the softmax), routed experts after every mixer, several residual
streams mixed between sublayers, and a run of layers that is gone through more than once.

``MurilornConfig.from_dict`` reads the model's ``config.json`` (the inner sizes of the low-rank projections come from the tensors),
``pack_tensors`` turns its tensors into the fused, padded ones of the layer-list engine (``serving.engine.LayeredEngineConfig``),
``engine_config`` describes the layers to it, the loop unrolled. All sizes and constants come from the configuration; every layer has its
own.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

import torch

from ..serving.engine import LayeredEngineConfig, LayerSpec
from .layered_common import ModelConfigError, check_tensors, known, need, pad_cols, pad_rows, positive_int, up

__all__ = ["MurilornConfig", "MurilornLayer", "engine_config", "expected_shapes", "layer_order", "pack_tensors", "random_tensors"]


@dataclass(frozen=True)
class MurilornLayer:
    type: str                   # "channel_delta" or "attention"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int = 0               # channel_delta: taps
    rank_decay: int = 0         # channel_delta: rows of a1, g1
    rank_gate: int = 0
    scale: float = 1.0          # attention
    softcap: float = 0.0
    window: int = 0
    keep_first: int = 0
    experts: int = 0            # 0: no feed-forward
    top: int = 0
    expert_ff: int = 0


@dataclass(frozen=True)
class MurilornConfig:
    vocab: int
    width: int
    embed_scale: float
    norm_eps: float
    streams: int = 0            # 0: one plain residual
    loop: tuple[int, int, int] | None = None      # layers [start, stop) run `times` times
    logit_scale: float = 1.0
    logit_softcap: float = 0.0
    layers: tuple[MurilornLayer, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], tensors: Mapping[str, torch.Tensor] | None = None) -> "MurilornConfig":
        """``tensors``: the checkpoint, for the sizes only its shapes give; without it the entries "rank_decay" and "rank_gate" of a mixer
        (written by ``to_dict``) are read."""
        known(raw, {"architecture", "embedding", "layers", "logit_scale", "logit_softcap", "loop", "norm", "streams", "vocab", "width"}, "config")
        layers = []
        for i, entry in enumerate(need(raw, "layers", "config")):
            where = f"layer {i}"
            known(entry, {"type", "mixer", "mlp"}, where)
            kind, m = need(entry, "type", where), need(entry, "mixer", where)
            if kind not in ("channel_delta", "attention"):
                raise ModelConfigError(f"{where}: unknown layer type {kind!r}")
            heads, kv_heads = positive_int(need(m, "heads", where), where), positive_int(need(m, "kv_heads", where), where)
            if heads % kv_heads:
                raise ModelConfigError(f"{where}: {heads} heads do not divide into {kv_heads} key / value heads")
            f: dict[str, Any] = {"dim": positive_int(need(m, "dim", where), where), "vdim": positive_int(need(m, "vdim", where), where)}
            sizes = {"heads", "kv_heads", "dim", "vdim"}
            if kind == "channel_delta":
                known(m, sizes | {"conv", "rank_decay", "rank_gate"}, where)
                f["conv"] = positive_int(need(m, "conv", where), where)
                for key, name in (("rank_decay", f"l{i}.mix.a1"), ("rank_gate", f"l{i}.mix.g1")):
                    if tensors is not None and name not in tensors:
                        raise ModelConfigError(f"{where}: {name} is missing")
                    f[key] = int(tensors[name].shape[0]) if tensors is not None else positive_int(need(m, key, where), where)
            else:
                known(m, sizes | {"mask", "scale", "softcap"}, where)
                f["scale"], f["softcap"] = float(need(m, "scale", where)), float(m.get("softcap") or 0.0)
                mask = m.get("mask")
                if mask is not None:
                    known(mask, {"size", "keep_first"}, where)
                    f["window"], f["keep_first"] = positive_int(need(mask, "size", where), where), positive_int(mask.get("keep_first") or 0, where, 0)
            mlp = entry.get("mlp")
            if mlp is not None:
                known(mlp, {"kind", "expert", "router"}, where)
                if need(mlp, "kind", where) != "moe":
                    raise ModelConfigError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
                known(need(mlp, "expert", where), {"ff"}, where)
                known(need(mlp, "router", where), {"experts", "top"}, where)
                f["expert_ff"] = positive_int(need(mlp["expert"], "ff", where), where)
                f["experts"], f["top"] = (positive_int(need(mlp["router"], k, where), where) for k in ("experts", "top"))
                if f["top"] > f["experts"]:
                    raise ModelConfigError(f"{where}: {f['top']} of {f['experts']} experts")
            layers.append(MurilornLayer(kind, heads, kv_heads, **f))
        if not layers:
            raise ModelConfigError("config: no layers")
        loop = raw.get("loop")
        if loop is not None:
            known(loop, {"start", "stop", "times"}, "loop")
            loop = tuple(positive_int(need(loop, k, "loop"), "loop", low) for k, low in (("start", 0), ("stop", 0), ("times", 1)))
            if not loop[0] <= loop[1] <= len(layers):
                raise ModelConfigError(f"loop: layers {loop[0]} .. {loop[1] - 1} of {len(layers)}")
        return cls(positive_int(need(raw, "vocab", "config"), "vocab"), positive_int(need(raw, "width", "config"), "width"),
                   float(need(need(raw, "embedding", "config"), "scale", "embedding")), float(need(need(raw, "norm", "config"), "eps", "norm")),
                   positive_int(raw.get("streams") or 0, "streams", 0), loop, float(1.0 if raw.get("logit_scale") is None else raw["logit_scale"]), float(raw.get("logit_softcap") or 0.0),
                   tuple(layers))

    def to_dict(self) -> dict:
        def layer(y: MurilornLayer) -> dict:
            m: dict[str, Any] = {"dim": y.dim, "heads": y.heads, "kv_heads": y.kv_heads, "vdim": y.vdim}
            if y.type == "channel_delta":
                m.update(conv=y.conv, rank_decay=y.rank_decay, rank_gate=y.rank_gate)
            else:
                m.update(scale=y.scale, softcap=y.softcap)
                if y.window:
                    m["mask"] = {"size": y.window, "keep_first": y.keep_first}
            mlp = {"kind": "moe", "expert": {"ff": y.expert_ff}, "router": {"experts": y.experts, "top": y.top}} if y.experts else None
            return {"type": y.type, "mixer": m, "mlp": mlp}

        out: dict[str, Any] = {"architecture": "Murilorn", "embedding": {"scale": self.embed_scale}, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                               "width": self.width, "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
                               "layers": [layer(y) for y in self.layers]}
        if self.streams:
            out["streams"] = self.streams
        if self.loop:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out


def layer_order(cfg: MurilornConfig) -> list[int]:
    """Layers in the order they run."""
    n = len(cfg.layers)
    if cfg.loop is None:
        return list(range(n))
    start, stop, times = cfg.loop
    return [*range(start), *list(range(start, stop)) * times, *range(stop, n)]


def expected_shapes(cfg: MurilornConfig) -> dict[str, tuple[int, ...]]:
    """Tensor names and shapes of a model of this configuration."""
    w = cfg.width
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab, w), "final.norm": (w,), "head": (cfg.vocab, w)}
    for i, y in enumerate(cfg.layers):
        p = f"l{i}."
        out[p + "norm1"] = (w,)
        delta = y.type == "channel_delta"
        for n, r in (("q", (y.kv_heads if delta else y.heads) * y.dim), ("k", y.kv_heads * y.dim), ("v", (y.heads if delta else y.kv_heads) * y.vdim)):
            out[p + f"mix.{n}"] = (r, w)
            if delta:
                out[p + f"mix.{n}.conv"] = (r, y.conv)
            else:
                out[p + f"mix.{n}.b"] = (r,)
        if delta:
            out.update({p + "mix.b": (y.heads, w), p + "mix.A_log": (y.heads,), p + "mix.norm": (y.vdim,), p + "mix.dt_bias": (y.heads * y.dim,),
                        p + "mix.a1": (y.rank_decay, w), p + "mix.a2": (y.heads * y.dim, y.rank_decay),
                        p + "mix.g1": (y.rank_gate, w), p + "mix.g2": (y.heads * y.vdim, y.rank_gate)})
        out[p + "mix.o"] = (w, y.heads * y.vdim)
        if y.experts:
            out[p + "norm2"], out[p + "mlp.router"] = (w,), (y.experts, w)
            for e in range(y.experts):
                out.update({p + f"mlp.e{e}.gate": (y.expert_ff, w), p + f"mlp.e{e}.up": (y.expert_ff, w), p + f"mlp.e{e}.down": (w, y.expert_ff)})
        for q in range(1, (3 if y.experts else 2) if cfg.streams else 0):
            out.update({p + f"hc{q}.in": (cfg.streams,), p + f"hc{q}.out": (cfg.streams,), p + f"hc{q}.mix": (cfg.streams, cfg.streams)})
    return out


def engine_config(cfg: MurilornConfig, **kw) -> LayeredEngineConfig:
    """``kw``: serving limits (``max_seq``, ``max_batch``, ``kv_tokens``, ``dtype``, ...). Later passes of the loop take the tensors of the
    first one and have caches and states of their own."""
    specs, first = [], {}
    for i in layer_order(cfg):
        y = cfg.layers[i]
        specs.append(LayerSpec(heads=y.heads, kv_heads=y.kv_heads, dim=y.dim, vdim=y.vdim, scale=y.scale, conv_taps=y.conv, window=y.window, ff_act="silu",
                               mixer="delta" if y.type == "channel_delta" else "attention", qkv_bias=int(y.type == "attention"), keep_first=y.keep_first,
                               softcap=y.softcap, sink=int(y.type == "attention"), rank_decay=y.rank_decay, rank_gate=y.rank_gate, experts=y.experts, top=y.top,
                               expert_ff=y.expert_ff, weights_of=first.get(i, -1)))
        first.setdefault(i, len(specs) - 1)
    return LayeredEngineConfig(layers=tuple(specs), width=cfg.width, vocab=cfg.vocab, embed_scale=cfg.embed_scale, norm_eps=cfg.norm_eps, chained=1,
                               streams=cfg.streams, untied_head=1, norm_offset=1.0, logit_scale=cfg.logit_scale, logit_softcap=cfg.logit_softcap, **kw)


def pack_tensors(cfg: MurilornConfig, tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The model's tensors under the engine's names: one input product per layer ([q | k | v], for delta layers followed by
    [beta | decay | gate] rows), the experts stacked, heads and widths padded with zeros to multiples of 16."""
    idle = tuple(f"l{i}.{n}" for i, y in enumerate(cfg.layers) if not y.experts for n in ("norm2", "hc2."))     # of a feed-forward that is not there
    T = check_tensors(expected_shapes(cfg), {n: t for n, t in tensors.items() if not (idle and n.startswith(idle))})
    wp = up(cfg.width)

    def rows(n: str, groups: int, to: int) -> torch.Tensor:          # [groups * k, width] -> [groups * to, wp]
        return pad_rows(pad_cols(T[n], 1, wp), groups, to)

    def vec(n: str) -> torch.Tensor:
        return pad_rows(T[n], 1, wp)

    out = {"embed": rows("embed", 1, up(cfg.vocab)), "head": rows("head", 1, up(cfg.vocab)), "final_norm": vec("final.norm")}
    seen: set[int] = set()
    for run, i in enumerate(layer_order(cfg)):
        if i in seen:
            continue
        seen.add(i)
        y, p, q = cfg.layers[i], f"l{i}.", f"layers.{run}."
        dp, vp = up(y.dim), up(y.vdim)
        delta = y.type == "channel_delta"
        heads = (("q", y.kv_heads if delta else y.heads, dp), ("k", y.kv_heads, dp), ("v", y.heads if delta else y.kv_heads, vp))
        parts = [rows(p + f"mix.{n}", g, to) for n, g, to in heads]
        if delta:
            ra, rg = up(y.rank_decay), up(y.rank_gate)
            parts += [rows(p + "mix.b", 1, up(y.heads)), rows(p + "mix.a1", 1, ra), rows(p + "mix.g1", 1, rg)]
            out[q + "conv"] = torch.cat([pad_rows(T[p + f"mix.{n}.conv"], g, to) for n, g, to in heads]).T.contiguous()
            out[q + "w_a2"] = pad_rows(pad_cols(T[p + "mix.a2"], 1, ra), y.heads, dp)
            out[q + "w_g2"] = pad_rows(pad_cols(T[p + "mix.g2"], 1, rg), y.heads, vp)
            out[q + "a_log"], out[q + "dt_bias"] = T[p + "mix.A_log"], pad_rows(T[p + "mix.dt_bias"], y.heads, dp)
            out[q + "out_norm"] = pad_rows(T[p + "mix.norm"], 1, vp)
        else:
            out[q + "bias_in"] = torch.cat([pad_rows(T[p + f"mix.{n}.b"], g, to) for n, g, to in heads])
        out[q + "norm1"], out[q + "w_in"] = vec(p + "norm1"), torch.cat(parts)
        out[q + "w_out"] = pad_rows(pad_cols(T[p + "mix.o"], y.heads, vp), 1, wp)
        if y.experts:
            fp = up(y.expert_ff)
            ex = range(y.experts)
            out[q + "norm2"], out[q + "router"] = vec(p + "norm2"), rows(p + "mlp.router", 1, up(y.experts))
            out[q + "w_gate_up"] = torch.stack([torch.cat([rows(p + f"mlp.e{e}.{n}", 1, fp) for n in ("gate", "up")]) for e in ex])
            out[q + "w_down"] = torch.stack([pad_rows(pad_cols(T[p + f"mlp.e{e}.down"], 1, fp), 1, wp) for e in ex])
        for k in range(1, (3 if y.experts else 2) if cfg.streams else 0):
            for n in ("in", "out", "mix"):
                out[q + f"hc{k}_{n}"] = T[p + f"hc{k}.{n}"]
    return out


def random_tensors(cfg: MurilornConfig, seed: int = 0, device: str = "cpu") -> dict[str, torch.Tensor]:
    """Random bf16 weights with activations of order one and decays that span short and long memories (tests, throughput runs)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for n, shape in expected_shapes(cfg).items():
        t, leaf = torch.randn(shape, generator=g, device=device), n.split(".", 1)[-1]
        if leaf == "mix.norm":
            t = 1 + 0.1 * t
        elif leaf in ("norm1", "norm2", "norm") or leaf.endswith(".b") and len(shape) == 1:
            t = 0.1 * t
        elif leaf == "mix.A_log":
            t = 0.5 * t - 1.0
        elif leaf == "mix.dt_bias":
            t = t - 1.0
        elif leaf.startswith("hc"):
            s = cfg.streams
            t = 0.2 * t + (torch.eye(s, device=device) if leaf.endswith("mix") else 1.0 / s if leaf.endswith("in") else 1.0)
        else:
            t = t / shape[-1] ** 0.5
        out[n] = t.to(torch.bfloat16)
    return out
