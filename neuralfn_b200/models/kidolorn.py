"""Kidolorn: a decoder whose sublayers have a norm before and one after them, each with a single factor, and read their input plus a short causal
convolution of it. Three kinds of mixers: linear attention with a constant decay per head ("lightning"), a gated recurrence that decides from the
current token alone ("mingru"), and latent attention over every earlier token with a learned sink per head and an output gate (a layer may read an earlier
one's cache). Feed-forwards have a clamped gate, dense with biases or routed with the softmax over the chosen experts as weights.

``KidolornConfig.from_dict`` reads the model's ``config.json``, ``pack_tensors`` turns its tensors into the fused, padded ones of the layer-list engine
(``serving.engine.LayeredEngineConfig``), ``engine_config`` describes the layers to it. All sizes and constants come from the configuration; every
layer has its own.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

import torch

from ..serving.engine import LayeredEngineConfig, LayerSpec
from .layered_common import ModelConfigError, check_tensors, known, need, pad_cols, pad_rows, positive_int, up

__all__ = ["KidolornConfig", "KidolornLayer", "engine_config", "expected_shapes", "pack_tensors", "random_tensors"]

MIXERS = ("lightning", "mingru", "latent_attention")
GATE_SLOPE = 1.702       # of the sigmoid in the feed-forward's gate


@dataclass(frozen=True)
class KidolornLayer:
    type: str
    heads: int = 1
    dim: int = 1
    vdim: int = 1               # mingru: its width
    decay: tuple[float, ...] = ()
    scale: float = 1.0          # latent attention
    rot_dim: int = 0
    rot_base: float = 10000.0
    kv_rank: int = 0
    kv_from: int = -1
    ff: int = 0                 # dense feed-forward
    experts: int = 0            # routed feed-forward
    top: int = 0
    expert_ff: int = 0
    limit: float = 0.0          # of either one's gate


@dataclass(frozen=True)
class KidolornConfig:
    vocab: int
    width: int
    norm_eps: float
    taps: int
    layers: tuple[KidolornLayer, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KidolornConfig":
        known(raw, {"architecture", "canon", "layers", "norm", "vocab", "width"}, "config")
        layers: list[KidolornLayer] = []
        for i, entry in enumerate(need(raw, "layers", "config")):
            where = f"layer {i}"
            known(entry, {"type", "mixer", "mlp"}, where)
            kind, m = need(entry, "type", where), need(entry, "mixer", where)
            if kind not in MIXERS:
                raise ModelConfigError(f"{where}: unknown layer type {kind!r}")
            size = lambda key, low=1: positive_int(need(m, key, where), f"{where}: {key}", low)  # noqa: B023, E731
            f: dict[str, Any] = {}
            if kind == "mingru":
                known(m, {"width"}, where)
                f["vdim"] = size("width")
            elif kind == "lightning":
                known(m, {"decay", "dim", "heads", "vdim"}, where)
                f.update(heads=size("heads"), dim=size("dim"), vdim=size("vdim"), decay=tuple(float(d) for d in need(m, "decay", where)))
                if len(f["decay"]) != f["heads"]:
                    raise ModelConfigError(f"{where}: {len(f['decay'])} decays for {f['heads']} heads")
            else:
                known(m, {"dim", "heads", "kv_from", "kv_rank", "rot", "rot_dim", "scale", "vdim"}, where)
                f.update(heads=size("heads"), dim=size("dim"), vdim=size("vdim"), kv_rank=size("kv_rank"), rot_dim=size("rot_dim"), scale=float(need(m, "scale", where)))
                rot = need(m, "rot", where)
                known(rot, {"base", "dims"}, f"{where}: rot")
                f["rot_base"] = float(need(rot, "base", where))
                if f["rot_dim"] % 2 or f["rot_base"] <= 0:
                    raise ModelConfigError(f"{where}: an even number of rotated dimensions and a positive base, not {dict(rot)}")
                if positive_int(need(rot, "dims", where), f"{where}: rot.dims") != f["rot_dim"]:
                    raise ModelConfigError(f"{where}: all of the rotated part turns, so rot.dims is rot_dim")
                if m.get("kv_from") is not None:
                    j = f["kv_from"] = positive_int(m["kv_from"], f"{where}: kv_from", 0)
                    o = layers[j] if j < i else None
                    if o is None or o.type != kind or o.kv_from >= 0:
                        raise ModelConfigError(f"{where}: kv_from names an earlier latent layer with a cache of its own")
                    if (o.kv_rank, o.rot_dim, o.rot_base) != (f["kv_rank"], f["rot_dim"], f["rot_base"]):
                        raise ModelConfigError(f"{where}: layer {j} caches another latent or rotation")
            mlp = entry.get("mlp")
            if mlp is not None:
                what = need(mlp, "kind", where)
                if what == "dense":
                    known(mlp, {"kind", "ff", "limit"}, f"{where}: mlp")
                    f.update(ff=positive_int(need(mlp, "ff", where), f"{where}: ff"), limit=float(need(mlp, "limit", where)))
                elif what == "moe":
                    known(mlp, {"kind", "expert", "router"}, f"{where}: mlp")
                    expert, router = need(mlp, "expert", where), need(mlp, "router", where)
                    known(expert, {"ff", "limit"}, f"{where}: expert")
                    known(router, {"experts", "top"}, f"{where}: router")
                    f.update(expert_ff=positive_int(need(expert, "ff", where), f"{where}: expert.ff"), limit=float(need(expert, "limit", where)))
                    f["experts"], f["top"] = (positive_int(need(router, k, where), f"{where}: {k}") for k in ("experts", "top"))
                    if f["top"] > f["experts"]:
                        raise ModelConfigError(f"{where}: {f['top']} of {f['experts']} experts")
                else:
                    raise ModelConfigError(f"{where}: unknown feed-forward kind {what!r}")
                if not f["limit"] > 0:
                    raise ModelConfigError(f"{where}: the gate's limit must be positive")
            layers.append(KidolornLayer(kind, **f))
        if not layers:
            raise ModelConfigError("config: no layers")
        canon = need(raw, "canon", "config")
        known(canon, {"taps"}, "canon")
        return cls(positive_int(need(raw, "vocab", "config"), "vocab"), positive_int(need(raw, "width", "config"), "width"),
                   float(need(need(raw, "norm", "config"), "eps", "norm")), positive_int(need(canon, "taps", "canon"), "canon.taps"), tuple(layers))

    def to_dict(self) -> dict:
        def layer(y: KidolornLayer) -> dict:
            if y.type == "mingru":
                m: dict[str, Any] = {"width": y.vdim}
            elif y.type == "lightning":
                m = {"heads": y.heads, "dim": y.dim, "vdim": y.vdim, "decay": list(y.decay)}
            else:
                m = {"heads": y.heads, "dim": y.dim, "vdim": y.vdim, "kv_rank": y.kv_rank, "rot_dim": y.rot_dim, "scale": y.scale, "rot": {"base": y.rot_base, "dims": y.rot_dim}}
                if y.kv_from >= 0:
                    m["kv_from"] = y.kv_from
            mlp: dict[str, Any] | None = {"kind": "dense", "ff": y.ff, "limit": y.limit} if y.ff else None
            if y.experts:
                mlp = {"kind": "moe", "expert": {"ff": y.expert_ff, "limit": y.limit}, "router": {"experts": y.experts, "top": y.top}}
            return {"type": y.type, "mixer": m, "mlp": mlp}

        return {"architecture": "Kidolorn", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "canon": {"taps": self.taps},
                "layers": [layer(y) for y in self.layers]}


def expected_shapes(cfg: KidolornConfig) -> dict[str, tuple[int, ...]]:
    """Tensor names and shapes of a model of this configuration."""
    w = cfg.width
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab, w), "final.norm": (), "head": (cfg.vocab, w)}
    for i, y in enumerate(cfg.layers):
        p, q, n = f"l{i}.mix.", f"l{i}.mlp.", y.heads * y.vdim
        for s in ("1", "2") if y.ff or y.experts else ("1",):
            out.update({f"l{i}.norm{s}": (), f"l{i}.norm{s}b": (), f"l{i}.canon{s}": (w, cfg.taps)})
        out.update({p + "g": (n, w), p + "o": (w, n)})
        if y.type == "mingru":
            out.update({p + "z": (n, w), p + "z.b": (n,), p + "x": (n, w), p + "x.b": (n,)})
        elif y.type == "lightning":
            out.update({p + "q": (y.heads * y.dim, w), p + "k": (y.heads * y.dim, w), p + "v": (n, w), p + "norm": (n,)})
        else:
            out.update({p + "q": (y.heads * (y.dim + y.rot_dim), w), p + "uk": (y.heads * y.dim, y.kv_rank), p + "uv": (n, y.kv_rank), p + "sink": (y.heads,)})
            if y.kv_from < 0:
                out.update({p + "dkv": (y.kv_rank + y.rot_dim, w), p + "dkv.norm": (y.kv_rank,)})
        if y.ff:
            for s, shape in (("gate", (y.ff, w)), ("up", (y.ff, w)), ("down", (w, y.ff))):
                out[q + s], out[q + s + ".b"] = shape, shape[:1]
        if y.experts:
            out[q + "router"] = (y.experts, w)
            for e in range(y.experts):
                out.update({q + f"e{e}.gate": (y.expert_ff, w), q + f"e{e}.up": (y.expert_ff, w), q + f"e{e}.down": (w, y.expert_ff)})
    return out


def engine_config(cfg: KidolornConfig, **kw) -> LayeredEngineConfig:
    """``kw``: serving limits (``max_seq``, ``max_batch``, ``kv_tokens``, ``dtype``, ...)."""
    specs = []
    for y in cfg.layers:
        f: dict[str, Any] = dict(heads=y.heads, kv_heads=y.heads, dim=y.dim, vdim=y.vdim, scale=y.scale)
        if y.type == "mingru":
            f.update(mixer="gru", qkv_bias=1)
        elif y.type == "lightning":
            f.update(mixer="linear", decay=y.decay)
        else:
            f.update(mixer="latent", kv_heads=1, kv_from=y.kv_from, kv_rank=y.kv_rank, rot_dim=y.rot_dim, rot_dims=y.rot_dim, rot_base=y.rot_base, sink=2, out_gate=1)
        if y.ff or y.experts:
            f.update(ff_act="clamped", ff_limit=y.limit, ff_slope=GATE_SLOPE)
        if y.ff:
            f.update(ff=y.ff, ff_bias=1)
        if y.experts:
            f.update(experts=y.experts, top=y.top, expert_ff=y.expert_ff, route_softmax=1, expert_weigh_out=1)
        specs.append(LayerSpec(**f))
    return LayeredEngineConfig(layers=tuple(specs), width=cfg.width, vocab=cfg.vocab, norm_eps=cfg.norm_eps, chained=1, untied_head=1, sandwich=1, scalar_norms=1,
                               input_taps=cfg.taps, **kw)


def _pairs(n: int) -> torch.Tensor:
    """Order in which dimensions that turn together, i and i + n / 2, stand side by side: scores do not depend on the order of the channels, and the
    engine's rotation takes neighbours."""
    return torch.stack([torch.arange(n // 2), torch.arange(n // 2, n)], 1).flatten()


def pack_tensors(cfg: KidolornConfig, tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The model's tensors under the engine's names: one input product per layer ([share | candidate | gate], [q | k | v | gate] or [q | latent | key
    part | gate]), rotated dimensions in pairs, key and value projections of a latent both as one matrix and, for the keys, transposed per head, the
    experts stacked, convolutions tap by tap, heads and widths padded with zeros to multiples of 16."""
    idle = {f"l{i}.{n}" for i, y in enumerate(cfg.layers) if not (y.ff or y.experts) for n in ("norm2", "norm2b", "canon2")}      # of a feed-forward that is not there
    T = check_tensors(expected_shapes(cfg), {n: t for n, t in tensors.items() if n not in idle})
    wp = up(cfg.width)

    def rows(n: str, groups: int, to: int) -> torch.Tensor:          # [groups * k, width] -> [groups * to, wp]
        return pad_rows(pad_cols(T[n], 1, wp), groups, to)

    def vec(n: str, to: int, groups: int = 1) -> torch.Tensor:
        return pad_rows(T[n], groups, to)

    out = {"embed": rows("embed", 1, up(cfg.vocab)), "head": rows("head", 1, up(cfg.vocab)), "final_norm": T["final.norm"].reshape(1)}
    for i, y in enumerate(cfg.layers):
        p, m, q = f"l{i}.mix.", f"l{i}.mlp.", f"layers.{i}."
        dp, vp = up(y.dim), up(y.vdim)
        for s in ("1", "2") if y.ff or y.experts else ("1",):
            out[q + "norm" + s], out[q + f"norm{s}_b"] = T[f"l{i}.norm{s}"].reshape(1), T[f"l{i}.norm{s}b"].reshape(1)
            out[q + "in_conv" + s] = pad_rows(T[f"l{i}.canon{s}"], 1, wp).T.contiguous()
        out[q + "w_out"] = pad_rows(pad_cols(T[p + "o"], y.heads, vp), 1, wp)
        gate = rows(p + "g", y.heads, vp)
        if y.type == "mingru":
            out[q + "w_in"] = torch.cat([rows(p + "z", 1, vp), rows(p + "x", 1, vp), gate])
            out[q + "bias_in"] = torch.cat([vec(p + "z.b", vp), vec(p + "x.b", vp), torch.zeros(vp, dtype=gate.dtype, device=gate.device)])
        elif y.type == "lightning":
            out[q + "w_in"] = torch.cat([rows(p + "q", y.heads, dp), rows(p + "k", y.heads, dp), rows(p + "v", y.heads, vp), gate])
            out[q + "out_norm"] = vec(p + "norm", vp, y.heads)
        else:
            rp, lr, order = up(y.rot_dim), up(y.kv_rank), _pairs(y.rot_dim)
            full = rows(p + "q", 1, y.heads * (y.dim + y.rot_dim)).reshape(y.heads, y.dim + y.rot_dim, wp)
            parts = [torch.cat([pad_rows(full[:, :y.dim].reshape(-1, wp), y.heads, dp).view(y.heads, dp, wp),
                                pad_rows(full[:, y.dim:][:, order].reshape(-1, wp), y.heads, rp).view(y.heads, rp, wp)], 1).reshape(-1, wp)]
            if y.kv_from < 0:
                dkv = pad_cols(T[p + "dkv"], 1, wp)
                parts += [pad_rows(dkv[:y.kv_rank], 1, lr), pad_rows(dkv[y.kv_rank:][order], 1, rp)]
                out[q + "c_norm"] = vec(p + "dkv.norm", lr)
            out[q + "w_in"] = torch.cat(parts + [gate])
            uk, uv = (pad_rows(pad_cols(T[p + n], 1, lr), y.heads, to) for n, to in (("uk", dp), ("uv", vp)))
            out[q + "w_ukv"], out[q + "w_uk_t"] = torch.cat([uk, uv]), uk.view(y.heads, dp, lr).transpose(1, 2).contiguous()
            out[q + "sink"] = T[p + "sink"]
        if y.ff:
            fp = up(y.ff)
            out[q + "w_gate_up"], out[q + "w_down"] = torch.cat([rows(m + n, 1, fp) for n in ("gate", "up")]), pad_rows(pad_cols(T[m + "down"], 1, fp), 1, wp)
            out[q + "bias_gate_up"], out[q + "bias_down"] = torch.cat([vec(m + n + ".b", fp) for n in ("gate", "up")]), vec(m + "down.b", wp)
        if y.experts:
            fp, ex = up(y.expert_ff), range(y.experts)
            out[q + "router"] = rows(m + "router", 1, up(y.experts))
            out[q + "w_gate_up"] = torch.stack([torch.cat([rows(m + f"e{e}.gate", 1, fp), rows(m + f"e{e}.up", 1, fp)]) for e in ex])
            out[q + "w_down"] = torch.stack([pad_rows(pad_cols(T[m + f"e{e}.down"], 1, fp), 1, wp) for e in ex])
    return out


def random_tensors(cfg: KidolornConfig, seed: int = 0, device: str = "cpu") -> dict[str, torch.Tensor]:
    """Random bf16 weights with activations of order one (tests, throughput runs)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for n, shape in expected_shapes(cfg).items():
        t, leaf = torch.randn(shape, generator=g, device=device), n.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            t = 1 + 0.1 * t
        elif leaf == "b":
            t = 0.5 * t
        elif leaf.startswith("canon"):
            t = t / (shape[-1] + 1) ** 0.5
        elif leaf != "sink" and n != "embed":
            t = t / shape[-1] ** 0.5
        out[n] = t.to(torch.bfloat16)
    return out
