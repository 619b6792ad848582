"""Vopozen: a decoder whose sublayers read the residual itself and have their norm on the output. Three kinds of mixers: grouped attention inside
chunks of positions (normed and rotated queries and keys, the keys as projected are the values), latent attention with a sliding window (one
cached latent and rotated key part per token for all heads; a layer may read an earlier one's cache), and time mixing with a token shift and
a recurrence that gives the current token a bonus. Feed-forwards are gated or routed: plain experts with grouped choice, a correction of the
choice and a shared expert.

``VopozenConfig.from_dict`` reads the model's ``config.json`` (the inner size of the decay projection comes from the tensors), ``pack_tensors``
turns its tensors into the fused, padded ones of the layer-list engine (``serving.engine.LayeredEngineConfig``), ``engine_config`` describes the
layers to it. All sizes and constants come from the configuration; every layer has its own.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

import torch

from ..serving.engine import LayeredEngineConfig, LayerSpec
from .layered_common import ModelConfigError, check_tensors, known, need, pad_cols, pad_rows, positive_int, up

__all__ = ["VopozenConfig", "VopozenLayer", "engine_config", "expected_shapes", "pack_tensors", "random_tensors"]

MIXERS = ("attention", "latent_attention", "wkv")
SHIFTED = "rkvgw"        # the inputs of time mixing, in the order of their tensors


@dataclass(frozen=True)
class VopozenLayer:
    type: str
    heads: int
    kv_heads: int               # attention
    dim: int
    vdim: int
    look: int = 0               # attention: chunk; latent attention: window; 0: every earlier key
    scale: float = 1.0
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_dim: int = 0            # latent attention
    kv_rank: int = 0
    kv_from: int = -1
    rank_decay: int = 0         # wkv: rows of w1
    ff: int = 0                 # gated feed-forward
    experts: int = 0            # routed feed-forward
    top: int = 0
    expert_ff: int = 0
    shared_ff: int = 0
    groups: int = 0
    keep: int = 0
    route_scale: float = 1.0


@dataclass(frozen=True)
class VopozenConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: tuple[VopozenLayer, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], tensors: Mapping[str, torch.Tensor] | None = None) -> "VopozenConfig":
        """``tensors``: the checkpoint, for the sizes only its shapes give; without it the entry "rank_decay" of a mixer (written by
        ``to_dict``) is read."""
        known(raw, {"architecture", "layers", "norm", "residual_mult", "vocab", "width"}, "config")
        layers: list[VopozenLayer] = []
        for i, entry in enumerate(need(raw, "layers", "config")):
            where = f"layer {i}"
            known(entry, {"type", "mixer", "mlp"}, where)
            kind, m = need(entry, "type", where), need(entry, "mixer", where)
            if kind not in MIXERS:
                raise ModelConfigError(f"{where}: unknown layer type {kind!r}")
            size = lambda key, low=1: positive_int(need(m, key, where), f"{where}: {key}", low)  # noqa: B023, E731
            f: dict[str, Any] = {"heads": size("heads"), "dim": size("dim")}
            if kind == "wkv":
                known(m, {"heads", "dim", "rank_decay"}, where)
                name = f"l{i}.mix.w1"
                if tensors is not None and name not in tensors:
                    raise ModelConfigError(f"{where}: {name} is missing")
                f.update(kv_heads=f["heads"], vdim=f["dim"], rank_decay=int(tensors[name].shape[0]) if tensors is not None else size("rank_decay"))
            else:
                f["vdim"], f["scale"] = size("vdim"), float(need(m, "scale", where))
                rot = need(m, "rot", where)
                known(rot, {"base", "dims"}, f"{where}: rot")
                f["rot_base"], f["rot_dims"] = float(need(rot, "base", where)), positive_int(need(rot, "dims", where), f"{where}: rot.dims", 0)
                if f["rot_dims"] % 2 or f["rot_base"] <= 0:
                    raise ModelConfigError(f"{where}: an even number of rotated dimensions and a positive base, not {dict(rot)}")
                mask = m.get("mask")
                if mask is not None:
                    known(mask, {"size"}, f"{where}: mask")
                    f["look"] = positive_int(need(mask, "size", where), f"{where}: mask.size")
                if kind == "attention":
                    known(m, {"heads", "dim", "kv_heads", "vdim", "scale", "rot", "mask"}, where)
                    f["kv_heads"] = size("kv_heads")
                    if f["heads"] % f["kv_heads"]:
                        raise ModelConfigError(f"{where}: {f['heads']} heads do not divide into {f['kv_heads']} key / value heads")
                    if f["vdim"] != f["dim"]:
                        raise ModelConfigError(f"{where}: the values are the keys, so vdim is dim")
                    if f["rot_dims"] > f["dim"]:
                        raise ModelConfigError(f"{where}: {f['rot_dims']} rotated dimensions of {f['dim']}")
                else:
                    known(m, {"heads", "dim", "kv_rank", "kv_from", "rot_dim", "vdim", "scale", "rot", "mask"}, where)
                    f.update(kv_heads=1, kv_rank=size("kv_rank"), rot_dim=size("rot_dim"))
                    if f["rot_dims"] != f["rot_dim"]:
                        raise ModelConfigError(f"{where}: all of the rotated part turns, so rot.dims is rot_dim")
                    if m.get("kv_from") is not None:
                        j = f["kv_from"] = positive_int(m["kv_from"], f"{where}: kv_from", 0)
                        o = layers[j] if j < i else None
                        if o is None or o.type != kind or o.kv_from >= 0:
                            raise ModelConfigError(f"{where}: kv_from names an earlier latent layer with a cache of its own")
                        if (o.kv_rank, o.rot_dim, o.rot_dims, o.rot_base) != (f["kv_rank"], f["rot_dim"], f["rot_dims"], f["rot_base"]):
                            raise ModelConfigError(f"{where}: layer {j} caches another latent or rotation")
            mlp = entry.get("mlp")
            if mlp is not None:
                what = need(mlp, "kind", where)
                if what == "dense":
                    known(mlp, {"kind", "ff"}, f"{where}: mlp")
                    f["ff"] = positive_int(need(mlp, "ff", where), f"{where}: ff")
                elif what == "moe":
                    known(mlp, {"kind", "expert", "router", "shared"}, f"{where}: mlp")
                    router = need(mlp, "router", where)
                    known(need(mlp, "expert", where), {"ff"}, f"{where}: expert")
                    known(router, {"experts", "top", "groups", "scale"}, f"{where}: router")
                    f["expert_ff"] = positive_int(need(mlp["expert"], "ff", where), f"{where}: expert.ff")
                    f["experts"], f["top"] = (positive_int(need(router, k, where), f"{where}: {k}") for k in ("experts", "top"))
                    f["route_scale"] = float(1.0 if router.get("scale") is None else router["scale"])
                    open_to = f["experts"]
                    if router.get("groups") is not None:
                        known(router["groups"], {"count", "keep"}, f"{where}: groups")
                        f["groups"], f["keep"] = (positive_int(need(router["groups"], k, where), f"{where}: groups.{k}") for k in ("count", "keep"))
                        if f["experts"] % f["groups"] or f["keep"] > f["groups"]:
                            raise ModelConfigError(f"{where}: {f['keep']} of {f['groups']} groups of {f['experts']} experts")
                        open_to = f["experts"] // f["groups"] * f["keep"]
                    if f["top"] > open_to:
                        raise ModelConfigError(f"{where}: {f['top']} of {open_to} experts")
                    if mlp.get("shared") is not None:
                        known(mlp["shared"], {"ff"}, f"{where}: shared")
                        f["shared_ff"] = positive_int(need(mlp["shared"], "ff", where), f"{where}: shared.ff")
                else:
                    raise ModelConfigError(f"{where}: unknown feed-forward kind {what!r}")
            layers.append(VopozenLayer(kind, **f))
        if not layers:
            raise ModelConfigError("config: no layers")
        return cls(positive_int(need(raw, "vocab", "config"), "vocab"), positive_int(need(raw, "width", "config"), "width"),
                   float(need(need(raw, "norm", "config"), "eps", "norm")), float(need(raw, "residual_mult", "config")), tuple(layers))

    def to_dict(self) -> dict:
        def layer(y: VopozenLayer) -> dict:
            m: dict[str, Any] = {"heads": y.heads, "dim": y.dim}
            if y.type == "wkv":
                m["rank_decay"] = y.rank_decay
            else:
                m.update(vdim=y.vdim, scale=y.scale, rot={"base": y.rot_base, "dims": y.rot_dims})
                if y.look:
                    m["mask"] = {"size": y.look}
                if y.type == "attention":
                    m["kv_heads"] = y.kv_heads
                else:
                    m.update(kv_rank=y.kv_rank, rot_dim=y.rot_dim)
                    if y.kv_from >= 0:
                        m["kv_from"] = y.kv_from
            mlp: dict[str, Any] | None = {"kind": "dense", "ff": y.ff} if y.ff else None
            if y.experts:
                mlp = {"kind": "moe", "expert": {"ff": y.expert_ff}, "router": {"experts": y.experts, "top": y.top, "scale": y.route_scale}}
                if y.groups:
                    mlp["router"]["groups"] = {"count": y.groups, "keep": y.keep}
                if y.shared_ff:
                    mlp["shared"] = {"ff": y.shared_ff}
            return {"type": y.type, "mixer": m, "mlp": mlp}

        return {"architecture": "Vopozen", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                "layers": [layer(y) for y in self.layers]}


def expected_shapes(cfg: VopozenConfig) -> dict[str, tuple[int, ...]]:
    """Tensor names and shapes of a model of this configuration."""
    w = cfg.width
    out: dict[str, tuple[int, ...]] = {"embed": (cfg.vocab, w), "final.norm": (w,), "head": (cfg.vocab, w)}
    for i, y in enumerate(cfg.layers):
        p, q = f"l{i}.mix.", f"l{i}.mlp."
        out[f"l{i}.norm1"], out[p + "o"] = (w,), (w, y.heads * y.vdim)
        if y.type == "attention":
            out.update({p + "q": (y.heads * y.dim, w), p + "k": (y.kv_heads * y.dim, w), p + "q.norm": (y.dim,), p + "k.norm": (y.dim,)})
        elif y.type == "latent_attention":
            out.update({p + "q": (y.heads * (y.dim + y.rot_dim), w), p + "uk": (y.heads * y.dim, y.kv_rank), p + "uv": (y.heads * y.vdim, y.kv_rank)})
            if y.kv_from < 0:
                out.update({p + "dkv": (y.kv_rank + y.rot_dim, w), p + "dkv.norm": (y.kv_rank,)})
        else:
            n = y.heads * y.dim
            out.update({p + s: (n, w) for s in "rkvg"})
            out.update({p + f"mu.{s}": (w,) for s in SHIFTED})
            out.update({p + "w1": (y.rank_decay, w), p + "w2": (n, y.rank_decay), p + "w0": (n,), p + "u": (y.heads, y.dim), p + "norm": (n,)})
        if y.ff or y.experts:
            out[f"l{i}.norm2"] = (w,)
        if y.ff:
            out.update({q + "gate": (y.ff, w), q + "up": (y.ff, w), q + "down": (w, y.ff)})
        if y.experts:
            out.update({q + "router": (y.experts, w), q + "correction": (y.experts,)})
            for e in range(y.experts):
                out.update({q + f"e{e}.up": (y.expert_ff, w), q + f"e{e}.down": (w, y.expert_ff)})
            if y.shared_ff:
                out.update({q + "shared.up": (y.shared_ff, w), q + "shared.down": (w, y.shared_ff)})
    return out


def engine_config(cfg: VopozenConfig, **kw) -> LayeredEngineConfig:
    """``kw``: serving limits (``max_seq``, ``max_batch``, ``kv_tokens``, ``dtype``, ...)."""
    specs = []
    for y in cfg.layers:
        f: dict[str, Any] = dict(heads=y.heads, kv_heads=y.kv_heads, dim=y.dim, vdim=y.vdim, scale=y.scale, ff=y.ff, ff_act="relu2" if y.experts else "silu")
        if y.type == "attention":
            f.update(chunk=y.look, qk_norm=1, rot_dims=y.rot_dims, rot_base=y.rot_base, key_values=1)
        elif y.type == "latent_attention":
            f.update(mixer="latent", window=y.look, kv_from=y.kv_from, kv_rank=y.kv_rank, rot_dim=y.rot_dim, rot_dims=y.rot_dims, rot_base=y.rot_base)
        else:
            f.update(mixer="wkv", rank_decay=y.rank_decay)
        if y.experts:
            f.update(experts=y.experts, top=y.top, expert_ff=y.expert_ff, expert_plain=1, shared_ff=y.shared_ff, route_correction=1, route_groups=y.groups,
                     route_keep=y.keep, route_normalise=1, route_scale=y.route_scale)
        specs.append(LayerSpec(**f))
    return LayeredEngineConfig(layers=tuple(specs), width=cfg.width, vocab=cfg.vocab, norm_eps=cfg.norm_eps, chained=1, untied_head=1, post_norm=1,
                               residual_mult=cfg.residual_mult, **kw)


def pack_tensors(cfg: VopozenConfig, tensors: Mapping[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The model's tensors under the engine's names: one input product per layer ([q | k] or [q | latent | key part]; time mixing: the r, k, v and
    gate matrices one after another), key and value projections of a latent both as one matrix and, for the keys, transposed per head, the
    experts stacked, heads and widths padded with zeros to multiples of 16."""
    idle = tuple(f"l{i}.norm2" for i, y in enumerate(cfg.layers) if not (y.ff or y.experts))      # of a feed-forward that is not there
    T = check_tensors(expected_shapes(cfg), {n: t for n, t in tensors.items() if n not in idle})
    wp = up(cfg.width)

    def rows(n: str, groups: int, to: int) -> torch.Tensor:          # [groups * k, width] -> [groups * to, wp]
        return pad_rows(pad_cols(T[n], 1, wp), groups, to)

    def vec(n: str, to: int = wp) -> torch.Tensor:
        return pad_rows(T[n], 1, to)

    out = {"embed": rows("embed", 1, up(cfg.vocab)), "head": rows("head", 1, up(cfg.vocab)), "final_norm": vec("final.norm")}
    for i, y in enumerate(cfg.layers):
        p, m, q = f"l{i}.mix.", f"l{i}.mlp.", f"layers.{i}."
        dp, vp = up(y.dim), up(y.vdim)
        out[q + "norm1"] = vec(f"l{i}.norm1")
        out[q + "w_out"] = pad_rows(pad_cols(T[p + "o"], y.heads, vp), 1, wp)
        if y.type == "attention":
            out[q + "w_in"] = torch.cat([rows(p + "q", y.heads, dp), rows(p + "k", y.kv_heads, dp)])
            out[q + "q_norm"], out[q + "k_norm"] = vec(p + "q.norm", dp), vec(p + "k.norm", dp)
        elif y.type == "latent_attention":
            rp, lr = up(y.rot_dim), up(y.kv_rank)
            full = rows(p + "q", 1, y.heads * (y.dim + y.rot_dim)).reshape(y.heads, y.dim + y.rot_dim, wp)
            parts = [torch.cat([pad_rows(full[:, :y.dim].reshape(-1, wp), y.heads, dp).view(y.heads, dp, wp),
                                pad_rows(full[:, y.dim:].reshape(-1, wp), y.heads, rp).view(y.heads, rp, wp)], 1).reshape(-1, wp)]
            if y.kv_from < 0:
                dkv = pad_cols(T[p + "dkv"], 1, wp)
                parts += [pad_rows(dkv[:y.kv_rank], 1, lr), pad_rows(dkv[y.kv_rank:], 1, rp)]
                out[q + "c_norm"] = vec(p + "dkv.norm", lr)
            out[q + "w_in"] = torch.cat(parts)
            uk, uv = (pad_rows(pad_cols(T[p + n], 1, lr), y.heads, to) for n, to in (("uk", dp), ("uv", vp)))
            out[q + "w_ukv"], out[q + "w_uk_t"] = torch.cat([uk, uv]), uk.view(y.heads, dp, lr).transpose(1, 2).contiguous()
        else:
            ra = up(y.rank_decay)
            out[q + "w_in"] = torch.cat([rows(p + s, y.heads, dp) for s in "rkvg"])
            out[q + "mu"] = torch.stack([vec(p + f"mu.{s}") for s in SHIFTED])
            w2 = pad_rows(pad_cols(T[p + "w2"], 1, ra), y.heads, dp)
            out[q + "w1"], out[q + "w2"] = rows(p + "w1", 1, ra), torch.cat([w2, w2], 1)
            out[q + "w0"], out[q + "out_norm"] = pad_rows(T[p + "w0"], y.heads, dp), pad_rows(T[p + "norm"], y.heads, dp)
            out[q + "u"] = pad_rows(T[p + "u"].reshape(-1), y.heads, dp)
        if y.ff or y.experts:
            out[q + "norm2"] = vec(f"l{i}.norm2")
        if y.ff:
            fp = up(y.ff)
            out[q + "w_gate_up"], out[q + "w_down"] = torch.cat([rows(m + n, 1, fp) for n in ("gate", "up")]), pad_rows(pad_cols(T[m + "down"], 1, fp), 1, wp)
        if y.experts:
            fp, sp = up(y.expert_ff), up(y.shared_ff)
            ex = range(y.experts)
            out[q + "router"], out[q + "correction"] = rows(m + "router", 1, up(y.experts)), pad_rows(T[m + "correction"], 1, up(y.experts))
            out[q + "w_gate_up"] = torch.stack([rows(m + f"e{e}.up", 1, fp) for e in ex])
            out[q + "w_down"] = torch.stack([pad_rows(pad_cols(T[m + f"e{e}.down"], 1, fp), 1, wp) for e in ex])
            if y.shared_ff:
                out[q + "w_shared_up"], out[q + "w_shared_down"] = rows(m + "shared.up", 1, sp), pad_rows(pad_cols(T[m + "shared.down"], 1, sp), 1, wp)
    return out


def random_tensors(cfg: VopozenConfig, seed: int = 0, device: str = "cpu") -> dict[str, torch.Tensor]:
    """Random bf16 weights with activations of order one and decays that span short and long memories (tests, throughput runs)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for n, shape in expected_shapes(cfg).items():
        t, leaf = torch.randn(shape, generator=g, device=device), n.split(".", 1)[-1]
        if leaf.endswith("norm") or leaf in ("norm1", "norm2"):
            t = 1 + 0.1 * t
        elif leaf.startswith("mix.mu."):
            t = torch.rand(shape, generator=g, device=device)
        elif leaf == "mix.w0":
            t = 1.5 * t - 2.0
        elif leaf == "mix.u":
            t = 0.5 + 0.5 * t
        elif leaf == "mlp.correction":
            t = 0.1 * t
        elif n != "embed":
            t = t / shape[-1] ** 0.5
        out[n] = t.to(torch.bfloat16)
    return out
