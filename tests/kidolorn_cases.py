"""Small Kidolorn configurations and weights for tests. Sublayers write about as much into the residual as the embedding, scores are loud, sinks and
gates matter, and memories are short and long. With random weights rounding flips close choices of experts; ``sharp_routing`` makes models whose
choices are never close: the last eight channels of the residual carry a code of the token that no sublayer touches, and the router listens
mostly to them."""
import math

import torch

from neuralfn_b200.models.kidolorn import KidolornConfig, random_tensors

CODES = 8


def dense(ff=48, limit=1.1):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(*, experts=8, top=3, ff=32, limit=0.9):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def lightning(*, heads=3, dim=24, vdim=40, decay=None, mlp=None):
    if decay is None:
        decay = [1 - 0.5 ** (1 + 8 * (i + 0.5) / heads) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def mingru(*, width=72, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def latent(*, heads=4, dim=24, rot=8, vdim=40, rank=48, base=500.0, scale=0.4, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def model(layers, *, vocab=96, width=64, eps=1e-5, taps=3, seed=0):
    cfg = {"architecture": "Kidolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}
    w = random_tensors(KidolornConfig.from_dict(cfg), seed)
    for i, y in enumerate(layers):
        if y["type"] == "lightning":                       # keys resemble queries: no read-out is a small difference of large terms before its norm
            w[f"l{i}.mix.k"] = (0.85 * w[f"l{i}.mix.q"].float() + 0.5 * w[f"l{i}.mix.k"].float()).to(torch.bfloat16)
        if y["type"] == "mingru":                          # from a few tokens to hundreds
            w[f"l{i}.mix.z.b"] = (-6 * torch.rand(y["mixer"]["width"], generator=torch.Generator().manual_seed(seed))).to(torch.bfloat16)
        if y["type"] == "latent_attention":                # some louder than all keys together, some hardly there
            w[f"l{i}.mix.sink"] = torch.linspace(7, -1, y["mixer"]["heads"]).to(torch.bfloat16)
    if any((y["mlp"] or {}).get("kind") == "moe" for y in layers):
        sharp_routing(cfg, w, seed)
    return cfg, w


def tokens_of(cfg, n, *, seed, below=None):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, below or cfg["vocab"], (n,), generator=g).tolist()


def sharp_routing(cfg, w, seed=0):
    width = cfg["width"]
    w["embed"][:, width - CODES:] = 3.0 * torch.eye(CODES, dtype=torch.bfloat16)[torch.arange(cfg["vocab"]) % CODES]
    for n, t in w.items():
        leaf = n.split(".", 1)[-1]
        if leaf.startswith("canon") or leaf == "mix.o" or ("down" in leaf):
            t[width - CODES:] = 0
    for i, layer in enumerate(cfg["layers"]):
        if (layer["mlp"] or {}).get("kind") != "moe":
            continue
        E = layer["mlp"]["router"]["experts"]
        g = torch.Generator().manual_seed(1000 * seed + 7 * i)
        levels = torch.linspace(-2, 2, E) if E > 1 else torch.zeros(1)
        z = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(CODES)])          # [codes, experts]
        r = 0.002 * torch.randn(E, width, generator=g)
        r[:, width - CODES:] = z.T / 1.5
        w[f"l{i}.mlp.router"] = r.to(torch.bfloat16)


def mark(cfg, w, *tokens):
    """A channel of the embedding for each of these tokens alone; returns vectors v with v . embed[token] = 1 and v . embed[other] = 0. (Directions that single a
    token out of random embeddings would be long, and rounding of the normed rows would be loud along them.)"""
    out = []
    for i, token in enumerate(tokens):
        w["embed"][:, cfg["width"] - 1 - i] = 0
        w["embed"][token, cfg["width"] - 1 - i] = 4
        v = torch.zeros(cfg["width"], dtype=torch.float64)
        v[cfg["width"] - 1 - i] = 0.25
        out.append(v)
    return out


def no_convolution(cfg, w):
    for n in w:
        if ".canon" in n:
            w[n].zero_()


def boost_needle(cfg, w, *, query, key):
    """One latent layer and nothing else: the score of `query` on `key` towers over the others in every head, in dimensions that do not turn, and the
    value of `key` is loud."""
    no_convolution(cfg, w)
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    to_q, to_k = mark(cfg, w, query, key)
    H, d, rank = m["heads"], m["dim"], m["kv_rank"]
    e = torch.zeros(rank, dtype=torch.float64)
    e[rank // 2] = 1
    u = torch.full((d,), d ** -0.5, dtype=torch.float64)
    t = w[p + "dkv"].double()
    t[:rank] = 0.5 * t[:rank] + 40 * e[:, None] * to_k
    w[p + "dkv"] = t.to(torch.bfloat16)
    w[p + "dkv.norm"].fill_(1.0)
    reach = 14.0 / (m["scale"] * math.sqrt(rank))          # score 14 at c = sqrt(rank) e
    q = w[p + "q"].double().view(H, d + m["rot_dim"], -1) * 0.3
    q[:, :d] += math.sqrt(reach) * u[None, :, None] * to_q
    w[p + "q"] = q.reshape(H * (d + m["rot_dim"]), -1).to(torch.bfloat16)
    uk = w[p + "uk"].double().view(H, d, rank) * 0.5
    w[p + "uk"] = (uk + math.sqrt(reach) * u[None, :, None] * e).reshape(H * d, rank).to(torch.bfloat16)


def lasting_memory(cfg, w, *, write, read):
    """One recurrent layer and nothing else: only `write` enters the state, nothing is forgotten (the decays of a lightning layer say how little), and a
    lightning layer's state is asked for by `read` alone."""
    no_convolution(cfg, w)
    layer, p = cfg["layers"][0], "l0.mix."
    m, (to_write, to_read) = layer["mixer"], mark(cfg, w, write, read)
    if layer["type"] == "lightning":
        u = torch.full((m["heads"] * m["dim"],), 1.0, dtype=torch.float64)
        for name, to in (("q", to_read), ("k", to_write)):
            w[p + name] = (6 * u[:, None] * to).to(torch.bfloat16)
        return
    w[p + "z"] = (26 * torch.ones(m["width"], 1, dtype=torch.float64) * to_write).to(torch.bfloat16)
    w[p + "z.b"].fill_(-13.0)
    w[p + "x"] = (w[p + "x"].double() + 3 * torch.linspace(-1, 1, m["width"], dtype=torch.float64)[:, None] * to_write).to(torch.bfloat16)
