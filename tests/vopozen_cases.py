"""Small Vopozen configurations and weights for tests. Sublayers write about as much into the residual as the embedding, scores are loud and decays span
short and long memories, so that a key too many, a lost state or a missing factor shows in the logits. With random weights rounding flips
close choices of experts; ``sharp_routing`` makes models whose choices are never close: the last eight channels of the residual carry a code
of the token that no sublayer touches, and the router listens mostly to them. Keys of a time mixing resemble its receptances, so that no read-out
is a small difference of large terms before its norm."""
import math

import torch

import vopozen_oracle as oracle
from neuralfn_b200.models.vopozen import VopozenConfig, random_tensors

CODES = 8


def dense(ff=48):
    return {"kind": "dense", "ff": ff}


def moe(*, experts=8, top=3, ff=32, groups=(4, 2), shared=40, scale=1.7):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def attention(*, heads=4, kv_heads=2, dim=32, rot=16, base=1000.0, chunk=0, scale=0.3, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(*, heads=4, dim=24, rot=8, vdim=40, rank=48, base=500.0, window=0, scale=0.4, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def wkv(*, heads=3, dim=24, rank=12, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank_decay": rank}, "mlp": mlp}


def model(layers, *, vocab=96, width=64, eps=1e-5, mult=0.7, seed=0):
    cfg = {"architecture": "Vopozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    w = random_tensors(VopozenConfig.from_dict(cfg), seed)
    for i, y in enumerate(layers):
        if y["type"] == "wkv":
            p = f"l{i}.mix."
            w[p + "k"] = (0.85 * w[p + "r"].float() + 0.5 * w[p + "k"].float()).to(torch.bfloat16)
            w[p + "mu.k"] = (0.7 * w[p + "mu.r"].float() + 0.3 * w[p + "mu.k"].float()).to(torch.bfloat16)
            w[p + "u"] = (w[p + "u"].float() + 0.5).to(torch.bfloat16)
    if any((y["mlp"] or {}).get("kind") == "moe" for y in layers):
        sharp_routing(cfg, w, seed)
    return cfg, w


def tokens_of(cfg, n, *, seed, below=None):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, below or cfg["vocab"], (n,), generator=g).tolist()


def sharp_routing(cfg, w, seed=0, gap=0.04):
    width = cfg["width"]
    w["embed"][:, width - CODES:] = 3.0 * torch.eye(CODES, dtype=torch.bfloat16)[torch.arange(cfg["vocab"]) % CODES]
    for i, layer in enumerate(cfg["layers"]):
        w[f"l{i}.norm1"][width - CODES:] = 0
        mlp = layer["mlp"]
        if not mlp:
            continue
        w[f"l{i}.norm2"][width - CODES:] = 0
        if mlp["kind"] != "moe":
            continue
        E = mlp["router"]["experts"]
        for s in range(10_000):
            g = torch.Generator().manual_seed(1000 * seed + 7 * i + 131 * s)
            levels = torch.linspace(-2, 2, E) if E > 1 else torch.zeros(1)
            z = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(CODES)])          # [codes, experts]
            corr = (torch.randn(E, generator=g) * 0.3 - 0.6).to(torch.bfloat16)                       # choice scores of either sign
            if min(oracle.routing_gap(torch.sigmoid(r.double()), corr.double(), mlp["router"]) for r in z) > gap:
                break
        else:
            raise AssertionError("no clear choice of experts found")
        r = 0.002 * torch.randn(E, width, generator=g)
        r[:, width - CODES:] = z.T / 3.0
        w[f"l{i}.mlp.router"], w[f"l{i}.mlp.correction"] = r.to(torch.bfloat16), corr


def finder(cfg, w, token):
    """v with v . embed[token] = 1 and v . embed[other] = 0 (as many tokens as channels at most)."""
    e = w["embed"].double()
    return torch.linalg.lstsq(e, torch.eye(cfg["vocab"], dtype=torch.float64)[:, token:token + 1]).solution[:, 0]


def boost_needle(cfg, w, *, query, key):
    """One attention or latent layer and nothing else: the score of `query` on `key` towers over the others in every head, in dimensions that do not
    turn, and the value of `key` is loud."""
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    to_q, to_k = finder(cfg, w, query), finder(cfg, w, key)
    H, d = m["heads"], m["dim"]
    if cfg["layers"][0]["type"] == "attention":
        u = torch.zeros(d, dtype=torch.float64)
        u[m["rot"]["dims"]:] = (d - m["rot"]["dims"]) ** -0.5
        for name, heads, to in (("q", H, to_q), ("k", m["kv_heads"], to_k)):
            t = w[p + name].double().view(heads, d, -1) * 0.3
            w[p + name] = (t + 30 * u[None, :, None] * to).reshape(heads * d, -1).to(torch.bfloat16)
            w[p + name + ".norm"].fill_(1.0)               # the needle's score is then dim * scale
        return
    rank, e = m["kv_rank"], torch.zeros(m["kv_rank"], dtype=torch.float64)
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
    """One wkv layer and nothing else: only `write` enters the state, nothing decays, and `read` asks for it."""
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    H, d = m["heads"], m["dim"]
    u = torch.full((H * d,), d ** -0.5, dtype=torch.float64)
    for name, token in (("r", read), ("k", write)):
        w[p + name] = (6 * u[:, None] * finder(cfg, w, token)).to(torch.bfloat16)
        w[p + f"mu.{name}"].zero_()
    w[p + "w1"].zero_()
    w[p + "w0"].fill_(-14.0)
