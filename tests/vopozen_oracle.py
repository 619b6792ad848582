"""Plain reference of the Vopozen decoder for tests: one function per mechanism, whole sequences at once, float64 by default, no cache and
no code shared with the framework. Configurations are the plain dictionaries of a ``config.json``, weights a name -> tensor map."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def rotate(x, first, dims, base):
    """x [T, heads, n] at positions first, first + 1, ...: neighbouring dimensions (2i, 2i + 1) of the first `dims` turn by p * base^(-2i / dims)."""
    T = x.shape[0]
    out = x.clone()
    p = torch.arange(first, first + T, dtype=torch.float64)
    for i in range(dims // 2):
        a = p * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def in_chunk(i, j, size):
    return (j <= i) & (i // size == j // size)


def in_window(i, j, size):
    return (j <= i) & (i - j < size)


def seen(T, rule, size):
    """[T, T]: does query i see key j (size 0: every earlier key)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return rule(i, j, size) if size else j <= i


def size_of(m):
    return (m.get("mask") or {}).get("size", 0)


def attend(scores, mask, v):
    return torch.softmax(scores.masked_fill(~mask, -math.inf), -1) @ v


def attention_mixer(h, W, p, m, eps):
    """Grouped heads, normed and rotated queries and keys; the values are the keys as projected."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, v = (h @ W[p + "q"].T).view(T, H, d), (h @ W[p + "k"].T).view(T, G, d)
    q, k = norm(q, W[p + "q.norm"], eps), norm(v, W[p + "k.norm"], eps)
    q, k = (rotate(t, 0, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    mask = seen(T, in_chunk, size_of(m))
    out = torch.stack([attend(q[:, x] @ k[:, x // (H // G)].T * m["scale"], mask, v[:, x // (H // G)]) for x in range(H)], 1)
    return out.reshape(T, -1) @ W[p + "o"].T


def latent_of(h, W, p, m, eps):
    """What a latent layer caches: the normed latent [T, rank] and the rotated key part [T, rot_dim] all heads share."""
    z, r = h @ W[p + "dkv"].T, m["kv_rank"]
    return norm(z[:, :r], W[p + "dkv.norm"], eps), rotate(z[:, None, r:], 0, m["rot"]["dims"], m["rot"]["base"])[:, 0]


def latent_mixer(h, W, p, m, latent):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    c, kr = latent
    q = (h @ W[p + "q"].T).view(T, H, d + e)
    qr = rotate(q[..., d:], 0, m["rot"]["dims"], m["rot"]["base"])
    k, v = (c @ W[p + "uk"].T).view(T, H, d), (c @ W[p + "uv"].T).view(T, H, m["vdim"])
    mask = seen(T, in_window, size_of(m))
    out = torch.stack([attend((q[:, x, :d] @ k[:, x].T + qr[:, x] @ kr.T) * m["scale"], mask, v[:, x]) for x in range(H)], 1)
    return out.reshape(T, -1) @ W[p + "o"].T


def shifted(h):
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_decays(z, W, p):
    """Factor of every key channel's state row after the token's read-out, from the token's own mix of the input."""
    return torch.exp(-torch.exp(torch.tanh(z @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]))


def wkv_rule(r, k, v, w, u):
    """r, k, v, w [T, H, d], u [H, d]: read the old state plus the bonus of the token itself, then let it decay and write."""
    T, H, d = r.shape
    S, out = torch.zeros(H, d, d, dtype=r.dtype), torch.zeros_like(r)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1)
        S = w[t][:, :, None] * S + kv
    return out


def wkv_mixer(h, W, p, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    back = shifted(h)
    mix = {s: h + (back - h) * W[p + f"mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + s].T).view(T, H, d) for s in "rkv")
    o = wkv_rule(r, k, v, wkv_decays(mix["w"], W, p).view(T, H, d), W[p + "u"])
    return (rms(o, eps).reshape(T, -1) * W[p + "norm"] * silu(mix["g"] @ W[p + "g"].T)) @ W[p + "o"].T


def dense(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert(h, W, p):
    return relu_squared(h @ W[p + "up"].T) @ W[p + "down"].T


def allowed(choice, groups):
    """Which experts are open to the choice: those of the groups whose two best members add up to most."""
    n = choice.numel() // groups["count"]
    score = choice.view(-1, n).sort(-1, descending=True).values[:, :2].sum(-1)
    best = torch.sort(score, descending=True, stable=True).indices[:groups["keep"]]
    ok = torch.zeros(groups["count"], n, dtype=torch.bool)
    ok[best] = True
    return ok.view(-1)


def closed(choice, ok):
    return choice.masked_fill(~ok, -math.inf)


def route(s, correction, router):
    """One token: chosen experts and their weights."""
    choice = s + correction
    if router.get("groups"):
        choice = closed(choice, allowed(choice, router["groups"]))
    e = torch.topk(choice, router["top"]).indices
    return e, s[e] / (s[e].sum() + 1e-20) * router.get("scale", 1.0)


def routing_gap(s, correction, router):
    """Smallest distance by which a choice of the token could have gone the other way: between groups and between experts."""
    choice, gap = s + correction, math.inf
    g = router.get("groups")
    if g:
        n = choice.numel() // g["count"]
        score = choice.view(-1, n).sort(-1, descending=True).values[:, :2].sum(-1).sort(descending=True).values
        if g["keep"] < g["count"]:
            gap = float(score[g["keep"] - 1] - score[g["keep"]])
        choice = choice.masked_fill(~allowed(choice, g), -math.inf)
    v = choice.sort(descending=True).values
    if router["top"] < v.numel() and v[router["top"]] > -math.inf:
        gap = min(gap, float(v[router["top"] - 1] - v[router["top"]]))
    return gap


def experts(h, W, p, mlp, gaps=None):
    s = 1 / (1 + torch.exp(-(h @ W[p + "router"].T)))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        if gaps is not None:
            gaps.append(routing_gap(s[t], W[p + "correction"], mlp["router"]))
        for e, a in zip(*route(s[t], W[p + "correction"], mlp["router"])):
            out[t] += a * expert(h[t], W, p + f"e{int(e)}.")
    return out + expert(h, W, p + "shared.") if mlp.get("shared") else out


def forward(cfg, weights, tokens, dtype=torch.float64, gaps=None):
    """-> logits [T, vocab], residual after every layer [layers, T, width]. gaps: a list that receives the routing gap of every token and
    routed layer."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        if layer["type"] == "attention":
            y = attention_mixer(x, W, p + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_of(x, W, p + "mix.", m, eps)
            y = latent_mixer(x, W, p + "mix.", m, latents[i if src is None else src])
        else:
            y = wkv_mixer(x, W, p + "mix.", m, eps)
        x = x + mult * norm(y, W[p + "norm1"], eps)
        if mlp:
            y = dense(x, W, p + "mlp.") if mlp["kind"] == "dense" else experts(x, W, p + "mlp.", mlp, gaps)
            x = x + mult * norm(y, W[p + "norm2"], eps)
        after.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T, torch.stack(after)
