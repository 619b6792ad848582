"""Plain reference of the Kidolorn decoder for tests: one function per mechanism, whole sequences at once, float64 by default, no cache and no code
shared with the framework. Configurations are the plain dictionaries of a ``config.json``, weights a name -> tensor map."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def short_conv(h, w):
    """Causal convolution of every channel over time: h [T, width], w [width, taps]; the newest input meets the last tap."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for back in range(min(taps, T)):
        out[back:] = out[back:] + h[:T - back] * w[:, taps - 1 - back]
    return out


def sublayer_input(x, W, p, which, eps):
    """Norm with a single factor, then the row plus its convolution."""
    h = rms(x, eps) * W[f"{p}norm{which}"]
    return h + short_conv(h, W[f"{p}canon{which}"])


def linear_rule(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], one decay per head: write first, then read."""
    T, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[-1], dtype=q.dtype), torch.zeros_like(v)
    f = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    for t in range(T):
        S = f * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def lightning_mixer(h, W, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k = (silu(h @ W[p + n].T).view(T, H, m["dim"]) for n in "qk")
    v = silu(h @ W[p + "v"].T).view(T, H, m["vdim"])
    o = linear_rule(q, k, v, m["decay"]).reshape(T, -1)
    return (rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def gated_rule(z, c):
    """z, c [T, n]: every channel moves from its state towards the candidate by the share z."""
    S, out = torch.zeros_like(z[0]), torch.zeros_like(z)
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out


def mingru_mixer(h, W, p):
    z, u = sigmoid(h @ W[p + "z"].T + W[p + "z.b"]), h @ W[p + "x"].T + W[p + "x.b"]
    return (gated_rule(z, candidate(u)) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def rotate_half(x, dims, base):
    """x [T, heads, n] at positions 0, 1, ...: dimensions i and i + dims / 2 turn together by p * base^(-2i / dims)."""
    out, p = x.clone(), torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = p * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i], out[:, :, i + dims // 2] = u * c - v * s, v * c + u * s
    return out


def latent_of(h, W, p, m, eps):
    """What a latent layer caches: the normed latent [T, rank] and the rotated key part [T, rot_dim] all heads share."""
    z, r = h @ W[p + "dkv"].T, m["kv_rank"]
    return rms(z[:, :r], eps) * W[p + "dkv.norm"], rotate_half(z[:, None, r:], m["rot"]["dims"], m["rot"]["base"])[:, 0]


def sink_softmax(scores, sink):
    """Rows of weights whose sum leaves room for one more score without a value."""
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_mixer(h, W, p, m, latent):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    c, kr = latent
    q = (h @ W[p + "q"].T).view(T, H, d + e)
    qr = rotate_half(q[..., d:], m["rot"]["dims"], m["rot"]["base"])
    k, v = (c @ W[p + "uk"].T).view(T, H, d), (c @ W[p + "uv"].T).view(T, H, m["vdim"])
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    out = []
    for x in range(H):
        s = ((q[:, x, :d] @ k[:, x].T + qr[:, x] @ kr.T) * m["scale"]).masked_fill(later, -math.inf)
        out.append(sink_softmax(s, W[p + "sink"][x]) @ v[:, x])
    return (torch.stack(out, 1).reshape(T, -1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def clamped_gate(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def dense(h, W, p, limit):
    lin = lambda x, n: x @ W[p + n].T + W[p + n + ".b"]  # noqa: E731
    return lin(clamped_gate(lin(h, "gate"), lin(h, "up"), limit), "down")


def expert(h, W, p, limit):
    return clamped_gate(W[p + "gate"] @ h, W[p + "up"] @ h, limit) @ W[p + "down"].T


def route(z, top):
    """One token's router logits: the experts with the largest ones, and the softmax over these alone."""
    best = torch.topk(z, top)
    return best.indices, torch.softmax(best.values, 0)


def experts(h, W, p, mlp, gaps=None):
    z, top = h @ W[p + "router"].T, mlp["router"]["top"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        if gaps is not None and top < z.shape[1]:
            s = z[t].sort(descending=True).values
            gaps.append(float(s[top - 1] - s[top]))
        for e, a in zip(*route(z[t], top)):
            out[t] += a * expert(h[t], W, p + f"e{int(e)}.", mlp["expert"]["limit"])
    return out


def forward(cfg, weights, tokens, dtype=torch.float64, gaps=None):
    """-> logits [T, vocab], residual after every layer [layers, T, width]. gaps: a list that receives, per token and routed layer, how far the last
    chosen router logit lies above the first one left out."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = sublayer_input(x, W, p, 1, eps)
        if layer["type"] == "lightning":
            y = lightning_mixer(h, W, p + "mix.", m, eps)
        elif layer["type"] == "mingru":
            y = mingru_mixer(h, W, p + "mix.")
        else:
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_of(h, W, p + "mix.", m, eps)
            y = latent_mixer(h, W, p + "mix.", m, latents[i if src is None else src])
        x = x + rms(y, eps) * W[p + "norm1b"]
        if mlp:
            h = sublayer_input(x, W, p, 2, eps)
            y = dense(h, W, p + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else experts(h, W, p + "mlp.", mlp, gaps)
            x = x + rms(y, eps) * W[p + "norm2b"]
        after.append(x)
    return rms(x, eps) * W["final.norm"] @ W["head"].T, torch.stack(after)
