"""Plain reference of the Bulidra decoder for tests: one function per mechanism, whole sequences at once, float64 by default, no cache
and no code shared with the framework. Configurations are the plain dictionaries of a ``config.json``, weights a name -> tensor map."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def short_conv(u, w):
    """u [T, C], w [C, taps]: y[t] = sum_j w[:, j] u[t - taps + 1 + j], zeros before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def query_temperature(pos, coef, every):
    return 1 + coef * math.log(math.floor((pos + 1) / every) + 1)


def slopes(heads):
    return [2.0 ** (-8 * (h + 1) / heads) for h in range(heads)]


def windowed_attention(q, k, v, *, scale, window, slope):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; key j of query i when 0 <= i - j < window."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        dist = torch.tensor([i - j for j in range(lo, i + 1)], dtype=q.dtype)
        for h in range(H):
            s = k[lo:i + 1, h // rep] @ q[i, h] * scale - slope[h] * dist
            out[i, h] = torch.softmax(s, 0) @ v[lo:i + 1, h // rep]
    return out


def project_kv(h, W, p, m):
    """Keys and values of a layer that owns them, as later layers reuse them."""
    G = m["kv_heads"]
    k = short_conv(h @ W[p + "mix.k"].T, W[p + "mix.k.conv"])
    v = short_conv(h @ W[p + "mix.v"].T, W[p + "mix.v.conv"])
    return k.view(-1, G, m["dim"]), v.view(-1, G, m["vdim"])


def attention_mixer(h, W, p, m, kv):
    T = h.shape[0]
    q = short_conv(h @ W[p + "mix.q"].T, W[p + "mix.q.conv"])
    if m.get("q_temp"):
        f = [query_temperature(i, m["q_temp"]["coef"], m["q_temp"]["every"]) for i in range(T)]
        q = q * torch.tensor(f, dtype=h.dtype)[:, None]
    k, v = kv
    o = windowed_attention(q.view(T, m["heads"], m["dim"]), k, v, scale=m["scale"], window=(m.get("mask") or {}).get("size", 0), slope=slopes(m["heads"]))
    o = o.reshape(T, -1) * torch.sigmoid(h @ W[p + "mix.g"].T)
    return o @ W[p + "mix.o"].T


def feed_forward(h, W, p):
    return (torch.relu(h @ W[p + "mlp.gate"].T) * (h @ W[p + "mlp.up"].T)) @ W[p + "mlp.down"].T


def side_input(x, tokens, W, p, layer, dim, eps):
    e = W["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return x + rms(y, eps) * W[p + "side.norm"]


def forward(cfg, weights, tokens, dtype=torch.float64):
    """-> logits [T, vocab], residual streams after every layer [layers, T, width]."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = W["embed"][tokens] * cfg["embedding"]["scale"]
    kvs, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms(x, eps) * W[p + "norm1"]
        src = m.get("kv_from")
        if src is None:
            kvs[i] = project_kv(h, W, p, m)
        y = attention_mixer(h, W, p, m, kvs[i if src is None else src])
        if layer.get("mlp"):
            y = y + feed_forward(h, W, p)
        x = x + y
        if cfg.get("token_side"):
            x = side_input(x, tokens, W, p, i, cfg["token_side"]["dim"], eps)
        after.append(x)
    logits = (rms(x, eps) * W["final.norm"]) @ W["embed"].T
    return logits, torch.stack(after)
