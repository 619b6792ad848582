"""Plain reference of the Murilorn decoder for tests: one function per mechanism, whole sequences at once, float64 by default, no cache and
no code shared with the framework. Configurations are the plain dictionaries of a ``config.json``, weights a name -> tensor map."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def short_conv(u, w):
    """u [T, C], w [C, taps]: y[t] = sum_j w[:, j] u[t - taps + 1 + j], zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decays(h, W, p, heads, dim):
    """[T, heads, dim]: factor of every key channel's state row before the token is written."""
    z = (h @ W[p + "mix.a1"].T) @ W[p + "mix.a2"].T + W[p + "mix.dt_bias"]
    soft = torch.where(z > 30, z, torch.log1p(torch.exp(z.clamp(max=30))))
    return torch.exp(-torch.exp(W[p + "mix.A_log"])[None, :, None] * soft.view(-1, heads, dim))


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H] -> [T, H, dv]; one token after another."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        seen = (S * k[t][:, :, None]).sum(1)
        u = beta[t][:, None] * (v[t] - seen)
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def delta_mixer(h, W, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ W[p + f"mix.{n}"].T, W[p + f"mix.{n}.conv"])) for n in "qkv")
    q, k = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d))
    of_head = [x // (H // G) for x in range(H)]
    beta = torch.sigmoid(h @ W[p + "mix.b"].T)
    o = delta_rule(q[:, of_head], k[:, of_head], v.view(T, H, dv), decays(h, W, p, H, d), beta)
    gate = torch.sigmoid((h @ W[p + "mix.g1"].T) @ W[p + "mix.g2"].T).view(T, H, dv)
    o = rms(o, eps) * W[p + "mix.norm"] * gate
    return o.reshape(T, -1) @ W[p + "mix.o"].T


def visible(i, size, keep):
    """Keys of position i: the first `keep` tokens and the last `size` ones (0: all)."""
    return [j for j in range(i + 1) if not size or i - j < size or j < keep]


def softmax_with_sink(s):
    """Over the scores of a row and one more of 0, whose share is lost."""
    top = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention_mixer(h, W, p, m):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[p + f"mix.{n}"].T + W[p + f"mix.{n}.b"] for n in "qkv")
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    mask = m.get("mask") or {}
    cap = m.get("softcap")
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    seen = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        seen[i, visible(i, mask.get("size", 0), mask.get("keep_first", 0))] = True
    for x in range(H):
        g = x // (H // G)
        s = q[:, x] @ k[:, g].T * m["scale"]
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(~seen, -math.inf)
        out[:, x] = softmax_with_sink(s) @ v[:, g]
    return out.reshape(T, -1) @ W[p + "mix.o"].T


def experts(h, W, p, mlp):
    z = h @ W[p + "mlp.router"].T
    s = 1 / (1 + torch.exp(-z))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(s[t], mlp["router"]["top"]).indices.tolist():
            a = s[t, e] * h[t]
            f = p + f"mlp.e{e}."
            out[t] += W[f + "down"] @ (silu(W[f + "gate"] @ a) * (W[f + "up"] @ a))
    return out


def routing_gap(z, top):
    """Smallest distance between a chosen and a left-out expert's logit over the rows (infinite when all are chosen)."""
    if top == z.shape[1]:
        return math.inf
    v = torch.sort(z, -1, descending=True).values
    return float((v[:, top - 1] - v[:, top]).min())


def mixed_in(xs, W, p):
    return sum(W[p + "in"][s] * x for s, x in enumerate(xs))


def mixed_out(xs, y, W, p):
    n = len(xs)
    return [sum(W[p + "mix"][s, t] * xs[s] for s in range(n)) + W[p + "out"][t] * y for t in range(n)]


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, weights, tokens, dtype=torch.float64, gaps=None):
    """-> logits [T, vocab], residual (sum of the streams) after every layer run [runs, T, width]. gaps: a list that receives the routing
    gap of every layer run."""
    W = {k: v.to(dtype) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = W["embed"][tokens] * cfg["embedding"]["scale"]
    hyper = bool(cfg.get("streams"))
    xs = [x] * (cfg.get("streams") or 1)
    after = []
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        for q, what in ((1, "mix"), (2, "mlp")):
            if what == "mlp" and not layer.get("mlp"):
                continue
            u = mixed_in(xs, W, p + f"hc{q}.") if hyper else xs[0]
            h = centred_norm(u, W[p + f"norm{q}"], eps)
            if what == "mlp":
                y = experts(h, W, p, layer["mlp"])
                if gaps is not None:
                    gaps.append(routing_gap(h @ W[p + "mlp.router"].T, layer["mlp"]["router"]["top"]))
            elif layer["type"] == "channel_delta":
                y = delta_mixer(h, W, p, layer["mixer"], eps)
            else:
                y = attention_mixer(h, W, p, layer["mixer"])
            xs = mixed_out(xs, y, W, p + f"hc{q}.") if hyper else [xs[0] + y]
        after.append(sum(xs))
    logits = centred_norm(sum(xs), W["final.norm"], eps) @ W["head"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return logits, torch.stack(after)
