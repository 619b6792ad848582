"""Kernels of the layer-list engine's newer mechanisms against plain PyTorch: paged attention with kept first tokens, a soft cap and a sink;
the gated delta rule; residual streams; routed experts."""
import math

import pytest
import torch

from neuralfn_b200.ops import layered as Y, paged as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def close(got, want, tol):
    assert torch.isfinite(got).all()
    assert float((got.float() - want).abs().max()) < tol * float(want.abs().max() + 1e-3)


def attend(q, k, v, pos, *, scale, window, keep, cap, sink):
    """q [R, H, d] at positions pos [R] over k [n, G, d], v [n, G, dv]."""
    rep = q.shape[1] // k.shape[1]
    j = torch.arange(k.shape[0], device=q.device)
    dist = pos[:, None] - j[None]
    seen = (dist >= 0) & ((dist < window) | (j[None] < keep) if window else torch.ones_like(dist, dtype=torch.bool))
    s = torch.einsum("rhd,nhd->hrn", q.double(), k.double().repeat_interleave(rep, 1)) * scale
    s = cap * torch.tanh(s / cap) if cap else s
    s = s.masked_fill(~seen, -math.inf)
    if sink:
        s = torch.cat([s, torch.zeros_like(s[..., :1])], -1)
    p = torch.softmax(s, -1)[..., :k.shape[0]]
    return torch.einsum("hrn,nhd->rhd", p, v.double().repeat_interleave(rep, 1)).reshape(q.shape[0], -1).float()


def problem(heads, kv_heads, dim, vdim, lengths, dtype=torch.bfloat16, seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    c = P.PagedCache(len(lengths), max(lengths), kv_heads, dim, vdim, DEV, dtype, seed)
    kv = []
    for s, n in enumerate(lengths):
        k, v = (torch.randn(n, kv_heads, w, generator=g, device=DEV).to(dtype).float() for w in (dim, vdim))
        c.write(s, k, v)
        kv.append((k, v))
    return c, kv, g


VARIANTS = [dict(window=0, keep=0, cap=5.0, sink=True), dict(window=100, keep=7, cap=0.0, sink=True), dict(window=64, keep=64, cap=3.0, sink=True),
            dict(window=1, keep=70, cap=8.0, sink=False), dict(window=200, keep=1, cap=5.0, sink=True), dict(window=30, keep=400, cap=0.0, sink=False)]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(8, 2, 128, 128), (4, 4, 16, 32), (12, 1, 64, 80), (40, 2, 96, 48), (4, 2, 256, 208)])
@pytest.mark.parametrize("variant", range(len(VARIANTS)))
def test_attention_rows(heads, kv_heads, dim, vdim, variant, dtype):
    o = VARIANTS[variant]
    lengths = [1500, 3, 64, 65, 900]
    c, kv, g = problem(heads, kv_heads, dim, vdim, lengths, dtype)
    rows = [(s, n - 1) for s, n in enumerate(lengths)] + [(0, 700), (4, 128), (-1, 0)]
    slot, pos = (torch.tensor([r[i] for r in rows], dtype=torch.int32, device=DEV) for i in (0, 1))
    q = torch.randn(len(rows), heads * dim, generator=g, device=DEV).to(dtype)
    scale = 3 * dim ** -0.5
    out = torch.zeros(len(rows), heads * vdim, device=DEV, dtype=dtype)
    for _ in range(2):      # the counters of the split form are left ready
        P.attention_rows(c, q, slot, pos, out, heads=heads, window=o["window"], scale=scale, keep_first=o["keep"], softcap=o["cap"], sink=o["sink"], max_keys=1500)
        for r, (s, p) in enumerate(rows):
            if s >= 0:
                close(out[r:r + 1], attend(q[r:r + 1].float().view(1, heads, dim), *kv[s], pos[r:r + 1].long(), scale=scale, **o), 0.02 if dtype == torch.bfloat16 else 2e-5)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(8, 2, 128, 128), (4, 4, 16, 32), (12, 1, 64, 80), (6, 2, 96, 48), (4, 2, 256, 240)])
@pytest.mark.parametrize("variant", range(len(VARIANTS)))
def test_attention_tiles(heads, kv_heads, dim, vdim, variant):
    o = VARIANTS[variant]
    lengths = [1100, 70, 64, 300]
    c, kv, g = problem(heads, kv_heads, dim, vdim, lengths, seed=1)
    step, parts = P.tile_rows(c, heads), [(0, 900, 200), (1, 0, 70), (2, 17, 47), (3, 299, 1)]     # slot, first position, rows
    tiles, base = [], 0
    for s, p0, n in parts:
        tiles += [[base + r, min(step, n - r), s, p0 + r] for r in range(0, n, step)]
        base += n
    q = torch.randn(base, heads * dim, generator=g, device=DEV).bfloat16()
    scale = 3 * dim ** -0.5
    out = torch.zeros(base, heads * vdim, device=DEV, dtype=torch.bfloat16)
    P.attention_tiles(c, q, torch.tensor(tiles, dtype=torch.int32, device=DEV), out, heads=heads, window=o["window"], scale=scale, keep_first=o["keep"], softcap=o["cap"], sink=o["sink"])
    from neuralfn_b200.ops import _lib
    _lib.assert_status_ok("paged tiles")
    base = 0
    for s, p0, n in parts:
        close(out[base:base + n], attend(q[base:base + n].float().view(n, heads, dim), *kv[s], torch.arange(p0, p0 + n, device=DEV), scale=scale, **o), 0.02)
        base += n


def rule(q, k, v, z, beta, rate, dim, S):
    """One sequence in float64: q, k [T, H, d], v [T, H, dv], z (decay + bias) [T, H, d], beta [T, H], S [H, d, dv] -> o, S."""
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)  # noqa: E731
    q, k = unit(q) * dim ** -0.5, unit(k)
    g = torch.exp(-torch.exp(rate)[None, :, None] * torch.nn.functional.softplus(z, threshold=40))
    out = []
    for t in range(q.shape[0]):
        S = g[t][..., None] * S
        u = torch.sigmoid(beta[t])[:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][..., None] * u[:, None]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_problem(heads, kv_heads, dim, vdim, lengths, dtype, seed, speed):
    """lengths: (slot, rows, position of the first one). Memory that spans thousands of tokens (slow), a few (fast), or both by channel."""
    g = torch.Generator(device=DEV).manual_seed(seed)
    up = lambda n: (n + 15) // 16 * 16  # noqa: E731
    dp, vp, R = up(dim), up(vdim), sum(n for _, n, _ in lengths)
    randn = lambda *s: torch.randn(*s, generator=g, device=DEV)  # noqa: E731
    q, k, v = randn(R, kv_heads, dim), randn(R, kv_heads, dim), randn(R, heads, vdim)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).reshape(R, -1)  # noqa: E731
    qkv = torch.cat([pad(q, dp), pad(k, dp), pad(v, vp)], 1).to(dtype).contiguous()
    beta, decay = randn(R, up(heads)).to(dtype), randn(R, heads * dp)
    a_log = (0.3 * randn(heads) + {"slow": -7.0, "mixed": -1.0, "fast": 2.0}[speed]).bfloat16()
    dt = (randn(heads * dp) * (4.0 if speed == "mixed" else 0.5)).bfloat16()
    slots = max(s for s, _, _ in lengths) + 2
    state = torch.zeros(slots, heads, dp, vp, device=DEV)
    state[:, :, :dim, :vdim] = randn(slots, heads, dim, vdim)
    seqs, at = [], 0
    for s, n, p in lengths:
        seqs.append([at, n, s, p])
        at += n
    return qkv, beta, decay, a_log, dt, state, torch.tensor(seqs, dtype=torch.int32, device=DEV), dp, vp


@pytest.mark.parametrize("speed", ["slow", "mixed", "fast"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 64, 64), (2, 1, 128, 128), (3, 3, 40, 24), (1, 1, 16, 16), (2, 2, 192, 80), (2, 1, 300, 48)])
@pytest.mark.parametrize("form,dtype", [("rows", torch.float32), ("rows", torch.bfloat16), ("chunks", torch.bfloat16), ("rounds", torch.bfloat16)])
def test_delta_rule(heads, kv_heads, dim, vdim, form, dtype, speed):
    lengths = [(0, 150, 0), (2, 16, 33), (1, 37, 1), (4, 64, 0), (3, 81, 500)] if form != "rows" else [(0, 70, 0), (2, 1, 33), (1, 7, 1), (4, 1, 0), (3, 16, 500)]
    qkv, beta, decay, a_log, dt, state, seqs, dp, vp = delta_problem(heads, kv_heads, dim, vdim, lengths, dtype, 3, speed)
    if form != "rows" and dp > 256:
        pytest.skip("wider heads go token after token")
    ws = None
    if form == "rounds":                                        # room for two chunks of every sequence: many rounds
        dk = 64 if dp <= 64 else 128 if dp <= 128 else 256
        ws, form = torch.empty(2 * len(lengths) * heads * (196 * dk + 128 * vp), device=DEV, dtype=torch.uint8), "chunks"
    before = state.double().clone()
    o = Y.delta_rule(qkv, beta, decay, a_log, dt, state, seqs, kv_heads=kv_heads, dim=dim, form=form, workspace=ws, longest=150)
    from neuralfn_b200.ops import _lib
    _lib.assert_status_ok("delta rule")
    idle = torch.tensor([[0, 1, -1, 5]], dtype=torch.int32, device=DEV)
    Y.delta_rule(qkv, beta, decay, a_log, dt, state, idle, kv_heads=kv_heads, dim=dim, form=form)       # padding: nothing happens
    rep, x = heads // kv_heads, qkv.double()
    tol = 2e-5 if form == "rows" else 1e-4                        # chunks: sixteen bits of every factor
    for at, n, slot, pos in seqs.tolist():
        r = slice(at, at + n)
        q, k = (x[r, i * kv_heads * dp:(i + 1) * kv_heads * dp].view(n, kv_heads, dp).repeat_interleave(rep, 1) for i in (0, 1))
        v = x[r, 2 * kv_heads * dp:].view(n, heads, vp)
        z = (decay[r].double() + dt.double()).view(n, heads, dp)
        want, S = rule(q, k, v, z, beta[r, :heads].double(), a_log.double(), dim, before[slot] if pos else torch.zeros_like(before[slot]))
        close(o[r], want.reshape(n, -1).float(), tol)
        close(state[slot], S.float(), tol)
    untouched = [s for s in range(state.shape[0]) if s not in seqs[:, 2].tolist()]
    assert torch.equal(state[untouched].double(), before[untouched])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_delta_out(dtype):
    g = torch.Generator(device=DEV).manual_seed(0)
    for heads, vdim, vp in ((3, 40, 48), (4, 128, 128), (2, 200, 208)):
        o, gate = torch.zeros(37, heads, vp, device=DEV), torch.randn(37, heads * vp, generator=g, device=DEV).to(dtype)
        o[..., :vdim] = torch.randn(37, heads, vdim, generator=g, device=DEV) * 0.1
        w = torch.randn(vp, generator=g, device=DEV).bfloat16()
        got = Y.delta_out(o.view(37, -1), gate, w, heads=heads, vdim=vdim, eps=1e-3)
        want = o / torch.sqrt((o * o).sum(-1, keepdim=True) / vdim + 1e-3) * w.float() * torch.sigmoid(gate.float().view(37, heads, vp))
        close(got, want.view(37, -1), 1e-5 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 6, 11])
@pytest.mark.parametrize("width,ld", [(40, 48), (1000, 1008), (4096, 4096)])
def test_stream_pass(width, ld, streams, dtype):
    g = torch.Generator(device=DEV).manual_seed(width + streams)

    def rows(*shape, dt=torch.float32):
        t = torch.zeros(*shape, ld, device=DEV, dtype=dt)
        t[..., :width] = torch.randn(*shape, width, generator=g, device=DEV).to(dt)
        return t

    coef = lambda *s: torch.randn(*s, generator=g, device=DEV).bfloat16()  # noqa: E731
    x, ys, w = rows(7, streams), rows(21, dt=dtype), rows(1, dt=torch.bfloat16)[0]
    mix, out, into = coef(streams, streams), coef(streams), coef(streams)
    index = torch.randperm(21, generator=torch.Generator().manual_seed(1)).int().to(DEV)
    src = torch.tensor([6, 0, 3, 3, 1], dtype=torch.int32, device=DEV)
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    for y_rows, y_index, pick in ((1, None, None), (3, None, None), (3, index, src), (2, index, None)):
        n = 7 if pick is None else 5
        h, xo = torch.empty(n, ld, device=DEV, dtype=dtype), torch.empty(n, streams, ld, device=DEV)
        Y.stream_pass(x, h, width=width, streams=streams, rows=n, ld=ld, f32=dtype == torch.float32, weight=w, eps=1e-3, weight_offset=1.0, x_out=xo, src_rows=pick, y=ys,
                      y_rows=y_rows, y_index=y_index, mix=mix, out=out, into=into)
        at = torch.arange(7, device=DEV) if pick is None else pick.long()
        items = at[:, None] * y_rows + torch.arange(y_rows, device=DEV)
        y = ys.double()[items if y_index is None else y_index.long()[items]].sum(1)
        want = torch.einsum("st,rsw->rtw", mix.double(), x.double()[at]) + out.double()[None, :, None] * y[:, None]
        u = torch.einsum("s,rsw->rw", into.double(), want)
        close(xo, want.float(), 2e-5)
        close(h, (u / torch.sqrt((u * u).sum(-1, keepdim=True) / width + 1e-3) * (1 + w.double())).float(), tol)
    # start (all streams are the scaled embedding) and end (the plain sum, nothing stored)
    emb, tok, h = rows(9, dt=torch.bfloat16), torch.tensor([3, 8, 0], dtype=torch.int32, device=DEV), torch.empty(3, ld, device=DEV, dtype=dtype)
    xo = torch.empty(3, streams, ld, device=DEV)
    Y.stream_pass(None, h, width=width, streams=streams, rows=3, ld=ld, f32=dtype == torch.float32, weight=w, eps=1e-3, x_out=xo, tokens=tok, embed=emb, embed_scale=2.5)
    e = emb.double()[tok.long()] * 2.5
    close(xo, e[:, None].expand(-1, streams, -1).float(), 1e-6)
    u = e * streams
    close(h, (u / torch.sqrt((u * u).sum(-1, keepdim=True) / width + 1e-3) * w.double()).float(), tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,experts,top", [(1, 4, 1), (3, 16, 2), (40, 6, 6), (130, 8, 3), (5, 300, 40), (64, 1, 1)])
def test_expert_rows(rows, experts, top, dtype):
    g = torch.Generator(device=DEV).manual_seed(rows)
    width, ff = 272, 144
    h, z = torch.randn(rows, width, generator=g, device=DEV).to(dtype), torch.randn(rows, experts, generator=g, device=DEV)
    if rows > 1:
        z[1] = z[1].round()                                     # ties: the lower index
    wg, wd = (torch.randn(experts, *s, generator=g, device=DEV).bfloat16() * s[1] ** -0.5 for s in ((2 * ff, width), (width, ff)))
    idx, weight, y = Y.expert_rows(h, z, wg, wd, experts=experts, top=top)
    order = torch.sort(-z.double() + torch.arange(experts, device=DEV) * 1e-9, dim=1).indices[:, :top]
    assert torch.equal(idx.long(), order)
    close(weight, torch.sigmoid(torch.gather(z, 1, order)), 1e-6)
    for j in range(top):
        a = h.double() * torch.sigmoid(torch.gather(z.double(), 1, order[:, j:j + 1]))
        gu = torch.einsum("rk,rnk->rn", a, wg.double()[order[:, j]])
        want = torch.einsum("rf,rnf->rn", torch.nn.functional.silu(gu[:, :ff]) * gu[:, ff:], wd.double()[order[:, j]])
        close(y[:, j], want.float(), 2e-5 if dtype == torch.float32 else 1e-2)


def test_logit_cap():
    x = torch.randn(5, 64, device=DEV) * 30
    want = 12.0 * torch.tanh(x.double() * 0.7 / 12.0)
    y = x.clone()
    Y.logit_cap(y, 0.7, 12.0)
    close(y, want.float(), 1e-6)
    Y.logit_cap(x, 0.5, 0.0)
