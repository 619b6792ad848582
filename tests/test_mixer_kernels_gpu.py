"""Kernels of rotated heads, chunk masks, latent attention, time mixing, output norms and grouped expert choice against plain PyTorch in float64."""
import math

import pytest
import torch

import vopozen_oracle as oracle
from neuralfn_b200.ops import layered as Y, paged as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
TOL = {torch.bfloat16: 0.02, torch.float32: 2e-5}
DTYPES = [torch.bfloat16, torch.float32]


def close(got, want, tol):
    assert torch.isfinite(got).all()
    assert float((got.double() - want.double()).abs().max()) < tol * float(want.abs().max() + 1e-3)


def gen(seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return lambda *s, dtype=torch.bfloat16: torch.randn(*s, generator=g, device=DEV).to(dtype)


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def spread_rows(parts, step):
    """(slot, first position, rows) -> tiles of `step` rows, total rows."""
    tiles, base = [], 0
    for s, p0, n in parts:
        tiles += [[base + r, min(step, n - r), s, p0 + r] for r in range(0, n, step)]
        base += n
    return ints(tiles), base


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,rot,values", [(4, 2, 64, 32, True), (5, 1, 24, 10, True), (3, 3, 144, 144, False), (2, 1, 300, 100, True), (8, 8, 16, 0, False)])
def test_head_rows(heads, kv, dim, rot, values, dtype):
    """Norm, rotation at near and far positions, keys and values in their pages."""
    rnd = gen()
    dp = (dim + 15) // 16 * 16
    entries = [(0, 5, 1, 0), (1, 100_003, 37, 0), (2, 0, 18, 0)]
    n = sum(e[2] for e in entries)
    c = P.PagedCache(3, 100_096, kv, dp, dp, DEV, dtype)
    x = torch.zeros(n, (heads + (1 if values else 2) * kv) * dp, device=DEV, dtype=dtype)
    x.view(n, -1, dp)[..., :dim] = rnd(n, x.shape[1] // dp, dim, dtype=dtype)
    qn, kn = rnd(dp), rnd(dp)
    q = torch.zeros(n, heads * dp, device=DEV, dtype=dtype)
    Y.head_rows(c, x, P.row_tiles(entries, DEV), q, heads=heads, dim=dim, freq=Y.frequencies(rot, 1234.5, DEV) if rot else None, rot_dims=rot, eps=1e-5, q_norm=qn, k_norm=kn, key_values=values)
    raw, base = x.double().cpu().view(n, -1, dp), 0
    tol = 0.01 if dtype == torch.bfloat16 else 3e-6
    for slot, p0, rows, _ in entries:
        part = raw[base:base + rows]
        for got, want, w in ((q.view(n, heads, dp)[base:base + rows], part[:, :heads], qn), (None, part[:, heads:heads + kv], kn)):
            ref = oracle.rotate(oracle.norm(want[..., :dim], w[:dim].double().cpu(), 1e-5), p0, rot, 1234.5)
            if got is None:
                got = torch.stack([c.k[int(c.table[slot, p // 64]), :, p % 64] for p in range(p0, p0 + rows)])
            close(got[..., :dim].cpu(), ref, tol)
        v = torch.stack([c.v[int(c.table[slot, p // 64]), :, :, p % 64] for p in range(p0, p0 + rows)])
        assert torch.equal(v.double().cpu(), part[:, heads:heads + kv] if values else part[:, heads + kv:])
        base += rows


def chunk_attend(q, k, v, pos, scale, chunk):
    j = torch.arange(k.shape[0], device=DEV)
    seen = (j[None] <= pos[:, None]) & (j[None] // chunk == pos[:, None] // chunk)
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("rhd,nhd->hrn", q.double(), k.double().repeat_interleave(rep, 1)) * scale
    return torch.einsum("hrn,nhd->rhd", torch.softmax(s.masked_fill(~seen, -math.inf), -1), v.double().repeat_interleave(rep, 1)).reshape(q.shape[0], -1)


@pytest.mark.parametrize("chunk", [1, 50, 64, 200, 1024])
@pytest.mark.parametrize("heads,kv,dim", [(8, 2, 128), (6, 6, 48), (4, 2, 160)])
def test_chunked_attention(heads, kv, dim, chunk):
    rnd = gen(1)
    lengths = [1500, 130, 64]
    k = [rnd(n, kv, dim) for n in lengths]
    v = [rnd(n, kv, dim) for n in lengths]
    scale = 2 * dim ** -0.5
    for dtype in DTYPES:
        c = P.PagedCache(3, 1536, kv, dim, dim, DEV, dtype)
        for s in range(3):
            c.write(s, k[s], v[s])
        rows = [(0, 1499), (0, 1024), (0, 1023), (1, 0), (1, 129), (2, 63), (-1, 0)]
        slot, pos = ints([r[0] for r in rows]), ints([r[1] for r in rows])
        q, out = rnd(len(rows), heads * dim, dtype=dtype), torch.zeros(len(rows), heads * dim, device=DEV, dtype=dtype)
        P.attention_rows(c, q, slot, pos, out, heads=heads, scale=scale, chunk=chunk)
        for r, (s, p) in enumerate(rows[:-1]):
            close(out[r:r + 1], chunk_attend(q[r:r + 1].view(1, heads, dim), k[s], v[s], pos[r:r + 1], scale, chunk), TOL[dtype])
        if dtype == torch.bfloat16:
            parts = [(0, 990, 300), (1, 0, 130), (2, 17, 47)]
            tiles, n = spread_rows(parts, P.tile_rows(c, heads))
            q, out, base = rnd(n, heads * dim), torch.zeros(n, heads * dim, device=DEV, dtype=dtype), 0
            P.attention_tiles(c, q, tiles, out, heads=heads, scale=scale, chunk=chunk)
            for s, p0, m in parts:
                close(out[base:base + m], chunk_attend(q[base:base + m].view(m, heads, dim), k[s], v[s], torch.arange(p0, p0 + m, device=DEV), scale, chunk), 0.02)
                base += m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,groups,n,k", [(1, 3, 48, 16), (8, 5, 512, 128), (9, 4, 64, 528), (16, 2, 16, 48), (30, 1, 176, 336), (75, 6, 128, 64)])
def test_group_products(rows, groups, n, k, dtype):
    rnd = gen(2)
    x, w = rnd(rows, groups, k + 16, dtype=dtype)[..., :k], rnd(groups, n, k)
    out = torch.zeros(groups, rows, n, device=DEV, dtype=dtype).transpose(0, 1)
    Y.group_products(x, w, out)
    want = torch.einsum("rgk,gnk->rgn", x.double(), w.double())
    close(out, want, 0.01 if dtype == torch.bfloat16 else 2e-6)
    tail, got = rnd(n + 32, k), torch.zeros(rows, n + 32, device=DEV)
    Y.group_products(x, w, out, act=4, tail_w=tail, tail_out=got, tail_in=(groups - 1) * x.stride(1))
    close(out, oracle.relu_squared(want), 0.01 if dtype == torch.bfloat16 else 2e-6)
    close(got, x[:, -1].double() @ tail.double().T, 2e-6)


def latent_problem(rank, rot, lengths, dtype, seed=3):
    rnd = gen(seed)
    c = Y.LatentCache(len(lengths), max(lengths), rank, rot, DEV, dtype, seed)
    z = [rnd(n, rank + rot, dtype=dtype) for n in lengths]
    for s, t in enumerate(z):
        c.write(s, t)
    return c, z, rnd


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [0, 1, 70, 1000])
@pytest.mark.parametrize("heads,rank,rot", [(16, 512, 64), (5, 48, 16), (20, 128, 32), (40, 256, 48), (33, 272, 16), (3, 528, 16)])
def test_latent_attention_rows(heads, rank, rot, window, dtype):
    lengths = [1500, 3, 64, 65, 900]
    c, z, rnd = latent_problem(rank, rot, lengths, dtype)
    rows = [(s, n - 1) for s, n in enumerate(lengths)] + [(0, 700), (4, 128), (-1, 0)]
    slot, pos = ints([r[0] for r in rows]), ints([r[1] for r in rows])
    q, out = rnd(len(rows), heads * (rank + rot), dtype=dtype), torch.zeros(len(rows), heads * rank, device=DEV, dtype=dtype)
    scale = 3 * (rank + rot) ** -0.5
    for max_keys in (1500, 64):                          # many shares, one
        Y.latent_attention_rows(c, q, slot, pos, out, heads=heads, window=window, scale=scale, max_keys=max_keys)
        for r, (s, p) in enumerate(rows[:-1]):
            keys = z[s][max(0, p - window + 1) if window else 0:p + 1].double()
            w = torch.softmax(q[r].double().view(heads, -1) @ keys.T * scale, -1)
            close(out[r].view(heads, rank), w @ keys[:, :rank], TOL[dtype])


@pytest.mark.parametrize("window", [0, 1, 70, 1000])
@pytest.mark.parametrize("heads,dim,vdim,rank,rot", [(4, 128, 128, 512, 64), (3, 32, 48, 64, 16), (2, 80, 16, 128, 80), (5, 16, 208, 32, 32)])
def test_latent_attention_tiles(heads, dim, vdim, rank, rot, window):
    lengths = [1100, 70, 64, 300]
    c, z, rnd = latent_problem(rank, rot, lengths, torch.bfloat16, 4)
    uk, uv = rnd(heads, dim, rank) * rank ** -0.5, rnd(heads, vdim, rank) * rank ** -0.5
    parts = [(0, 900, 200), (1, 0, 70), (2, 17, 47), (3, 299, 1)]
    spans, base, at = [], [0] * 4, 0
    for s, p0, n in parts:
        first = (max(0, p0 - window + 1) if window else 0) // 64
        pages = (p0 + n - 1) // 64 + 1 - first
        spans.append([s, first, pages, at])
        base[s] = at - 64 * first
        at += 64 * pages
    lat = Y.latent_gather(c, ints(spans), torch.zeros(at, rank, device=DEV, dtype=torch.bfloat16))
    x = torch.cat([(lat.float() @ uk.reshape(-1, rank).float().T), lat.float() @ uv.reshape(-1, rank).float().T], 1).bfloat16()
    tiles, n = spread_rows(parts, 128)
    q, out = rnd(n, heads * (dim + rot)), torch.zeros(n, heads * vdim, device=DEV, dtype=torch.bfloat16)
    scale = 3 * (dim + rot) ** -0.5
    Y.latent_attention_tiles(c, q, x, ints(base), tiles, out, heads=heads, dim=dim, vdim=vdim, window=window, scale=scale)
    row = 0
    for s, p0, m in parts:
        lt, kr = z[s][:, :rank].float(), z[s][:, rank:].double()
        k, v = ((lt @ w.reshape(-1, rank).float().T).bfloat16().double().view(-1, heads, w.shape[1]) for w in (uk, uv))
        i, j = torch.arange(p0, p0 + m, device=DEV)[:, None], torch.arange(lt.shape[0], device=DEV)[None]
        seen = (j <= i) & (i - j < window if window else j <= i)
        qq = q[row:row + m].double().view(m, heads, dim + rot)
        sc = (torch.einsum("rhd,nhd->hrn", qq[..., :dim], k) + torch.einsum("rhd,nd->hrn", qq[..., dim:], kr)) * scale
        want = torch.einsum("hrn,nhd->rhd", torch.softmax(sc.masked_fill(~seen, -math.inf), -1), v).reshape(m, -1)
        close(out[row:row + m], want, 0.02)
        row += m


def test_latent_rows_norm_and_rotation():
    rnd = gen(5)
    heads, dim, rot_dim, rot, rank, rank_p = 3, 32, 10, 16, 40, 48
    c = Y.LatentCache(2, 4096, rank_p, rot, DEV, torch.float32)
    entries = [(0, 130, 3, 0), (1, 3001, 40, 0)]          # short rows come first
    x = torch.zeros(43, heads * (dim + rot) + rank_p + rot, device=DEV)
    x[:, :heads * (dim + rot)].view(43, heads, dim + rot)[..., :dim + rot_dim] = rnd(43, heads, dim + rot_dim, dtype=torch.float32)
    x[:, heads * (dim + rot):][:, :rank] = rnd(43, rank, dtype=torch.float32)
    x[:, heads * (dim + rot) + rank_p:][:, :rot_dim] = rnd(43, rot_dim, dtype=torch.float32)
    before, w = x.clone().double().cpu(), rnd(rank_p)
    q_lat = torch.zeros(3, heads * (rank_p + rot), device=DEV)
    Y.latent_rows(c, x, P.row_tiles(entries, DEV), heads=heads, dim=dim, rot_dim=rot_dim, rank=rank, c_norm=w, eps=1e-5, freq=Y.frequencies(rot_dim, 300.0, DEV), q_row0=3, q_lat=q_lat)
    base = 0
    for slot, p0, n, _ in entries:
        rows = before[base:base + n]
        q = rows[:, :heads * (dim + rot)].view(n, heads, dim + rot)
        turned = oracle.rotate(q[..., dim:], p0, rot_dim, 300.0)
        got = q_lat.view(3, heads, -1)[..., rank_p:] if base == 0 else x[base:base + n, :heads * (dim + rot)].view(n, heads, dim + rot)[..., dim:]
        close(got.cpu(), turned, 2e-6)
        kv = rows[:, heads * (dim + rot):]
        page = torch.stack([c.k[int(c.table[slot, p // 64]), 0, p % 64] for p in range(p0, p0 + n)]).cpu()
        close(page[:, :rank], oracle.norm(kv[:, :rank], w[:rank].double().cpu(), 1e-5), 2e-6)
        close(page[:, rank_p:], oracle.rotate(kv[:, None, rank_p:], p0, rot_dim, 300.0)[:, 0], 2e-6)
        base += n


def wkv_problem(heads, dim, lengths, dtype, seed=6):
    rnd = gen(seed)
    dp, n = (dim + 15) // 16 * 16, sum(lengths)
    x = torch.zeros(n, 4, heads, dp, device=DEV, dtype=dtype)
    x[..., :dim] = rnd(n, 4, heads, dim, dtype=dtype)
    z = 2 * torch.randn(n, heads * dp, device=DEV) - 1.5
    w0, u = rnd(heads * dp), rnd(heads * dp)
    state = torch.zeros(len(lengths) + 1, heads, dp, dp, device=DEV)
    state[:, :, :dim, :dim] = rnd(len(lengths) + 1, heads, dim, dim, dtype=torch.float32)
    return x.view(n, -1), z, w0, u, state, dp


def wkv_reference(x, z, w0, u, state, heads, dim, dp):
    """One sequence from `state` [heads, dp, dp]: read-outs and the state it leaves."""
    n = x.shape[0]
    r, k, v = (t[..., :dim] for t in x.double().view(n, -1, heads, dp).unbind(1)[:3])
    w = torch.exp(-torch.exp(z.double() + w0.double())).view(n, heads, dp)[..., :dim]
    S, out = state.double()[:, :dim, :dim].clone(), torch.zeros_like(r)
    uu = u.double().view(heads, dp)[:, :dim]
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + uu[:, :, None] * kv) * r[t][:, :, None]).sum(1)
        S = w[t][:, :, None] * S + kv
    return out, S


FORMS = [(torch.float32, "rows"), (torch.bfloat16, "rows"), (torch.bfloat16, "chunks"), (torch.bfloat16, "segments")]


@pytest.mark.parametrize("heads,dim,dtype,form", [(h, d, t, f) for h, d in ((3, 64), (2, 24), (2, 128), (5, 80), (1, 200), (2, 16)) for t, f in FORMS])
def test_wkv_rule(heads, dim, dtype, form):
    """Token after token; sixteen at a time, a few chunks per round; rounds in segments that run side by side."""
    lengths = [1, 15, 16, 17, 100, 333, 700]
    x, z, w0, u, state, dp = wkv_problem(heads, dim, lengths, dtype)
    seqs, base = [], 0
    for s, n in enumerate(lengths):
        seqs.append([base, n, s, 0 if s % 2 else 40])     # every second one starts from zero whatever its slot holds
        base += n
    before = state.clone()
    ws = torch.empty(len(lengths) * heads * 3 * 65536, device=DEV, dtype=torch.uint8) if form == "chunks" else None      # a few chunks per round
    o = Y.wkv_rule(x, z, w0, u, state, ints(seqs + [[0, 5, -1, 0]]), dim=dim, form="rows" if form == "rows" else "chunks", workspace=ws, longest=700)
    tol = 3e-5 if form == "rows" else 1e-3
    for b, n, s, p in seqs:
        want, S = wkv_reference(x[b:b + n], z[b:b + n], w0, u, before[s] * (p > 0), heads, dim, dp)
        close(o[b:b + n].view(n, heads, dp)[..., :dim], want, tol)
        close(state[s, :, :dim, :dim], S, tol)
    assert torch.equal(state[-1], before[-1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rank", [(3, 64, 16), (2, 24, 48), (4, 128, 64), (1, 16, 16)])
def test_wkv_step(heads, dim, rank, dtype):
    n, rnd = 5, gen(9)
    x, _, w0, u, state, dp = wkv_problem(heads, dim, [1] * n, dtype, 8)
    low, w2, wt = rnd(n, rank, dtype=torch.float32), rnd(heads * dp, 2 * rank) * rank ** -0.5, rnd(heads * dp)
    before, out = state.clone(), torch.zeros(n, heads * dp, device=DEV, dtype=dtype)
    tiles = P.row_tiles([(s, 0 if s == 2 else 7, 1, 0) for s in range(n)], DEV)
    Y.wkv_step(x, low, w2, w0, u, state, wt, out, tiles, dim=dim, eps=1e-5)
    z = torch.tanh(low.double()) @ w2[:, :rank].double().T
    for s in range(n):
        o, S = wkv_reference(x[s:s + 1], z[s:s + 1], w0, u, before[s] * (s != 2), heads, dim, dp)
        gate = oracle.silu(x[s].double().view(4, heads, dp)[3, :, :dim])
        close(out[s].view(heads, dp)[:, :dim], oracle.rms(o[0], 1e-5) * wt.double().view(heads, dp)[:, :dim] * gate, 0.01 if dtype == torch.bfloat16 else 1e-5)
        close(state[s, :, :dim, :dim], S, 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_shift_rows(dtype):
    rnd = gen(10)
    ld, entries = 1040, [(0, 0, 1, 0), (1, 33, 1, 1), (2, 0, 40, 0), (3, 17, 19, 1)]
    n = sum(e[2] for e in entries)
    x, mu, prev = rnd(n, ld, dtype=torch.float32), rnd(5, ld), rnd(2, 4, ld, dtype=torch.float32)
    old, out = prev.clone(), torch.zeros(5, n, ld, device=DEV, dtype=dtype)
    Y.shift_rows(x, mu, prev, out, P.row_tiles(entries, DEV))
    base = 0
    for slot, p0, m, parity in entries:
        h = x[base:base + m].double()
        first = old[parity, slot].double() if p0 else torch.zeros(ld, device=DEV, dtype=torch.float64)
        back = torch.cat([first[None], h[:-1]])
        for s in range(5):
            close(out[s, base:base + m], h + (back - h) * mu[s].double(), 0.01 if dtype == torch.bfloat16 else 1e-6)
        assert torch.equal(prev[1 - parity, slot], x[base + m - 1]) and torch.equal(prev[parity, slot], old[parity, slot])
        base += m


RULES = [dict(), dict(groups=4, keep=2), dict(groups=8, keep=1), dict(groups=2, keep=2), dict(groups=16, keep=3)]


@pytest.mark.parametrize("experts,top", [(16, 2), (48, 3), (64, 4), (256, 8), (112, 7)])
@pytest.mark.parametrize("rule", RULES, ids=str)
def test_expert_choice(experts, top, rule):
    """Both routing kernels against the plain rule, with choice scores of either sign."""
    if rule.get("groups") and rule["keep"] * (experts // rule["groups"]) < top:
        pytest.skip("the kept groups hold too few experts")
    rnd, T = gen(11), 60
    z, corr = rnd(T, experts, dtype=torch.float32), (rnd(experts) * 0.5 - 0.7)
    idx, weight, counts = Y.expert_choice(z, top, correction=corr, normalise=True, scale=1.3, **rule)
    h, up, down = rnd(T, 32), rnd(experts, 16, 32) * 0.2, rnd(experts, 32, 16) * 0.2
    mid, sd, ys = rnd(T, 48), rnd(32, 48) * 0.2, torch.zeros(T, 32, device=DEV, dtype=torch.bfloat16)
    idx2, weight2, y = Y.expert_rows(h, z, up, down, experts=experts, top=top, act=4, plain=True, shared_mid=mid, shared_down=sd, y_shared=ys, correction=corr, normalise=True, scale=1.3,
                                     **rule)
    close(ys, mid.double() @ sd.double().T, 0.02)
    assert torch.equal(counts, torch.bincount(idx.long().view(-1), minlength=experts).int())
    router = {"top": top, "scale": 1.3}
    if rule:
        router["groups"] = {"count": rule["groups"], "keep": rule["keep"]}
    for t in range(T):
        s = torch.sigmoid(z[t].double().cpu())
        if oracle.routing_gap(s, corr.double().cpu(), router) < 1e-6:
            continue
        e, a = oracle.route(s, corr.double().cpu(), router)
        for i, w in ((idx, weight), (idx2, weight2)):
            assert i[t].tolist() == e.tolist()
            close(w[t].cpu(), a, 1e-5)
        want = torch.stack([down[k].double() @ oracle.relu_squared(up[k].double() @ h[t].double()) for k in e.tolist()])
        close(y[t], want, 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [40, 1000, 4096, 5000])
@pytest.mark.parametrize("rows", [3, 400])
def test_stream_pass_with_a_norm_on_the_update(width, rows, dtype):
    """Weighted rows plus a row of their own, normed, scaled and added; the new residual out as it is or normed for the head."""
    rnd = gen(12)
    ld = (width + 15) // 16 * 16
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - width)).contiguous()  # noqa: E731
    x, y, plus, wy, wh = pad(rnd(rows, width, dtype=torch.float32)), pad(rnd(3 * rows, width, dtype=dtype)), pad(rnd(rows, width, dtype=dtype)), pad(rnd(width)), pad(rnd(width))
    item, order = torch.rand(rows * 3, device=DEV), torch.randperm(3 * rows, device=DEV).int()
    f = (y.double()[order.long()].view(rows, 3, ld) * item.double().view(rows, 3, 1)).sum(1) + plus.double()
    new = x.double() + 0.6 * torch.nn.functional.pad(oracle.rms(f[:, :width], 1e-5), (0, ld - width)) * wy.double()
    h, out = torch.zeros(rows, ld, device=DEV, dtype=dtype), torch.zeros(rows, ld, device=DEV)
    kw = dict(width=width, streams=1, ld=ld, f32=dtype == torch.float32, eps=1e-5, y=y, y_rows=3, y_index=order, y_item=item, y_plus=plus, y_weight=wy, y_scale=0.6)
    Y.stream_pass(x, h, rows=rows, x_out=out, **kw)
    close(out, new, 1e-5)
    close(h, new, 0.01 if dtype == torch.bfloat16 else 1e-5)
    pick = ints([rows - 1, 0])
    Y.stream_pass(x, h, rows=2, src_rows=pick, weight=wh, **kw)
    close(h[:2, :width], oracle.rms(new[pick.long()][:, :width], 1e-5) * wh.double()[:width], 0.01 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_ff_rows(dtype):
    rnd = gen(13)
    x = rnd(35, 96, dtype=dtype)
    for act, fn in ((3, oracle.silu), (4, oracle.relu_squared)):
        out = Y.ff_rows(x, torch.zeros(35, 48, device=DEV, dtype=dtype), off_gate=0, off_up=48, act=act)
        close(out, fn(x[:, :48].double()) * x[:, 48:].double(), 0.01 if dtype == torch.bfloat16 else 1e-6)
        close(Y.ff_rows(x, out, off_gate=48, off_up=-1, act=act), fn(x[:, 48:].double()), 0.01 if dtype == torch.bfloat16 else 1e-6)
