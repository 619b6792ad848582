"""Linear attention with a decay per head, the gated recurrence, convolutions on a sublayer's input, learned sinks, clamped gates and the softmax over chosen
experts: each kernel against plain PyTorch in float64."""
import math

import pytest
import torch

import kidolorn_oracle as oracle
from neuralfn_b200.ops import layered as Y, paged as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.bfloat16, torch.float32]


def close(got, want, tol):
    assert torch.isfinite(got).all()
    assert float((got.double() - want.double()).abs().max()) < tol * float(want.abs().max() + 1e-3)


def gen(seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return lambda *s, dtype=torch.bfloat16: torch.randn(*s, generator=g, device=DEV).to(dtype)


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def padded(n):
    return (n + 15) // 16 * 16


def decays(heads):
    return ([0.9999, 0.5, 0.97, 1.0, 0.0, 0.9] * heads)[:heads]


def linear_problem(heads, dim, vdim, lengths, dtype, seed=6):
    """Rows [q | k | v] and a state per sequence, padding zero."""
    rnd, n, dp, vp = gen(seed), sum(lengths), padded(dim), padded(vdim)
    x = torch.zeros(n, 2 * heads * dp + heads * vp, device=DEV, dtype=dtype)
    x[:, :2 * heads * dp].view(n, 2, heads, dp)[..., :dim] = rnd(n, 2, heads, dim, dtype=dtype)
    x[:, 2 * heads * dp:].view(n, heads, vp)[..., :vdim] = rnd(n, heads, vdim, dtype=dtype)
    state = torch.zeros(len(lengths) + 1, heads, dp, vp, device=DEV)
    state[:, :, :dim, :vdim] = rnd(len(lengths) + 1, heads, dim, vdim, dtype=torch.float32)
    return x, state, dp, vp


def linear_reference(x, state, heads, dp, vp, decay, act=lambda t: t):
    n = x.shape[0]
    q, k = act(x.double()[:, :2 * heads * dp]).view(n, 2, heads, dp).unbind(1)
    v = act(x.double()[:, 2 * heads * dp:2 * heads * dp + heads * vp]).view(n, heads, vp)
    S, out = state.double().clone(), torch.zeros_like(v)
    f = torch.tensor(decay, dtype=torch.float64, device=x.device)[:, None, None]
    for t in range(n):
        S = f * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out.reshape(n, -1), S


FORMS = [(torch.float32, "rows"), (torch.bfloat16, "rows"), (torch.bfloat16, "chunks"), (torch.bfloat16, "segments")]


@pytest.mark.parametrize("heads,dim,vdim,dtype,form", [(h, d, v, t, f) for h, d, v in ((3, 64, 64), (2, 24, 200), (5, 128, 128), (1, 80, 16), (2, 16, 72)) for t, f in FORMS] +
                         [(2, 200, 48, torch.bfloat16, "rows"), (1, 512, 16, torch.float32, "rows")])
def test_linear_rule(heads, dim, vdim, dtype, form):
    """Token after token; 64 at a time; a sequence in segments that run side by side."""
    lengths = [1, 15, 63, 64, 65, 333, 700]
    x, state, dp, vp = linear_problem(heads, dim, vdim, lengths, dtype)
    seqs, base = [], 0
    for s, n in enumerate(lengths):
        seqs.append([base, n, s, 0 if s % 2 else 40])     # every second one starts from zero whatever its slot holds
        base += n
    before, d = state.clone(), decays(heads)
    ws = torch.empty(1, device=DEV, dtype=torch.uint8) if form == "chunks" else None
    o = Y.linear_rule(x, Y.powers(d, DEV), state, ints(seqs + [[0, 5, -1, 0]]), form="rows" if form == "rows" else "chunks", workspace=ws, longest=700)
    for b, n, s, p in seqs:
        want, S = linear_reference(x[b:b + n], before[s] * (p > 0), heads, dp, vp, d)
        close(o[b:b + n], want, 3e-5 if form == "rows" else 1e-4)
        close(state[s], S, 3e-5 if form == "rows" else 1e-4)
    assert torch.equal(state[-1], before[-1])


def test_linear_segments_of_one_long_sequence():
    heads, dim, n = 2, 64, 3001
    x, state, dp, vp = linear_problem(heads, dim, dim, [n], torch.bfloat16)
    before, d = state.clone(), [0.9995, 0.95]
    o = Y.linear_rule(x, Y.powers(d, DEV), state, ints([[0, n, 0, 7]]), form="chunks")
    want, S = linear_reference(x, before[0], heads, dp, vp, d)
    close(o, want, 1e-4)
    close(state[0], S, 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(3, 64, 64), (2, 24, 40), (32, 128, 128), (1, 16, 16), (3, 320, 208), (2, 48, 512)])
def test_linear_step(heads, dim, vdim, dtype):
    n, rnd = 5, gen(9)
    dp, vp = padded(dim), padded(vdim)
    x, state, _, _ = linear_problem(heads, dim, vdim, [1] * n, dtype, 8)
    g, wt = torch.zeros(n, heads, vp, device=DEV, dtype=dtype), rnd(heads * vp)
    g[..., :vdim] = rnd(n, heads, vdim, dtype=dtype)
    x = torch.cat([x, g.view(n, -1)], 1)
    before, d, counters = state.clone(), decays(heads), torch.zeros(n, dtype=torch.int32, device=DEV)
    tiles = P.row_tiles([(s, 0 if s == 2 else 7, 1, 0) for s in range(n)], DEV)
    for again in range(2):                                # the counters are ready for the next call
        state.copy_(before)
        out = torch.zeros(n, heads * vp, device=DEV, dtype=dtype)
        Y.linear_step(x, Y.powers(d, DEV), state, wt, out, tiles, counters, vdim=vdim, eps=1e-5)
        assert not counters.any()
        for s in range(n):
            o, S = linear_reference(x[s:s + 1], before[s] * (s != 2), heads, dp, vp, d, oracle.silu)
            want = o[0] / torch.sqrt((o[0] ** 2).sum() / (heads * vdim) + 1e-5) * wt.double() * oracle.sigmoid(g[s].double().flatten())
            close(out[s], want, 0.01 if dtype == torch.bfloat16 else 2e-5)
            close(state[s], S, 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols,live", [(16, 5), (1040, 1040), (6000, 5990)])
def test_row_out(cols, live, dtype):
    rnd = gen(3)
    o, g, w = torch.zeros(7, cols, device=DEV), rnd(7, cols, dtype=dtype), rnd(cols)
    o[:, :live] = rnd(7, live, dtype=torch.float32)
    want = o.double() / torch.sqrt((o.double() ** 2).sum(-1, keepdim=True) / live + 1e-5) * w.double() * oracle.sigmoid(g.double())
    close(Y.row_out(o, g, w, live=live, eps=1e-5), want, 0.01 if dtype == torch.bfloat16 else 2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [16, 48, 400])
def test_gru_rows(width, dtype):
    rnd = gen(4)
    lengths = [1, 3, 15, 16, 255, 256, 257, 1100]
    n, n_short = sum(lengths), 3
    x = 2 * rnd(n, 3 * width, dtype=torch.float32)
    x[:, :width // 2] -= 9                                # half of the channels remember for thousands of tokens
    x = x.to(dtype)
    state, out = rnd(len(lengths) + 1, width, dtype=torch.float32), torch.zeros(n, width, device=DEV, dtype=dtype)
    before, seqs, base = state.clone(), [], 0
    for s, m in enumerate(lengths):
        seqs.append([base, m, s, 0 if s % 2 else 40])
        base += m
    Y.gru_rows(x, state, out, ints(seqs[:n_short] + [[0, 1, -1, 0]] + seqs[n_short:] + [[0, 20, -1, 0]]), n_short + 1)
    for b, m, s, p in seqs:
        a, c, g = x[b:b + m].double().split(width, 1)
        z, c, S = oracle.sigmoid(a), oracle.candidate(c), before[s].double() * (p > 0)
        want = torch.zeros(m, width, device=DEV, dtype=torch.float64)
        for t in range(m):
            S = (1 - z[t]) * S + z[t] * c[t]
            want[t] = S * oracle.silu(g[t])
        close(out[b:b + m], want, 0.006 if dtype == torch.bfloat16 else 3e-6)
        close(state[s], S, 3e-6)
    assert torch.equal(state[-1], before[-1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_input_convolution(taps, dtype):
    """The launch of its own and the one inside the stream pass, over what earlier steps left."""
    rnd = gen(10)
    ld, width, entries = 1040, 1030, [(0, 0, 1, 0), (1, 33, 1, 1), (2, 0, 40, 0), (3, 17, 19, 1), (4, 1, 2, 0), (5, 2, 3, 1)]
    n = sum(e[2] for e in entries)
    h, w, hist = rnd(n, ld, dtype=dtype), rnd(taps, ld), rnd(2, 6, max(taps - 1, 1), ld, dtype=dtype)
    old, out = hist.clone(), torch.zeros(n, ld, device=DEV, dtype=dtype)
    Y.input_conv(h, w, hist, out, P.row_tiles(entries, DEV))
    tol, base = 0.01 if dtype == torch.bfloat16 else 1e-6, 0

    def past(slot, p0, parity):
        rows = old[parity, slot, :taps - 1].double()
        rows = rows.clone()
        if p0 < taps - 1:
            rows[:taps - 1 - p0] = 0                      # nothing before the sequence's start
        return rows

    for slot, p0, m, parity in entries:
        before = past(slot, p0, parity)
        rows = torch.cat([before, h[base:base + m].double()])
        want = rows[taps - 1:] + sum(rows[j:j + m] * w[j].double() for j in range(taps))
        close(out[base:base + m], want, tol)
        if taps > 1:
            assert torch.equal(hist[1 - parity, slot].double(), rows[-(taps - 1):]) and torch.equal(hist[parity, slot], old[parity, slot])
        base += m
    # one row per sequence, behind a norm with a single factor
    singles = [(0, 0, 1, 0), (1, 33, 1, 1), (2, 1, 1, 0), (-1, 0, 1, 0), (4, 2, 1, 1)]
    x, g, hist = rnd(5, ld, dtype=torch.float32), rnd(1), old.clone()
    x[:, width:] = 0
    h = torch.zeros(5, ld, device=DEV, dtype=dtype)
    Y.stream_pass(x, h, width=width, streams=1, rows=5, ld=ld, f32=dtype == torch.float32, weight=g, scalar_norms=True, conv=w, history=hist, tiles=P.row_tiles(singles, DEV))
    row = torch.zeros(5, ld, device=DEV, dtype=torch.float64)
    row[:, :width] = oracle.rms(x[:, :width].double(), 1e-5) * g.double()
    for i, (slot, p0, _, parity) in enumerate(singles):
        if slot < 0:
            continue
        rows = torch.cat([past(slot, p0, parity), row[i:i + 1]])
        close(h[i], rows[-1] + (rows * w.double()).sum(0), tol)
        if taps > 1:
            close(hist[1 - parity, slot], rows[1:], tol)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_of_latent_attention(dtype):
    """Single rows with one share and with many, prompt tiles with a gate."""
    rnd, heads, rank, rot, dim, vdim = gen(12), 5, 64, 16, 32, 48
    lengths = [700, 3, 65]
    c = Y.LatentCache(3, 704, rank, rot, DEV, dtype)
    z = [rnd(n, rank + rot, dtype=dtype) for n in lengths]
    for s, t in enumerate(z):
        c.write(s, t)
    sinks, scale = torch.linspace(-3, 12, heads, device=DEV).bfloat16(), 3 * (rank + rot) ** -0.5
    slot, pos = ints([0, 1, 2, 0]), ints([699, 2, 64, 0])
    q, out = rnd(4, heads * (rank + rot), dtype=dtype), torch.zeros(4, heads * rank, device=DEV, dtype=dtype)
    for max_keys in (700, 64):
        Y.latent_attention_rows(c, q, slot, pos, out, heads=heads, window=0, scale=scale, max_keys=max_keys, sinks=sinks)
        for r, (s, p) in enumerate(zip(slot.tolist(), pos.tolist())):
            keys = z[s][:p + 1].double()
            sc = torch.cat([q[r].double().view(heads, -1) @ keys.T * scale, sinks.double()[:, None]], 1)
            close(out[r].view(heads, rank), torch.softmax(sc, -1)[:, :-1] @ keys[:, :rank], 0.02 if dtype == torch.bfloat16 else 2e-5)
    if dtype == torch.float32:
        return
    x, n = rnd(704, heads * (dim + vdim)), 200
    q, gate, out = rnd(n, heads * (dim + rot)), rnd(n, heads * vdim), torch.zeros(n, heads * vdim, device=DEV, dtype=dtype)
    tiles = ints([[0, 128, 0, 500], [128, 72, 0, 628]])
    Y.latent_attention_tiles(c, q, x, ints([0, 0, 0]), tiles, out, heads=heads, dim=dim, vdim=vdim, window=0, scale=scale, sinks=sinks, gate=gate)
    k, v = x[:700, :heads * dim].double().view(-1, heads, dim), x[:700, heads * dim:].double().view(-1, heads, vdim)
    qq = q.double().view(n, heads, -1)
    sc = (torch.einsum("rhd,nhd->hrn", qq[..., :dim], k) + torch.einsum("rhd,nd->hrn", qq[..., dim:], z[0][:, rank:].double())) * scale
    sc = sc.masked_fill(torch.arange(700, device=DEV)[None] > torch.arange(500, 700, device=DEV)[:, None], -math.inf)
    sc = torch.softmax(torch.cat([sc, sinks.double()[:, None, None].expand(heads, n, 1)], 2), -1)[..., :-1]
    want = torch.einsum("hrn,nhd->rhd", sc, v).reshape(n, -1) * oracle.sigmoid(gate.double())
    close(out, want, 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv", [5, 1])
def test_sinks_of_paged_attention(kv, dtype):
    rnd, heads, dim, n = gen(14), 5, 64, 300
    c = P.PagedCache(1, 320, kv, dim, dim, DEV, dtype)
    k, v = rnd(n, kv, dim), rnd(n, kv, dim)
    c.write(0, k, v)
    sinks, scale, at = torch.linspace(8, -2, heads, device=DEV).bfloat16(), 2 * dim ** -0.5, [299, 0, 64]
    rep = heads // kv

    def want(q, pos):
        s = torch.einsum("rhd,nhd->hrn", q.double().view(len(pos), heads, dim), k.double().repeat_interleave(rep, 1)) * scale
        s = s.masked_fill(torch.arange(n, device=DEV)[None] > torch.tensor(pos, device=DEV)[:, None], -math.inf)
        s = torch.softmax(torch.cat([s, sinks.double()[:, None, None].expand(heads, len(pos), 1)], 2), -1)[..., :-1]
        return torch.einsum("hrn,nhd->rhd", s, v.double().repeat_interleave(rep, 1)).reshape(len(pos), -1)

    q, out = rnd(3, heads * dim, dtype=dtype), torch.zeros(3, heads * dim, device=DEV, dtype=dtype)
    for max_keys in (300, 32):
        P.attention_rows(c, q, ints([0, 0, 0]), ints(at), out, heads=heads, scale=scale, sinks=sinks, max_keys=max_keys)
        close(out, want(q, at), 0.02 if dtype == torch.bfloat16 else 2e-5)
    if dtype == torch.bfloat16:
        rows, step = 100, P.tile_rows(c, heads)
        q, out = rnd(rows, heads * dim), torch.zeros(rows, heads * dim, device=DEV, dtype=dtype)
        P.attention_tiles(c, q, ints([[r, min(step, rows - r), 0, 200 + r] for r in range(0, rows, step)]), out, heads=heads, scale=scale, sinks=sinks)
        close(out, want(q, list(range(200, 300))), 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gate_of_group_products(dtype):
    rnd = gen(15)
    for rows, groups, n, k in ((1, 3, 48, 64), (9, 2, 80, 128), (40, 5, 32, 48)):
        x, w, gate, out = rnd(rows, groups, k, dtype=dtype), rnd(groups, n, k) * k ** -0.5, rnd(rows, groups, n, dtype=dtype), torch.zeros(rows, groups, n, device=DEV, dtype=dtype)
        Y.group_products(x, w, out, gate=gate)
        close(out, torch.einsum("rgk,gnk->rgn", x.double(), w.double()) * oracle.sigmoid(gate.double()), 0.01 if dtype == torch.bfloat16 else 2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_gate(dtype):
    x = 3 * gen(16)(35, 96, dtype=dtype)
    out = Y.ff_rows(x, torch.zeros(35, 48, device=DEV, dtype=dtype), off_gate=0, off_up=48, act=7, clamp=(1.3, 1.702, 1.0))
    close(out, oracle.clamped_gate(x[:, :48].double(), x[:, 48:].double(), 1.3), 0.01 if dtype == torch.bfloat16 else 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [3, 12, 60])
@pytest.mark.parametrize("experts,top", [(1, 1), (16, 4), (48, 48), (64, 3), (256, 8)])
def test_softmax_routing_and_experts_weighted_at_their_output(experts, top, rows, dtype):
    rnd, width, ff = gen(17), 48, 32
    z, h = 2 * rnd(rows, experts, dtype=torch.float32), rnd(rows, width, dtype=dtype)
    gu, down = rnd(experts, 2 * ff, width) * 0.3, rnd(experts, width, ff) * 0.3
    idx, weight, counts = Y.expert_choice(z, top, softmax=True)
    idx2, weight2, y = Y.expert_rows(h, z, gu, down, experts=experts, top=top, act=7, weigh_output=True, clamp=(0.9, 1.702, 1.0), softmax=True)
    assert torch.equal(counts, torch.bincount(idx.long().view(-1), minlength=experts).int())
    for t in range(rows):
        e, a = oracle.route(z[t].double(), top)
        for i, w in ((idx, weight), (idx2, weight2)):
            assert i[t].tolist() == e.tolist()
            close(w[t], a, 1e-5)
        mid = torch.stack([oracle.clamped_gate(*(gu[k].double() @ h[t].double()).split(ff), 0.9) for k in e.tolist()])
        close(y[t], torch.einsum("ewf,ef->ew", down[e].double(), mid), 0.02 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("rows,experts,width", [(1, 1, 16), (8, 32, 4096), (9, 40, 2064), (32, 100, 336)])
def test_router_rows(rows, experts, width):
    rnd = gen(18)
    h, w = rnd(rows, width), rnd(experts, width)
    close(Y.router_rows(h, w), h.double() @ w.double().T, 3e-6)
