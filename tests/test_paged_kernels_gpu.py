"""Kernels of the layer-list engine against plain PyTorch in fp32: attention over shuffled pages (single rows, split keys, tcgen05
tiles), the residual product of every GEMM path, the row pass and the row mix."""
import math

import pytest
import torch

from neuralfn_b200.ops import paged as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def reference(q, k, v, pos, *, scale, window, slopes, gate):
    """q [R, H, d] at positions pos [R] over k [n, G, d], v [n, G, dv]."""
    rep = q.shape[1] // k.shape[1]
    j = torch.arange(k.shape[0], device=q.device)
    dist = pos[:, None] - j[None]
    seen = (dist >= 0) & ((dist < window) if window else True)
    s = torch.einsum("rhd,nhd->hrn", q, k.repeat_interleave(rep, 1)) * scale - slopes[:, None, None] * dist
    s = s.masked_fill(~seen, -math.inf)
    o = torch.einsum("hrn,nhd->rhd", torch.softmax(s, -1), v.repeat_interleave(rep, 1)).reshape(q.shape[0], -1)
    return o * torch.sigmoid(gate)


def problem(heads, kv_heads, dim, vdim, lengths, dtype=torch.bfloat16, seed=0):
    g = torch.Generator(device=DEV).manual_seed(seed)
    c = P.PagedCache(len(lengths), max(lengths), kv_heads, dim, vdim, DEV, dtype, seed)
    kv = []
    for s, n in enumerate(lengths):
        k, v = (torch.randn(n, kv_heads, w, generator=g, device=DEV).to(dtype).float() for w in (dim, vdim))
        c.write(s, k, v)
        kv.append((k, v))
    slopes = torch.tensor([2.0 ** (-8 * (h + 1) / heads) for h in range(heads)], device=DEV)
    return c, kv, slopes, g


def close(got, want, tol):
    assert torch.isfinite(got).all()
    assert float((got.float() - want).abs().max()) < tol * float(want.abs().max() + 1e-3)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(8, 2, 128, 128), (4, 4, 16, 32), (12, 1, 64, 80), (40, 2, 96, 48), (4, 2, 256, 208), (2, 1, 288, 64)])
@pytest.mark.parametrize("window", [0, 1, 100, 700])
def test_rows(heads, kv_heads, dim, vdim, window):
    lengths = [1500, 3, 64, 65, 900]
    c, kv, slopes, g = problem(heads, kv_heads, dim, vdim, lengths)
    rows = [(s, n - 1) for s, n in enumerate(lengths)] + [(0, 700), (4, 128), (-1, 0)]
    slot, pos = (torch.tensor([r[i] for r in rows], dtype=torch.int32, device=DEV) for i in (0, 1))
    q, gate = (torch.randn(len(rows), heads * w, generator=g, device=DEV).bfloat16() for w in (dim, vdim))
    out = torch.zeros(len(rows), heads * vdim, device=DEV, dtype=torch.bfloat16)
    for _ in range(2):      # the counters of the split form are left ready
        P.attention_rows(c, q, slot, pos, out, heads=heads, window=window, scale=dim ** -0.5, slopes=slopes, gate=gate, max_keys=1500)
        for r, (s, p) in enumerate(rows):
            if s < 0:
                continue
            want = reference(q[r:r + 1].float().view(1, heads, dim), *kv[s], pos[r:r + 1].long(), scale=dim ** -0.5, window=window, slopes=slopes, gate=gate[r:r + 1].float())
            close(out[r:r + 1], want, 0.02)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(8, 2, 128, 128), (4, 4, 16, 32), (12, 1, 64, 80), (6, 2, 96, 48), (4, 2, 256, 240), (128, 1, 32, 16)])
@pytest.mark.parametrize("window", [0, 1, 64, 100, 700])
def test_tiles(heads, kv_heads, dim, vdim, window):
    lengths = [1100, 70, 64, 300]
    c, kv, slopes, g = problem(heads, kv_heads, dim, vdim, lengths, seed=1)
    step, parts = P.tile_rows(c, heads), [(0, 900, 200), (1, 0, 70), (2, 17, 47), (3, 299, 1)]     # slot, first position, rows
    tiles, base = [], 0
    for s, p0, n in parts:
        tiles += [[base + r, min(step, n - r), s, p0 + r] for r in range(0, n, step)]
        base += n
    q, gate = (torch.randn(base, heads * w, generator=g, device=DEV).bfloat16() for w in (dim, vdim))
    out = torch.zeros(base, heads * vdim, device=DEV, dtype=torch.bfloat16)
    P.attention_tiles(c, q, torch.tensor(tiles, dtype=torch.int32, device=DEV), out, heads=heads, window=window, scale=dim ** -0.5, slopes=slopes, gate=gate)
    from neuralfn_b200.ops import _lib
    _lib.assert_status_ok("paged tiles")
    base = 0
    for s, p0, n in parts:
        want = reference(q[base:base + n].float().view(n, heads, dim), *kv[s], torch.arange(p0, p0 + n, device=DEV), scale=dim ** -0.5, window=window, slopes=slopes,
                         gate=gate[base:base + n].float())
        close(out[base:base + n], want, 0.02)
        base += n


@pytest.mark.parametrize("m,n,k", [(1, 320, 512), (2, 4096, 1024), (8, 2048, 1024), (16, 96, 64), (40, 512, 4096), (100, 2048, 8192), (300, 272, 528), (1100, 2048, 512), (16384, 256, 256)])
def test_residual_product(m, n, k):
    g = torch.Generator(device=DEV).manual_seed(m)
    a, b = (torch.randn(r, k, generator=g, device=DEV).bfloat16() for r in (m, n))
    x = torch.randn(m, n, generator=g, device=DEV) * 3
    want = x + a.float() @ b.float().T
    copy = torch.zeros(m, n, device=DEV, dtype=torch.bfloat16)
    P.residual_gemm(a, b, x, copy, torch.empty(16 << 20, device=DEV))
    assert float((x - want).abs().max()) < 2e-5 * k ** 0.5 * 10
    assert torch.equal(copy, x.bfloat16())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ld", [(40, 48), (1000, 1008), (4096, 4096), (12288, 12288)])
def test_row_pass(width, ld, dtype):
    g = torch.Generator(device=DEV).manual_seed(width)

    def rows(n, dt=torch.float32):
        t = torch.zeros(n, ld, device=DEV, dtype=dt)
        t[:, :width] = torch.randn(n, width, generator=g, device=DEV).to(dt)
        return t

    x, y, w, wy = rows(7), rows(5, dtype), rows(1, torch.bfloat16)[0], rows(1, torch.bfloat16)[0]
    src = torch.tensor([6, 0, 3, 3, 1], dtype=torch.int32, device=DEV)
    h, xo = torch.empty(5, ld, device=DEV, dtype=dtype), torch.empty(5, ld, device=DEV)
    P.row_norm(x, w, h, eps=1e-3, width=width, y=y, y_weight=wy, x_out=xo, src_rows=src)
    yf = y.float()
    base = x[src.long()] + yf / torch.sqrt((yf * yf).sum(-1, keepdim=True) / width + 1e-3) * wy.float()
    want = base / torch.sqrt((base * base).sum(-1, keepdim=True) / width + 1e-3) * w.float()
    close(xo, base, 1e-5)
    close(h, want, 1e-5 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [0, 1, 2, 3, 4, 6])
def test_row_mix(taps, dtype):
    heads, kv_heads, dim, vdim, ff = 3, 1, 32, 48, 80
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    ch = nq + nk + nv
    g = torch.Generator(device=DEV).manual_seed(taps)
    c = P.PagedCache(3, 256, kv_heads, dim, vdim, DEV, dtype, seed=3)
    conv = torch.randn(taps, ch, generator=g, device=DEV).bfloat16() if taps else None
    state = torch.zeros(2, 3, max(taps - 1, 1), ch, device=DEV, dtype=dtype)
    lengths = {0: [40, 1, 1, 3, 17], 2: [1, 1, 70, 2, 16]}
    full = {s: torch.randn(sum(n), ch + 2 * ff, generator=g, device=DEV).to(dtype) for s, n in lengths.items()}
    q_all = {s: [] for s in lengths}
    done, parity = {s: 0 for s in lengths}, 0
    for i in range(5):
        entries = [(s, done[s], lengths[s][i], parity) for s in lengths]
        x = torch.cat([full[s][done[s]:done[s] + n] for s, _, n, _ in entries]).contiguous()
        q, f = torch.empty(x.shape[0], nq, device=DEV, dtype=dtype), torch.empty(x.shape[0], ff, device=DEV, dtype=dtype)
        P.mix_rows(c, x, P.row_tiles(entries, DEV), q, f, heads=heads, off_gate=ch, off_up=ch + ff, ff=ff, conv=conv, state=state, temp=(0.5, 7))
        close(f, torch.relu(x[:, ch:ch + ff].float()) * x[:, ch + ff:].float(), 1e-6 if dtype == torch.float32 else 6e-3)
        base = 0
        for s, _, n, _ in entries:
            q_all[s].append(q[base:base + n])
            base += n
            done[s] += n
        parity ^= 1
    for s in lengths:
        u = full[s][:, :ch].float()
        y = u.clone()
        if taps:
            y = torch.zeros_like(u)
            for j in range(taps):
                d = taps - 1 - j
                y[d:] += conv[j].float() * u[:u.shape[0] - d]
        pos = torch.arange(u.shape[0], device=DEV)
        y[:, :nq] *= (1 + 0.5 * torch.log(torch.floor((pos + 1) / 7) + 1))[:, None]
        tol = 1e-5 if dtype == torch.float32 else 6e-3
        close(torch.cat(q_all[s]), y[:, :nq], tol)
        for p in range((u.shape[0] + 63) // 64):
            n, page = min(64, u.shape[0] - p * 64), int(c.table[s, p])
            rows = y[p * 64:p * 64 + n]
            close(c.k[page, 0, :n], rows[:, nq:nq + nk], tol)
            close(c.v[page, 0, :, :n].T, rows[:, nq + nk:], tol)
