"""ctypes bindings of the layer-list engine's kernels (csrc/kernels/paged_*.cu) on torch tensors: attention over cache pages, the row
pass and the step after the input projection. The engine calls them from C++; these wrappers serve kernel tests and timing."""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib

__all__ = ["PAGE", "PagedCache", "attention_rows", "attention_tiles", "mix_rows", "residual_gemm", "row_norm", "row_tiles", "tile_rows"]

PAGE = 64


class _Attention(C.Structure):
    _fields_ = [("f32", C.c_int), ("q", C.c_void_p), ("ld_q", C.c_int), ("k_pool", C.c_void_p), ("v_pool", C.c_void_p), ("kv_heads", C.c_int),
                ("dim_p", C.c_int), ("vdim_p", C.c_int), ("pages", C.c_longlong), ("table", C.c_void_p), ("table_ld", C.c_int), ("heads", C.c_int),
                ("window", C.c_int), ("scale", C.c_float), ("slopes", C.c_void_p), ("gate", C.c_void_p), ("ld_gate", C.c_int), ("out", C.c_void_p),
                ("ld_o", C.c_int), ("row_slot", C.c_void_p), ("row_pos", C.c_void_p), ("rows", C.c_int), ("row0", C.c_int), ("max_keys", C.c_int),
                ("workspace", C.c_void_p), ("workspace_bytes", C.c_longlong), ("tiles", C.c_void_p), ("n_tiles", C.c_int), ("total_rows", C.c_int),
                ("keep_first", C.c_int), ("softcap", C.c_float), ("sink", C.c_int), ("chunk", C.c_int), ("sinks", C.c_void_p)]


class _Mix(C.Structure):
    _fields_ = [("f32", C.c_int), ("in_", C.c_void_p), ("ld_in", C.c_int), ("nq", C.c_int), ("nk", C.c_int), ("nv", C.c_int), ("off_gate", C.c_int),
                ("off_up", C.c_int), ("ff", C.c_int), ("act", C.c_int), ("conv", C.c_void_p), ("taps", C.c_int), ("conv_act", C.c_int), ("state", C.c_void_p),
                ("state_half", C.c_longlong), ("q_out", C.c_void_p), ("ld_q", C.c_int), ("k_pool", C.c_void_p), ("v_pool", C.c_void_p), ("kv_heads", C.c_int),
                ("dim_p", C.c_int), ("vdim_p", C.c_int), ("table", C.c_void_p), ("table_ld", C.c_int), ("temp_coef", C.c_float), ("temp_every", C.c_int),
                ("ff_out", C.c_void_p), ("ld_ff", C.c_int), ("tiles", C.c_void_p), ("n_tiles", C.c_int), ("tile_rows", C.c_int), ("rows", C.c_int)]


class _RowNorm(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("width", C.c_int), ("ld", C.c_int), ("x", C.c_void_p), ("x_out", C.c_void_p),
                ("src_rows", C.c_void_p), ("tokens", C.c_void_p), ("embed", C.c_void_p), ("embed_scale", C.c_float), ("vocab", C.c_int), ("y", C.c_void_p),
                ("y_weight", C.c_void_p), ("h", C.c_void_p), ("weight", C.c_void_p), ("eps", C.c_float)]


def _p(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


class PagedCache:
    """Key and value pools of one layer, a page table per slot, workspace. Pages are handed out in the order of ``order``."""

    def __init__(self, slots: int, max_seq: int, kv_heads: int, dim: int, vdim: int, device, dtype=torch.bfloat16, seed: int = 0) -> None:
        per_slot = (max_seq + PAGE - 1) // PAGE
        self.pages, self.kv_heads, self.dim, self.vdim, self.dtype = slots * per_slot, kv_heads, dim, vdim, dtype
        self.k = torch.zeros(self.pages, kv_heads, PAGE, dim, device=device, dtype=dtype)
        self.v = torch.zeros(self.pages, kv_heads, vdim, PAGE, device=device, dtype=dtype)
        g = torch.Generator().manual_seed(seed)
        self.table = torch.randperm(self.pages, generator=g).view(slots, per_slot).to(device=device, dtype=torch.int32)
        lib = _lib.load()
        lib.nfn_paged_attention_workspace_bytes.restype = C.c_longlong
        self.ws = torch.zeros(lib.nfn_paged_attention_workspace_bytes(1, 1, 1), device=device, dtype=torch.uint8)

    def write(self, slot: int, k: torch.Tensor, v: torch.Tensor) -> None:
        """k [n, kv_heads, dim], v [n, kv_heads, vdim] to positions 0 .. n - 1 of the slot."""
        for p in range((k.shape[0] + PAGE - 1) // PAGE):
            page, part = int(self.table[slot, p]), slice(p * PAGE, min((p + 1) * PAGE, k.shape[0]))
            n = part.stop - part.start
            self.k[page, :, :n] = k[part].transpose(0, 1).to(self.dtype)
            self.v[page, :, :, :n] = v[part].permute(1, 2, 0).to(self.dtype)


def _args(c: PagedCache, q, out, heads, window, scale, slopes, gate, keep_first=0, softcap=0.0, sink=False, chunk=0, sinks=None) -> _Attention:
    a = _Attention()
    a.keep_first, a.softcap, a.sink, a.chunk, a.sinks = keep_first, softcap, int(sink), chunk, _p(sinks)
    a.f32, a.q, a.ld_q, a.k_pool, a.v_pool = int(c.dtype == torch.float32), _p(q), q.stride(0), _p(c.k), _p(c.v)
    a.kv_heads, a.dim_p, a.vdim_p, a.pages, a.table, a.table_ld = c.kv_heads, c.dim, c.vdim, c.pages, _p(c.table), c.table.stride(0)
    a.heads, a.window, a.scale, a.slopes, a.gate, a.ld_gate = heads, window, scale, _p(slopes), _p(gate), gate.stride(0) if gate is not None else 0
    a.out, a.ld_o, a.workspace, a.workspace_bytes, a.total_rows = _p(out), out.stride(0), _p(c.ws), c.ws.numel(), q.shape[0]
    return a


def attention_rows(c: PagedCache, q: torch.Tensor, row_slot: torch.Tensor, row_pos: torch.Tensor, out: torch.Tensor, *, heads: int, window: int = 0,
                   scale: float, slopes: torch.Tensor | None = None, gate: torch.Tensor | None = None, max_keys: int = 0, keep_first: int = 0,
                   softcap: float = 0.0, sink: bool = False, chunk: int = 0, sinks: torch.Tensor | None = None) -> torch.Tensor:
    a = _args(c, q, out, heads, window, scale, slopes, gate, keep_first, softcap, sink, chunk, sinks)
    a.row_slot, a.row_pos, a.rows = _p(row_slot), _p(row_pos), q.shape[0]
    a.max_keys = max_keys or chunk or (window + keep_first if window else c.table.shape[1] * PAGE)
    _lib.check(_lib.load().nfn_paged_attention_rows(C.byref(a), C.c_void_p(_lib.stream_ptr())), "paged_attention_rows")
    return out


def tile_rows(c: PagedCache, heads: int) -> int:
    return _lib.load().nfn_paged_tile_rows(int(c.dtype == torch.float32), heads, c.kv_heads, c.dim, c.vdim)


def attention_tiles(c: PagedCache, q: torch.Tensor, tiles: torch.Tensor, out: torch.Tensor, *, heads: int, window: int = 0, scale: float,
                    slopes: torch.Tensor | None = None, gate: torch.Tensor | None = None, keep_first: int = 0, softcap: float = 0.0,
                    sink: bool = False, chunk: int = 0, sinks: torch.Tensor | None = None) -> torch.Tensor:
    """``tiles``: int32 [n, 4] = first row, rows (<= ``tile_rows``), slot, position of the first row."""
    a = _args(c, q, out, heads, window, scale, slopes, gate, keep_first, softcap, sink, chunk, sinks)
    a.tiles, a.n_tiles = _p(tiles), tiles.shape[0]
    _lib.check(_lib.load().nfn_paged_attention_tiles(C.byref(a), C.c_void_p(_lib.stream_ptr())), "paged_attention_tiles")
    return out


def row_tiles(entries: list[tuple[int, int, int, int]], device) -> torch.Tensor:
    """Row tiles of a step from its entries (slot, position of the first row, rows, parity), rows one entry after another."""
    out, base = [], 0
    for slot, pos0, n, parity in entries:
        r = 0
        while r < n:
            k = min(n - r, 16 - (pos0 + r) % 16)
            out.append([base + r, k, base, n, pos0, slot, parity, 0])
            r += k
        base += n
    return torch.tensor(out, dtype=torch.int32, device=device)


def mix_rows(c: PagedCache, x: torch.Tensor, tiles: torch.Tensor, q_out: torch.Tensor, ff_out: torch.Tensor | None, *, heads: int, own_kv: bool = True,
             off_gate: int = 0, off_up: int = 0, ff: int = 0, act: int = 6, conv: torch.Tensor | None = None, state: torch.Tensor | None = None,
             temp: tuple[float, int] = (0.0, 0), conv_act: int = 0) -> None:
    m = _Mix()
    m.conv_act = conv_act
    m.f32, m.in_, m.ld_in, m.nq = int(c.dtype == torch.float32), _p(x), x.stride(0), heads * c.dim
    m.nk, m.nv = (c.kv_heads * c.dim, c.kv_heads * c.vdim) if own_kv else (0, 0)
    m.off_gate, m.off_up, m.ff, m.act, m.conv, m.taps = off_gate, off_up, ff, act, _p(conv), 0 if conv is None else conv.shape[0]
    m.state, m.state_half = _p(state), 0 if state is None else state[0].numel()
    m.q_out, m.ld_q, m.k_pool, m.v_pool, m.kv_heads, m.dim_p, m.vdim_p = _p(q_out), q_out.stride(0), _p(c.k), _p(c.v), c.kv_heads, c.dim, c.vdim
    m.table, m.table_ld, m.temp_coef, m.temp_every = _p(c.table), c.table.stride(0), temp[0], temp[1]
    m.ff_out, m.ld_ff = _p(ff_out), 0 if ff_out is None else ff_out.stride(0)
    m.tiles, m.n_tiles, m.tile_rows, m.rows = _p(tiles), tiles.shape[0], 1 if tiles.shape[0] == x.shape[0] else 16, x.shape[0]
    _lib.check(_lib.load().nfn_mix_rows(C.byref(m), C.c_void_p(_lib.stream_ptr())), "mix_rows")


def row_norm(x: torch.Tensor, weight: torch.Tensor, h: torch.Tensor, *, eps: float, width: int | None = None, y: torch.Tensor | None = None,
             y_weight: torch.Tensor | None = None, x_out: torch.Tensor | None = None, src_rows: torch.Tensor | None = None) -> None:
    a = _RowNorm()
    a.f32, a.rows, a.width, a.ld, a.x, a.x_out = int(h.dtype == torch.float32), h.shape[0], width or x.shape[1], x.shape[1], _p(x), _p(x_out)
    a.src_rows, a.y, a.y_weight, a.h, a.weight, a.eps = _p(src_rows), _p(y), _p(y_weight), _p(h), _p(weight), eps
    _lib.check(_lib.load().nfn_row_norm(C.byref(a), C.c_void_p(_lib.stream_ptr())), "row_norm")


def residual_gemm(a: torch.Tensor, b: torch.Tensor, x: torch.Tensor, copy: torch.Tensor, workspace: torch.Tensor | None = None) -> None:
    """x (fp32) += a . b^T (bf16 operands), copy = bf16(x): the product that feeds a 32-bit residual stream."""
    g = _lib.GemmArgs()
    g.a, g.b, g.c, g.m, g.n, g.k = _p(a), _p(b), _p(x), a.shape[0], b.shape[0], a.shape[1]
    g.lda, g.ldb, g.ldc, g.alpha = a.stride(0), b.stride(0), x.stride(0), 1.0
    g.flags = (1 << 4) | (1 << 5) | (1 << 6)                     # NFN_EPI_ACCUM | NFN_EPI_OUT_F32 | NFN_EPI_COPY_BF16
    g.aux_out, g.ld_aux_out = _p(copy), copy.stride(0)
    if workspace is not None:
        g.workspace, g.workspace_bytes = _p(workspace), workspace.numel() * workspace.element_size()
    _lib.check(_lib.load().nfn_gemm_bf16(C.byref(g), C.c_void_p(_lib.stream_ptr())), "residual_gemm")
