"""ctypes bindings of the layer-list engine's other kernels on torch tensors: residual streams (csrc/kernels/stream_rows.cu), the gated
delta rule (delta_*.cu), the bonus recurrence (wkv_*.cu), linear attention (linear_*.cu), the gated recurrence (gru_rows.cu), rotated heads and latent attention (head_rows.cu, latent_decode.cu,
paged_prefill.cu) and routed experts (moe.cu, moe_rows.cu, the grouped GEMM). The engine calls them from C++; these wrappers serve kernel
tests and timing."""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib
from .paged import PAGE, PagedCache, _Attention

__all__ = ["LatentCache", "delta_out", "delta_rule", "expert_choice", "expert_rows", "ff_rows", "frequencies", "group_products", "gru_rows", "head_rows", "input_conv",
           "latent_attention_rows", "latent_attention_tiles", "latent_gather", "latent_rows", "linear_rule", "linear_step", "logit_cap", "router_rows", "row_out", "shift_rows", "stream_pass", "wkv_rule", "wkv_step"]


class _Stream(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("width", C.c_int), ("ld", C.c_int), ("streams", C.c_int), ("x", C.c_void_p), ("x_out", C.c_void_p),
                ("src_rows", C.c_void_p), ("tokens", C.c_void_p), ("embed", C.c_void_p), ("embed_scale", C.c_float), ("vocab", C.c_int), ("y", C.c_void_p),
                ("y_rows", C.c_int), ("y_index", C.c_void_p), ("mix", C.c_void_p), ("out", C.c_void_p), ("in_", C.c_void_p), ("h", C.c_void_p),
                ("weight", C.c_void_p), ("eps", C.c_float), ("weight_offset", C.c_float), ("y_item", C.c_void_p), ("y_plus", C.c_void_p), ("y_weight", C.c_void_p),
                ("y_scale", C.c_float), ("scalar_norms", C.c_int), ("conv", C.c_void_p), ("conv_taps", C.c_int), ("history", C.c_void_p), ("history_half", C.c_longlong),
                ("tiles", C.c_void_p)]


class _Delta(C.Structure):
    _fields_ = [("f32", C.c_int), ("qkv", C.c_void_p), ("ld_qkv", C.c_int), ("beta", C.c_void_p), ("ld_beta", C.c_int), ("decay", C.c_void_p), ("ld_decay", C.c_int),
                ("a_log", C.c_void_p), ("dt_bias", C.c_void_p), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("dim_p", C.c_int), ("vdim_p", C.c_int),
                ("unit_eps", C.c_float), ("state", C.c_void_p), ("o", C.c_void_p), ("ld_o", C.c_int), ("seqs", C.c_void_p), ("n_seqs", C.c_int)]


class RouteRule(C.Structure):
    """``nfn_route_rule``"""
    _fields_ = [("correction", C.c_void_p), ("groups", C.c_int), ("keep_groups", C.c_int), ("normalise", C.c_int), ("scale", C.c_float), ("softmax", C.c_int)]


class _Experts(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("width", C.c_int), ("ff", C.c_int), ("experts", C.c_int), ("top", C.c_int), ("act", C.c_int),
                ("logits", C.c_void_p), ("ld_logits", C.c_int), ("h", C.c_void_p), ("ld_h", C.c_int), ("w_gate_up", C.c_void_p), ("w_down", C.c_void_p),
                ("idx", C.c_void_p), ("weight", C.c_void_p), ("order", C.c_void_p), ("offsets", C.c_void_p), ("active", C.c_void_p), ("mid", C.c_void_p),
                ("y", C.c_void_p), ("ld_y", C.c_int), ("plain", C.c_int), ("rule", RouteRule), ("shared_ff", C.c_int),
                ("shared_mid", C.c_void_p), ("w_shared_down", C.c_void_p), ("y_shared", C.c_void_p), ("weigh_output", C.c_int), ("limit", C.c_float), ("slope", C.c_float),
                ("shift", C.c_float)]


def _p(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def _call(name: str, args: C.Structure) -> None:
    _lib.check(getattr(_lib.load(), "nfn_" + name)(C.byref(args), C.c_void_p(_lib.stream_ptr())), name)


def stream_pass(x: torch.Tensor | None, h: torch.Tensor | None, *, width: int, streams: int, rows: int, ld: int, f32: bool, weight: torch.Tensor | None = None, eps: float = 1e-5,
                weight_offset: float = 0.0, x_out: torch.Tensor | None = None, src_rows: torch.Tensor | None = None, y: torch.Tensor | None = None, y_rows: int = 1,
                y_index: torch.Tensor | None = None, mix: torch.Tensor | None = None, out: torch.Tensor | None = None, into: torch.Tensor | None = None,
                tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0, y_item: torch.Tensor | None = None,
                y_plus: torch.Tensor | None = None, y_weight: torch.Tensor | None = None, y_scale: float = 1.0, scalar_norms: bool = False, conv: torch.Tensor | None = None,
                history: torch.Tensor | None = None, tiles: torch.Tensor | None = None) -> None:
    """x fp32 [rows, streams, ld]; see ``nfn_stream_args``. ``into``: weights of the streams in the next sublayer's input. conv bf16 [taps, ld], history
    [2, slots, taps - 1, ld]: the convolution of rows that are entries of their own."""
    a = _Stream(int(f32), rows, width, ld, streams, _p(x), _p(x_out), _p(src_rows), _p(tokens), _p(embed), embed_scale, 0 if embed is None else embed.shape[0], _p(y), y_rows,
                _p(y_index), _p(mix), _p(out), _p(into), _p(h), _p(weight), eps, weight_offset, _p(y_item), _p(y_plus), _p(y_weight), y_scale, int(scalar_norms), _p(conv),
                0 if conv is None else conv.shape[0], _p(history), 0 if history is None else history.stride(0), _p(tiles))
    _call("stream_pass", a)


def delta_rule(qkv: torch.Tensor, beta: torch.Tensor, decay: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, state: torch.Tensor, seqs: torch.Tensor, *,
               kv_heads: int, dim: int, unit_eps: float = 1e-6, form: str = "rows", workspace: torch.Tensor | None = None, longest: int = 0) -> torch.Tensor:
    """qkv [rows, 2 * kv_heads * dim_p + heads * vdim_p] after convolution and activation (bf16 or fp32), beta [rows, heads], decay fp32 [rows, heads * dim_p],
    state fp32 [slots, heads, dim_p, vdim_p], seqs int32 [n, 4] = first row, rows, slot, position. Returns the read-outs, fp32 [rows, heads * vdim_p].
    form: "rows" (token after token) or "chunks" (sixteen at a time, bf16; ``longest``: most rows of a sequence)."""
    _, heads, dim_p, vdim_p = state.shape
    o = torch.zeros(qkv.shape[0], heads * vdim_p, device=qkv.device)
    a = _Delta(int(qkv.dtype == torch.float32), _p(qkv), qkv.stride(0), _p(beta), beta.stride(0), _p(decay), decay.stride(0), _p(a_log), _p(dt_bias), heads, kv_heads, dim,
               dim_p, vdim_p, unit_eps, _p(state), _p(o), o.stride(0), _p(seqs), seqs.shape[0])
    if form == "rows":
        _call("delta_rows", a)
        return o
    lib = _lib.load()
    lib.nfn_delta_chunk_workspace_bytes.restype = C.c_longlong
    ws = workspace if workspace is not None else torch.empty(lib.nfn_delta_chunk_workspace_bytes(heads, dim_p, vdim_p, seqs.shape[0]), device=qkv.device, dtype=torch.uint8)
    _lib.check(lib.nfn_delta_chunks(C.byref(a), C.c_int(longest or qkv.shape[0]), C.c_void_p(_p(ws)), C.c_longlong(ws.numel()), C.c_void_p(_lib.stream_ptr())), "delta_chunks")
    return o


def delta_out(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, *, heads: int, vdim: int, eps: float) -> torch.Tensor:
    out = torch.empty_like(gate)
    vdim_p = o.shape[1] // heads
    _lib.check(_lib.load().nfn_delta_out(C.c_int(int(gate.dtype == torch.float32)), C.c_void_p(_p(o)), C.c_int(o.stride(0)), C.c_void_p(_p(gate)), C.c_int(gate.stride(0)),
                                         C.c_void_p(_p(weight)), C.c_float(eps), C.c_void_p(_p(out)), C.c_int(out.stride(0)), C.c_int(o.shape[0]), C.c_int(heads),
                                         C.c_int(vdim), C.c_int(vdim_p), C.c_void_p(_lib.stream_ptr())), "delta_out")
    return out


def _rule(correction=None, groups=0, keep=0, normalise=False, scale=1.0, softmax=False) -> RouteRule:
    return RouteRule(_p(correction), groups, keep, int(normalise), scale, int(softmax))


def expert_choice(logits: torch.Tensor, top: int, **rule) -> tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """Chosen experts [rows, top], weights, tokens per expert. ``rule``: correction (bf16 [experts]), groups, keep, normalise, scale, softmax."""
    T, E = logits.shape
    idx, weight = torch.zeros(T, top, dtype=torch.int32, device=logits.device), torch.zeros(T, top, device=logits.device)
    counts = torch.zeros(E, dtype=torch.int32, device=logits.device)
    _lib.check(_lib.load().nfn_moe_choose(C.c_void_p(_p(logits)), C.c_int(logits.stride(0)), C.c_int(T), C.c_int(E), C.c_int(top), C.byref(_rule(**rule)), C.c_void_p(_p(idx)),
                                          C.c_void_p(_p(weight)), C.c_void_p(_p(counts)), C.c_void_p(_lib.stream_ptr())), "moe_choose")
    return idx, weight, counts


def expert_rows(h: torch.Tensor, logits: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor, *, experts: int, top: int, act: int = 3, plain: bool = False,
                shared_mid: torch.Tensor | None = None, shared_down: torch.Tensor | None = None, y_shared: torch.Tensor | None = None, weigh_output: bool = False,
                clamp: tuple[float, float, float] = (0.0, 0.0, 0.0), **rule):
    """Returns the chosen experts [rows, top], their weights and outputs y [rows, top, width]. plain: w_gate_up holds one matrix per expert. shared_mid [rows, f],
    shared_down [width, f]: y_shared [rows, width] is their product. clamp: limit, slope and shift of activation 7."""
    rows, width, ff = h.shape[0], h.shape[1], w_down.shape[2]
    i32 = dict(dtype=torch.int32, device=h.device)
    idx, order, offsets, active = (torch.zeros(n, **i32) for n in (rows * top, rows * top, experts + 1, experts + 1))
    weight = torch.zeros(rows * top, device=h.device)
    mid, y = torch.zeros(rows * top, ff, device=h.device, dtype=h.dtype), torch.zeros(rows * top, width, device=h.device, dtype=h.dtype)
    a = _Experts(int(h.dtype == torch.float32), rows, width, ff, experts, top, act, _p(logits), logits.stride(0), _p(h), h.stride(0), _p(w_gate_up), _p(w_down), _p(idx),
                 _p(weight), _p(order), _p(offsets), _p(active), _p(mid), _p(y), y.stride(0), int(plain), _rule(**rule), 0 if shared_mid is None else shared_mid.shape[1], _p(shared_mid),
                 _p(shared_down), _p(y_shared), int(weigh_output), *clamp)
    _call("moe_rows", a)
    return idx.view(rows, top), weight.view(rows, top), y.view(rows, top, width)


def router_rows(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h bf16 [rows, width], w bf16 [experts, width] -> fp32 [rows, experts]."""
    out = torch.zeros(h.shape[0], w.shape[0], device=h.device)
    _lib.check(_lib.load().nfn_router_rows(C.c_void_p(_p(h)), C.c_int(h.stride(0)), C.c_void_p(_p(w)), C.c_int(h.shape[0]), C.c_int(w.shape[0]), C.c_int(h.shape[1]), C.c_void_p(_p(out)),
                                           C.c_int(out.stride(0)), C.c_void_p(_lib.stream_ptr())), "router_rows")
    return out


def logit_cap(logits: torch.Tensor, scale: float, cap: float) -> None:
    _lib.check(_lib.load().nfn_logit_cap(C.c_void_p(_p(logits)), C.c_int(logits.stride(0)), C.c_int(logits.shape[0]), C.c_int(logits.shape[1]), C.c_float(scale),
                                         C.c_float(cap), C.c_void_p(_lib.stream_ptr())), "logit_cap")


# ---- rotated heads, latent attention -------------------------------------------------------------------------------------------
class _Heads(C.Structure):
    _fields_ = [("f32", C.c_int), ("in_", C.c_void_p), ("ld_in", C.c_int), ("off_k", C.c_int), ("off_v", C.c_int), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int),
                ("dim_p", C.c_int), ("vdim_p", C.c_int), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("eps", C.c_float), ("freq", C.c_void_p), ("rot_dims", C.c_int),
                ("q_out", C.c_void_p), ("ld_q", C.c_int), ("k_pool", C.c_void_p), ("v_pool", C.c_void_p), ("table", C.c_void_p), ("table_ld", C.c_int), ("tiles", C.c_void_p),
                ("n_tiles", C.c_int), ("tile_rows", C.c_int)]


class _Latent(C.Structure):
    _fields_ = [("f32", C.c_int), ("in_", C.c_void_p), ("ld_in", C.c_int), ("off_kv", C.c_int), ("heads", C.c_int), ("dim_p", C.c_int), ("rot_dim", C.c_int), ("rot_p", C.c_int),
                ("rank", C.c_int), ("rank_p", C.c_int), ("c_norm", C.c_void_p), ("eps", C.c_float), ("freq", C.c_void_p), ("q_out", C.c_void_p), ("ld_q", C.c_int),
                ("q_row0", C.c_int), ("q_lat", C.c_void_p), ("k_pool", C.c_void_p), ("table", C.c_void_p), ("table_ld", C.c_int), ("tiles", C.c_void_p), ("n_tiles", C.c_int),
                ("tile_rows", C.c_int)]


class _Groups(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("groups", C.c_int), ("n", C.c_int), ("k", C.c_int), ("in_", C.c_void_p), ("ld_in", C.c_longlong), ("in_group", C.c_longlong),
                ("w", C.c_void_p), ("out", C.c_void_p), ("ld_out", C.c_longlong), ("out_group", C.c_longlong), ("act", C.c_int), ("tail_n", C.c_int), ("tail_in", C.c_longlong),
                ("tail_w", C.c_void_p), ("tail_out", C.c_void_p), ("ld_tail", C.c_int), ("gate", C.c_void_p), ("ld_gate", C.c_longlong), ("gate_group", C.c_longlong)]


class _Expanded(C.Structure):
    _fields_ = [("x", C.c_void_p), ("x_rows", C.c_int), ("dim_u", C.c_int), ("rot_p", C.c_int), ("rank_p", C.c_int), ("x_base", C.c_void_p)]


def frequencies(dims: int, base: float, device) -> torch.Tensor:
    """base^(-2i / dims) in two fp32 parts, [dims / 2, 2]."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    hi = f.float()
    return torch.stack([hi, (f - hi.double()).float()], 1).contiguous().to(device)


def head_rows(c: PagedCache, x: torch.Tensor, tiles: torch.Tensor, q_out: torch.Tensor, *, heads: int, dim: int, freq: torch.Tensor | None, rot_dims: int, eps: float,
              q_norm: torch.Tensor | None = None, k_norm: torch.Tensor | None = None, key_values: bool = False) -> None:
    """x: rows [q | k | v] (``key_values``: [q | k]); tiles: ``ops.paged.row_tiles``."""
    off_k = heads * c.dim
    a = _Heads(int(c.dtype == torch.float32), _p(x), x.stride(0), off_k, off_k + (0 if key_values else c.kv_heads * c.dim), heads, c.kv_heads, dim, c.dim, c.vdim, _p(q_norm), _p(k_norm), eps,
               _p(freq), rot_dims, _p(q_out), q_out.stride(0), _p(c.k), _p(c.v), _p(c.table), c.table.stride(0), _p(tiles), tiles.shape[0], 1 if tiles.shape[0] == x.shape[0] else 16)
    _call("head_rows", a)


class LatentCache:
    """The pages of one latent layer, [page][64][rank_p + rot_p], a page table per slot, workspace."""

    def __init__(self, slots: int, max_seq: int, rank: int, rot: int, device, dtype=torch.bfloat16, seed: int = 0) -> None:
        self._c = PagedCache(slots, max_seq, 1, rank + rot, 16, device, dtype, seed)
        self.k, self.table, self.ws, self.rank, self.rot, self.dtype = self._c.k, self._c.table, self._c.ws, rank, rot, dtype

    def write(self, slot: int, rows: torch.Tensor) -> None:
        """rows [n, rank + rot] to positions 0 .. n - 1."""
        for p in range((rows.shape[0] + PAGE - 1) // PAGE):
            part = rows[p * PAGE:(p + 1) * PAGE]
            self.k[int(self.table[slot, p]), 0, :part.shape[0]] = part.to(self.dtype)

    def args(self, q: torch.Tensor, out: torch.Tensor, heads: int, window: int, scale: float, sinks: torch.Tensor | None = None) -> _Attention:
        a = _Attention()
        a.sinks = _p(sinks)
        a.f32, a.q, a.ld_q, a.k_pool, a.pages = int(self.dtype == torch.float32), _p(q), q.stride(0), _p(self.k), self.k.shape[0]
        a.table, a.table_ld, a.heads, a.window, a.scale, a.out, a.ld_o = _p(self.table), self.table.stride(0), heads, window, scale, _p(out), out.stride(0)
        a.workspace, a.workspace_bytes, a.total_rows = _p(self.ws), self.ws.numel(), q.shape[0]
        return a


def latent_rows(c: LatentCache, x: torch.Tensor, tiles: torch.Tensor, *, heads: int, dim: int, rot_dim: int, rank: int, c_norm: torch.Tensor, eps: float, freq: torch.Tensor,
                q_row0: int = 0, q_lat: torch.Tensor | None = None) -> None:
    """x: rows [heads x (dim | rot) | latent | key part], rotated in place; rows before ``q_row0`` have their rotated parts in ``q_lat``."""
    a = _Latent(int(c.dtype == torch.float32), _p(x), x.stride(0), heads * (dim + c.rot), heads, dim, rot_dim, c.rot, rank, c.rank, _p(c_norm), eps, _p(freq), _p(x), x.stride(0), q_row0,
                _p(q_lat), _p(c.k), _p(c.table), c.table.stride(0), _p(tiles), tiles.shape[0], 1 if tiles.shape[0] == x.shape[0] else 16)
    _call("latent_rows", a)


def group_products(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, act: int = 0, tail_w: torch.Tensor | None = None, tail_out: torch.Tensor | None = None,
                   tail_in: int = 0, gate: torch.Tensor | None = None) -> torch.Tensor:
    """x [rows, groups, k], w bf16 [groups, n, k] -> out [rows, groups, n] (any strides over rows and groups); tail_w bf16 [m, k]: one more product, of the input
    ``tail_in`` elements into each row, into tail_out fp32 [rows, m]. gate [rows, groups, n]: its sigmoid multiplies the result."""
    a = _Groups(int(x.dtype == torch.float32), x.shape[0], w.shape[0], w.shape[1], w.shape[2], _p(x), x.stride(0), x.stride(1), _p(w), _p(out), out.stride(0), out.stride(1), act,
                0 if tail_w is None else tail_w.shape[0], tail_in, _p(tail_w), _p(tail_out), 0 if tail_out is None else tail_out.stride(0),
                _p(gate), 0 if gate is None else gate.stride(0), 0 if gate is None else gate.stride(1))
    _call("group_products", a)
    return out


def latent_attention_rows(c: LatentCache, q: torch.Tensor, row_slot: torch.Tensor, row_pos: torch.Tensor, out: torch.Tensor, *, heads: int, window: int, scale: float,
                          max_keys: int = 0, sinks: torch.Tensor | None = None) -> torch.Tensor:
    """q [rows, heads * (rank + rot)], out [rows, heads * rank]: sums of latents."""
    a = c.args(q, out, heads, window, scale, sinks)
    a.kv_heads, a.dim_p, a.vdim_p = 1, c.rank + c.rot, c.rank
    a.row_slot, a.row_pos, a.rows, a.max_keys = _p(row_slot), _p(row_pos), q.shape[0], max_keys or window or c.table.shape[1] * PAGE
    _call("paged_attention_rows", a)
    return out


def latent_gather(c: LatentCache, spans: torch.Tensor, out: torch.Tensor, max_pages: int | None = None) -> torch.Tensor:
    """spans int32 [n, 4] = slot, first page, pages, first row of ``out`` [rows, rank]."""
    _lib.check(_lib.load().nfn_latent_gather(C.c_int(int(c.dtype == torch.float32)), C.c_void_p(_p(c.k)), C.c_int(c.rank + c.rot), C.c_int(c.rank), C.c_void_p(_p(c.table)),
                                             C.c_int(c.table.stride(0)), C.c_void_p(_p(spans)), C.c_int(spans.shape[0]), C.c_int(max_pages or int(spans[:, 2].max())), C.c_void_p(_p(out)),
                                             C.c_void_p(_lib.stream_ptr())), "latent_gather")
    return out


def latent_attention_tiles(c: LatentCache, q: torch.Tensor, x: torch.Tensor, x_base: torch.Tensor, tiles: torch.Tensor, out: torch.Tensor, *, heads: int, dim: int, vdim: int,
                           window: int, scale: float, sinks: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> torch.Tensor:
    """q [rows, heads * (dim + rot)]; x [n, heads * dim keys | heads * vdim values] formed from the gathered latents; tiles as in ``ops.paged.attention_tiles``."""
    a = c.args(q, out, heads, window, scale, sinks)
    a.gate, a.ld_gate = _p(gate), 0 if gate is None else gate.stride(0)
    a.kv_heads, a.dim_p, a.vdim_p, a.tiles, a.n_tiles = heads, dim + c.rot, vdim, _p(tiles), tiles.shape[0]
    e = _Expanded(_p(x), x.shape[0], dim, c.rot, c.rank, _p(x_base))
    _lib.check(_lib.load().nfn_latent_attention_tiles(C.byref(a), C.byref(e), C.c_void_p(_lib.stream_ptr())), "latent_attention_tiles")
    return out


# ---- time mixing ---------------------------------------------------------------------------------------------------------------
class _Shift(C.Structure):
    _fields_ = [("f32", C.c_int), ("src_act", C.c_int), ("width", C.c_int), ("ld", C.c_int), ("n", C.c_int), ("src", C.c_void_p), ("mu", C.c_void_p), ("prev", C.c_void_p),
                ("prev_half", C.c_longlong), ("out", C.c_void_p), ("out_stride", C.c_longlong), ("tiles", C.c_void_p), ("n_tiles", C.c_int)]


class _Wkv(C.Structure):
    _fields_ = [("f32", C.c_int), ("rkv", C.c_void_p), ("ld_rkv", C.c_int), ("z", C.c_void_p), ("ld_z", C.c_int), ("w0", C.c_void_p), ("u", C.c_void_p), ("heads", C.c_int), ("dim", C.c_int),
                ("dim_p", C.c_int), ("state", C.c_void_p), ("o", C.c_void_p), ("ld_o", C.c_int), ("seqs", C.c_void_p), ("n_seqs", C.c_int)]


class _WkvStep(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("rkvg", C.c_void_p), ("ld_rkvg", C.c_int), ("low", C.c_void_p), ("ld_low", C.c_int), ("rank_p", C.c_int), ("w2", C.c_void_p),
                ("ld_w2", C.c_int), ("w0", C.c_void_p), ("u", C.c_void_p), ("heads", C.c_int), ("dim", C.c_int), ("dim_p", C.c_int), ("state", C.c_void_p), ("weight", C.c_void_p),
                ("eps", C.c_float), ("out", C.c_void_p), ("ld_out", C.c_int), ("tiles", C.c_void_p)]


def shift_rows(src: torch.Tensor, mu: torch.Tensor, prev: torch.Tensor, out: torch.Tensor, tiles: torch.Tensor) -> torch.Tensor:
    """src [rows, ld], mu bf16 [n, ld], prev fp32 [2, slots, ld], out [n, rows, ld]."""
    a = _Shift(int(out.dtype == torch.float32), int(src.dtype == torch.bfloat16), src.shape[1], src.shape[1], mu.shape[0], _p(src), _p(mu), _p(prev), prev.stride(0), _p(out), out.stride(0),
               _p(tiles), tiles.shape[0])
    _call("shift_rows", a)
    return out


def wkv_rule(rkv: torch.Tensor, z: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, state: torch.Tensor, seqs: torch.Tensor, *, dim: int, form: str = "rows",
             workspace: torch.Tensor | None = None, longest: int = 0) -> torch.Tensor:
    """rkv [rows, 3 * heads * dim_p], z fp32 [rows, heads * dim_p], state fp32 [slots, heads, dim_p, dim_p], seqs int32 [n, 4] = first row, rows, slot, position.
    Returns the read-outs, fp32 [rows, heads * dim_p]. form: "rows" or "chunks"."""
    _, heads, dim_p, _ = state.shape
    o = torch.zeros(rkv.shape[0], heads * dim_p, device=rkv.device)
    a = _Wkv(int(rkv.dtype == torch.float32), _p(rkv), rkv.stride(0), _p(z), z.stride(0), _p(w0), _p(u), heads, dim, dim_p, _p(state), _p(o), o.stride(0), _p(seqs), seqs.shape[0])
    if form == "rows":
        _call("wkv_rows", a)
        return o
    lib = _lib.load()
    lib.nfn_wkv_chunk_workspace_bytes.restype = C.c_longlong
    ws = workspace if workspace is not None else torch.empty(lib.nfn_wkv_chunk_workspace_bytes(heads, dim_p, seqs.shape[0]), device=rkv.device, dtype=torch.uint8)
    _lib.check(lib.nfn_wkv_chunks(C.byref(a), C.c_int(longest or rkv.shape[0]), C.c_void_p(_p(ws)), C.c_longlong(ws.numel()), C.c_void_p(_lib.stream_ptr())), "wkv_chunks")
    return o


def wkv_step(rkvg: torch.Tensor, low: torch.Tensor, w2: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, state: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, tiles: torch.Tensor,
             *, dim: int, eps: float) -> torch.Tensor:
    """One token per row: rkvg [rows, 4 * heads * dim_p], low fp32 [rows, rank_p], w2 bf16 [heads * dim_p, >= rank_p]."""
    _, heads, dim_p, _ = state.shape
    a = _WkvStep(int(rkvg.dtype == torch.float32), rkvg.shape[0], _p(rkvg), rkvg.stride(0), _p(low), low.stride(0), low.shape[1], _p(w2), w2.stride(0), _p(w0), _p(u), heads, dim, dim_p,
                 _p(state), _p(weight), eps, _p(out), out.stride(0), _p(tiles))
    _call("wkv_step", a)
    return out


class _Clamp(C.Structure):
    _fields_ = [("limit", C.c_float), ("slope", C.c_float), ("shift", C.c_float)]


def ff_rows(x: torch.Tensor, out: torch.Tensor, *, off_gate: int, off_up: int, act: int, clamp: tuple[float, float, float] = (0.0, 0.0, 0.0)) -> torch.Tensor:
    _lib.check(_lib.load().nfn_ff_rows(C.c_int(int(x.dtype == torch.float32)), C.c_void_p(_p(x)), C.c_int(x.stride(0)), C.c_int(off_gate), C.c_int(off_up), C.c_int(out.shape[1]),
                                       C.c_int(act), C.byref(_Clamp(*clamp)), C.c_void_p(_p(out)), C.c_int(out.stride(0)), C.c_int(x.shape[0]), C.c_void_p(_lib.stream_ptr())), "ff_rows")
    return out


# ---- linear attention, gated recurrence, convolutions on a sublayer's input ------------------------------------------------------
class _Linear(C.Structure):
    _fields_ = [("f32", C.c_int), ("qkv", C.c_void_p), ("ld_qkv", C.c_int), ("powers", C.c_void_p), ("heads", C.c_int), ("dim_p", C.c_int), ("vdim_p", C.c_int), ("state", C.c_void_p),
                ("o", C.c_void_p), ("ld_o", C.c_int), ("seqs", C.c_void_p), ("n_seqs", C.c_int)]


class _LinearStep(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("qkvg", C.c_void_p), ("ld_qkvg", C.c_int), ("powers", C.c_void_p), ("heads", C.c_int), ("vdim", C.c_int), ("dim_p", C.c_int),
                ("vdim_p", C.c_int), ("state", C.c_void_p), ("o", C.c_void_p), ("ld_o", C.c_int), ("counters", C.c_void_p), ("weight", C.c_void_p), ("eps", C.c_float), ("out", C.c_void_p),
                ("ld_out", C.c_int), ("tiles", C.c_void_p)]


class _Gru(C.Structure):
    _fields_ = [("f32", C.c_int), ("width", C.c_int), ("in_", C.c_void_p), ("ld_in", C.c_int), ("state", C.c_void_p), ("out", C.c_void_p), ("ld_out", C.c_int), ("seqs", C.c_void_p),
                ("n_seqs", C.c_int), ("n_short", C.c_int)]


class _InputConv(C.Structure):
    _fields_ = [("f32", C.c_int), ("ld", C.c_int), ("taps", C.c_int), ("h", C.c_void_p), ("conv", C.c_void_p), ("history", C.c_void_p), ("history_half", C.c_longlong), ("out", C.c_void_p),
                ("tiles", C.c_void_p), ("n_tiles", C.c_int)]


LINEAR_CHUNK = 64


def powers(decay, device) -> torch.Tensor:
    """decay_h^0 .. decay_h^LINEAR_CHUNK, fp32 [heads, LINEAR_CHUNK + 1]."""
    d = torch.tensor(list(decay), dtype=torch.float64)[:, None]
    return (d ** torch.arange(LINEAR_CHUNK + 1, dtype=torch.float64)).float().contiguous().to(device)


def linear_rule(qkv: torch.Tensor, pw: torch.Tensor, state: torch.Tensor, seqs: torch.Tensor, *, form: str = "rows", workspace: torch.Tensor | None = None, longest: int = 0) -> torch.Tensor:
    """qkv [rows, heads * (2 dim_p + vdim_p)] after its activation, state fp32 [slots, heads, dim_p, vdim_p], seqs int32 [n, 4] = first row, rows, slot, position. Returns
    the read-outs, fp32 [rows, heads * vdim_p]. form: "rows" or "chunks" (without a workspace of its own: segments side by side where they pay)."""
    _, heads, dim_p, vdim_p = state.shape
    o = torch.zeros(qkv.shape[0], heads * vdim_p, device=qkv.device)
    a = _Linear(int(qkv.dtype == torch.float32), _p(qkv), qkv.stride(0), _p(pw), heads, dim_p, vdim_p, _p(state), _p(o), o.stride(0), _p(seqs), seqs.shape[0])
    if form == "rows":
        _call("linear_rows", a)
        return o
    lib = _lib.load()
    lib.nfn_linear_chunk_workspace_bytes.restype = C.c_longlong
    ws = workspace if workspace is not None else torch.empty(lib.nfn_linear_chunk_workspace_bytes(heads, dim_p, vdim_p, seqs.shape[0]), device=qkv.device, dtype=torch.uint8)
    _lib.check(lib.nfn_linear_chunks(C.byref(a), C.c_int(longest or qkv.shape[0]), C.c_void_p(_p(ws)), C.c_longlong(ws.numel()), C.c_void_p(_lib.stream_ptr())), "linear_chunks")
    return o


def linear_step(qkvg: torch.Tensor, pw: torch.Tensor, state: torch.Tensor, weight: torch.Tensor, out: torch.Tensor, tiles: torch.Tensor, counters: torch.Tensor, *, vdim: int, eps: float) -> torch.Tensor:
    """One token per row: qkvg [rows, heads * (2 dim_p + 2 vdim_p)] before its activations; counters int32 [rows], zero (and zero again afterwards)."""
    _, heads, dim_p, vdim_p = state.shape
    o = torch.zeros(qkvg.shape[0], heads * vdim_p, device=qkvg.device)
    a = _LinearStep(int(qkvg.dtype == torch.float32), qkvg.shape[0], _p(qkvg), qkvg.stride(0), _p(pw), heads, vdim, dim_p, vdim_p, _p(state), _p(o), o.stride(0), _p(counters), _p(weight), eps,
                    _p(out), out.stride(0), _p(tiles))
    _call("linear_step", a)
    return out


def row_out(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, *, live: int, eps: float) -> torch.Tensor:
    out = torch.empty_like(gate)
    _lib.check(_lib.load().nfn_row_out(C.c_int(int(gate.dtype == torch.float32)), C.c_void_p(_p(o)), C.c_int(o.stride(0)), C.c_void_p(_p(gate)), C.c_int(gate.stride(0)), C.c_void_p(_p(weight)),
                                       C.c_float(eps), C.c_void_p(_p(out)), C.c_int(out.stride(0)), C.c_int(o.shape[0]), C.c_int(o.shape[1]), C.c_int(live), C.c_void_p(_lib.stream_ptr())), "row_out")
    return out


def gru_rows(x: torch.Tensor, state: torch.Tensor, out: torch.Tensor, seqs: torch.Tensor, n_short: int) -> torch.Tensor:
    """x [rows, 3 * width], state fp32 [slots, width], out [rows, width], seqs as in ``linear_rule``, the first ``n_short`` of them of few rows."""
    a = _Gru(int(x.dtype == torch.float32), state.shape[1], _p(x), x.stride(0), _p(state), _p(out), out.stride(0), _p(seqs), seqs.shape[0], n_short)
    _call("gru_rows", a)
    return out


def input_conv(h: torch.Tensor, conv: torch.Tensor, history: torch.Tensor, out: torch.Tensor, tiles: torch.Tensor) -> torch.Tensor:
    """h, out [rows, ld], conv bf16 [taps, ld], history [2, slots, taps - 1, ld] of h's type."""
    a = _InputConv(int(h.dtype == torch.float32), h.shape[1], conv.shape[0], _p(h), _p(conv), _p(history), history.stride(0), _p(out), _p(tiles), tiles.shape[0])
    _call("input_conv", a)
    return out
