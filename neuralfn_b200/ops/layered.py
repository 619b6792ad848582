"""ctypes bindings of the layer-list engine's other kernels on torch tensors: residual streams (csrc/kernels/stream_rows.cu), the gated
delta rule (delta_*.cu) and routed experts (moe.cu, moe_rows.cu, the grouped GEMM). The engine calls them from C++; these wrappers serve
kernel tests and timing."""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib

__all__ = ["delta_out", "delta_rule", "expert_rows", "logit_cap", "stream_pass"]


class _Stream(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("width", C.c_int), ("ld", C.c_int), ("streams", C.c_int), ("x", C.c_void_p), ("x_out", C.c_void_p),
                ("src_rows", C.c_void_p), ("tokens", C.c_void_p), ("embed", C.c_void_p), ("embed_scale", C.c_float), ("vocab", C.c_int), ("y", C.c_void_p),
                ("y_rows", C.c_int), ("y_index", C.c_void_p), ("mix", C.c_void_p), ("out", C.c_void_p), ("in_", C.c_void_p), ("h", C.c_void_p),
                ("weight", C.c_void_p), ("eps", C.c_float), ("weight_offset", C.c_float), ("y_item", C.c_void_p), ("y_plus", C.c_void_p), ("y_weight", C.c_void_p),
                ("y_scale", C.c_float)]


class _Delta(C.Structure):
    _fields_ = [("f32", C.c_int), ("qkv", C.c_void_p), ("ld_qkv", C.c_int), ("beta", C.c_void_p), ("ld_beta", C.c_int), ("decay", C.c_void_p), ("ld_decay", C.c_int),
                ("a_log", C.c_void_p), ("dt_bias", C.c_void_p), ("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("dim_p", C.c_int), ("vdim_p", C.c_int),
                ("unit_eps", C.c_float), ("state", C.c_void_p), ("o", C.c_void_p), ("ld_o", C.c_int), ("seqs", C.c_void_p), ("n_seqs", C.c_int)]


class RouteRule(C.Structure):
    """``nfn_route_rule``"""
    _fields_ = [("correction", C.c_void_p), ("groups", C.c_int), ("keep_groups", C.c_int), ("normalise", C.c_int), ("scale", C.c_float)]


class _Experts(C.Structure):
    _fields_ = [("f32", C.c_int), ("rows", C.c_int), ("width", C.c_int), ("ff", C.c_int), ("experts", C.c_int), ("top", C.c_int), ("act", C.c_int),
                ("logits", C.c_void_p), ("ld_logits", C.c_int), ("h", C.c_void_p), ("ld_h", C.c_int), ("w_gate_up", C.c_void_p), ("w_down", C.c_void_p),
                ("idx", C.c_void_p), ("weight", C.c_void_p), ("order", C.c_void_p), ("offsets", C.c_void_p), ("active", C.c_void_p), ("mid", C.c_void_p),
                ("y", C.c_void_p), ("ld_y", C.c_int), ("plain", C.c_int), ("rule", RouteRule)]


def _p(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def _call(name: str, args: C.Structure) -> None:
    _lib.check(getattr(_lib.load(), "nfn_" + name)(C.byref(args), C.c_void_p(_lib.stream_ptr())), name)


def stream_pass(x: torch.Tensor | None, h: torch.Tensor | None, *, width: int, streams: int, rows: int, ld: int, f32: bool, weight: torch.Tensor | None = None, eps: float = 1e-5,
                weight_offset: float = 0.0, x_out: torch.Tensor | None = None, src_rows: torch.Tensor | None = None, y: torch.Tensor | None = None, y_rows: int = 1,
                y_index: torch.Tensor | None = None, mix: torch.Tensor | None = None, out: torch.Tensor | None = None, into: torch.Tensor | None = None,
                tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0) -> None:
    """x fp32 [rows, streams, ld]; see ``nfn_stream_args``. ``into``: weights of the streams in the next sublayer's input."""
    a = _Stream(int(f32), rows, width, ld, streams, _p(x), _p(x_out), _p(src_rows), _p(tokens), _p(embed), embed_scale, 0 if embed is None else embed.shape[0], _p(y), y_rows,
                _p(y_index), _p(mix), _p(out), _p(into), _p(h), _p(weight), eps, weight_offset)
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


def expert_rows(h: torch.Tensor, logits: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor, *, experts: int, top: int, act: int = 3):
    """Returns the chosen experts [rows, top], their weights and outputs y [rows, top, width]."""
    rows, width, ff = h.shape[0], h.shape[1], w_down.shape[2]
    i32 = dict(dtype=torch.int32, device=h.device)
    idx, order, offsets, active = (torch.zeros(n, **i32) for n in (rows * top, rows * top, experts + 1, experts + 1))
    weight = torch.zeros(rows * top, device=h.device)
    mid, y = torch.zeros(rows * top, ff, device=h.device, dtype=h.dtype), torch.zeros(rows * top, width, device=h.device, dtype=h.dtype)
    a = _Experts(int(h.dtype == torch.float32), rows, width, ff, experts, top, act, _p(logits), logits.stride(0), _p(h), h.stride(0), _p(w_gate_up), _p(w_down), _p(idx),
                 _p(weight), _p(order), _p(offsets), _p(active), _p(mid), _p(y), y.stride(0))
    _call("moe_rows", a)
    return idx.view(rows, top), weight.view(rows, top), y.view(rows, top, width)


def logit_cap(logits: torch.Tensor, scale: float, cap: float) -> None:
    _lib.check(_lib.load().nfn_logit_cap(C.c_void_p(_p(logits)), C.c_int(logits.stride(0)), C.c_int(logits.shape[0]), C.c_int(logits.shape[1]), C.c_float(scale),
                                         C.c_float(cap), C.c_void_p(_lib.stream_ptr())), "logit_cap")
