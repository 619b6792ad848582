"""Python API of the resident inference engine (``csrc/engine``): weights, KV caches and
activations stay on the GPU; Python passes token ids in and gets token ids back.

    eng = ResidentEngine(EngineConfig.gpt2(cfg, max_batch=8))
    eng.load_dense_checkpoint("model_00001000.bin")      # or eng.load_named_tensors(...)
    out = eng.generate([[15496, 11], [40]], max_new_tokens=32, sampling=Sampling(temperature=0.8, top_p=0.95))

``generate`` is a continuous-batching loop: prompts are prefetched into free slots as
earlier sequences finish, and every decode step advances all live slots at once. Engines of
layer-list models (``LayeredEngineConfig``) also run arbitrary steps - portions of some prompts
beside single tokens of other sequences, ``ResidentEngine.step`` - and ``generate`` drives them
through the scheduler of ``serving.scheduler``.
Counterpart of the reference's ``_native_inference`` module and its Python wrapper
(``csrc/native_gpt2/resident_binding.cpp``, ``neuralfn/native_inference.py``).
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, fields
from typing import Iterable, Sequence

import torch

from ..ops import _lib

__all__ = ["EngineConfig", "LayerSpec", "LayeredEngineConfig", "StepEntry", "Sampling", "ResidentEngine", "resident_inference_abi_version", "resident_inference_capabilities"]


class _CConfig(C.Structure):
    _fields_ = [("family", C.c_int), ("n_layer", C.c_int), ("d_model", C.c_int), ("n_head", C.c_int), ("n_kv_head", C.c_int),
                ("head_dim", C.c_int), ("d_ff", C.c_int), ("vocab", C.c_int), ("padded_vocab", C.c_int), ("max_seq", C.c_int),
                ("max_batch", C.c_int), ("qk_norm", C.c_int), ("rope_hf", C.c_int), ("rope_theta", C.c_float),
                ("norm_eps", C.c_float), ("qk_norm_eps", C.c_float), ("logit_softcap", C.c_float), ("tie_embeddings", C.c_int),
                ("window", C.c_int), ("global_every", C.c_int), ("embed_scale", C.c_float), ("use_cuda_graph", C.c_int),
                ("gated_attention", C.c_int), ("sandwich_norms", C.c_int), ("centered_norms", C.c_int), ("embed_norm", C.c_int),
                ("rope_local_only", C.c_int), ("q_scale", C.c_float), ("output_multiplier", C.c_float), ("post_norm_eps", C.c_float),
                ("mlp_activation", C.c_int), ("kv_cache_mode", C.c_int)]


class _CSampling(C.Structure):
    _fields_ = [("temperature", C.c_float), ("top_k", C.c_int), ("top_p", C.c_float), ("seed", C.c_uint64)]


@dataclass
class Sampling:
    temperature: float = 0.0
    top_k: int = 0
    top_p: float = 1.0
    seed: int = 0

    def c(self) -> _CSampling:
        return _CSampling(self.temperature, self.top_k, self.top_p, self.seed)


class _CLayer(C.Structure):
    _fields_ = [("heads", C.c_int), ("kv_heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("conv_taps", C.c_int), ("window", C.c_int),
                ("kv_from", C.c_int), ("scale", C.c_float), ("alibi", C.c_float), ("q_temp_coef", C.c_float), ("q_temp_every", C.c_int),
                ("out_gate", C.c_int), ("ff", C.c_int), ("ff_act", C.c_int), ("mixer", C.c_int), ("qkv_bias", C.c_int), ("keep_first", C.c_int),
                ("softcap", C.c_float), ("sink", C.c_int), ("rank_decay", C.c_int), ("rank_gate", C.c_int), ("experts", C.c_int), ("top", C.c_int),
                ("expert_ff", C.c_int), ("weights_of", C.c_int), ("chunk", C.c_int), ("qk_norm", C.c_int), ("rot_dims", C.c_int), ("rot_base", C.c_double),
                ("key_values", C.c_int), ("kv_rank", C.c_int), ("rot_dim", C.c_int), ("expert_plain", C.c_int), ("shared_ff", C.c_int), ("route_correction", C.c_int),
                ("route_groups", C.c_int), ("route_keep", C.c_int), ("route_normalise", C.c_int), ("route_scale", C.c_float),
                ("route_softmax", C.c_int), ("expert_weigh_out", C.c_int), ("ff_limit", C.c_float), ("ff_slope", C.c_float), ("ff_bias", C.c_int), ("decay", C.POINTER(C.c_double))]


class _CLayeredConfig(C.Structure):
    _fields_ = [("n_layer", C.c_int), ("width", C.c_int), ("vocab", C.c_int), ("side_dim", C.c_int), ("embed_scale", C.c_float),
                ("norm_eps", C.c_float), ("dtype", C.c_int), ("max_seq", C.c_int), ("max_batch", C.c_int), ("kv_tokens", C.c_int),
                ("max_step_rows", C.c_int), ("use_cuda_graph", C.c_int), ("chained", C.c_int), ("streams", C.c_int), ("untied_head", C.c_int),
                ("norm_offset", C.c_float), ("logit_scale", C.c_float), ("logit_softcap", C.c_float), ("post_norm", C.c_int), ("residual_mult", C.c_float),
                ("sandwich", C.c_int), ("scalar_norms", C.c_int), ("input_taps", C.c_int)]


class _CEntry(C.Structure):
    _fields_ = [("slot", C.c_int32), ("count", C.c_int32)]


KV_PAGE = 64   # tokens per cache page of a layer-list engine


@dataclass(frozen=True)
class LayerSpec:
    """One layer of a layer-list model (field meanings: ``nfn_layer_desc`` in csrc/engine/nfn_engine.h)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv_taps: int = 0
    window: int = 0
    kv_from: int = -1
    alibi: float = 0.0
    q_temp_coef: float = 0.0
    q_temp_every: int = 0
    out_gate: int = 0
    ff: int = 0
    ff_act: str = "relu"
    mixer: str = "attention"
    qkv_bias: int = 0
    keep_first: int = 0
    softcap: float = 0.0
    sink: int = 0
    rank_decay: int = 0
    rank_gate: int = 0
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    weights_of: int = -1
    chunk: int = 0
    qk_norm: int = 0
    rot_dims: int = 0
    rot_base: float = 0.0
    key_values: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    expert_plain: int = 0
    shared_ff: int = 0
    route_correction: int = 0
    route_groups: int = 0
    route_keep: int = 0
    route_normalise: int = 0
    route_scale: float = 0.0
    route_softmax: int = 0
    expert_weigh_out: int = 0
    ff_limit: float = 0.0
    ff_slope: float = 0.0
    ff_bias: int = 0
    decay: tuple[float, ...] = ()

    FF_ACT_IDS = {"gelu": 1, "silu": 3, "relu2": 4, "relu": 6, "clamped": 7}
    MIXER_IDS = {"attention": 0, "delta": 1, "latent": 2, "wkv": 3, "linear": 4, "gru": 5}

    def c(self) -> _CLayer:
        return _CLayer(self.heads, self.kv_heads, self.dim, self.vdim, self.conv_taps, self.window, self.kv_from, self.scale, self.alibi,
                       self.q_temp_coef, self.q_temp_every, self.out_gate, self.ff, self.FF_ACT_IDS[self.ff_act], self.MIXER_IDS[self.mixer], self.qkv_bias, self.keep_first,
                       self.softcap, self.sink, self.rank_decay, self.rank_gate, self.experts, self.top, self.expert_ff, self.weights_of,
                       self.chunk, self.qk_norm, self.rot_dims, self.rot_base, self.key_values, self.kv_rank, self.rot_dim, self.expert_plain, self.shared_ff,
                       self.route_correction, self.route_groups, self.route_keep, self.route_normalise, self.route_scale, self.route_softmax, self.expert_weigh_out, self.ff_limit,
                       self.ff_slope, self.ff_bias, (C.c_double * len(self.decay))(*self.decay) if self.decay else None)

    @property
    def paged(self) -> bool:
        return self.mixer in ("attention", "latent")

    @property
    def look(self) -> int:
        """Most positions a query sees (0: all)."""
        return self.chunk or self.window

    @property
    def cache_row(self) -> int:
        """Values one token adds to this layer's pages."""
        if self.kv_from >= 0 or not self.paged:
            return 0
        return self.kv_rank + self.rot_dim if self.mixer == "latent" else self.kv_heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class LayeredEngineConfig:
    """A model given layer by layer, served from paged caches. ``dtype`` "bfloat16": products and activations in bf16, norms, softmax,
    residual stream and constants in 32-bit; "float32": everything in 32-bit (no TF32). ``kv_tokens``: tokens the cache pool holds for
    all sequences together, each rounded up to a page of 64 (0: ``max_batch`` sequences of ``max_seq``)."""
    layers: tuple[LayerSpec, ...]
    width: int
    vocab: int
    side_dim: int = 0
    embed_scale: float = 1.0
    norm_eps: float = 1e-5
    dtype: str = "bfloat16"
    max_seq: int = 4096
    max_batch: int = 8
    kv_tokens: int = 0
    max_step_rows: int = 8192
    use_cuda_graph: int = 1
    chained: int = 0
    streams: int = 0
    untied_head: int = 0
    norm_offset: float = 0.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0
    post_norm: int = 0
    residual_mult: float = 1.0
    sandwich: int = 0
    scalar_norms: int = 0
    input_taps: int = 0

    family = 2
    kv_cache_mode = 0

    def __post_init__(self) -> None:
        if self.dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype must be bfloat16 or float32")

    @property
    def d_model(self) -> int:
        return self.width

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def window(self) -> int:
        """Most tokens behind a sequence's end whose pages stay (widest window or chunk plus kept first tokens, in whole pages) when every
        layer with pages has a limit, else 0."""
        paged = [y for y in self.layers if y.paged]
        if any(y.look == 0 for y in paged):
            return 0
        return max((y.look + (y.keep_first + KV_PAGE - 1) // KV_PAGE * KV_PAGE for y in paged), default=0)

    def create(self, lib, device: int):
        cc = _CLayeredConfig(len(self.layers), self.width, self.vocab, self.side_dim, self.embed_scale, self.norm_eps,
                             int(self.dtype == "float32"), self.max_seq, self.max_batch, self.kv_tokens, self.max_step_rows, self.use_cuda_graph, self.chained,
                             self.streams, self.untied_head, self.norm_offset, self.logit_scale, self.logit_softcap, self.post_norm, self.residual_mult,
                             self.sandwich, self.scalar_norms, self.input_taps)
        for i, y in enumerate(self.layers):
            if y.mixer == "linear" and len(y.decay) != y.heads:
                raise ValueError(f"layer {i}: {len(y.decay)} decays for {y.heads} heads")
        specs = [y.c() for y in self.layers]
        arr = (_CLayer * len(specs))(*specs)
        return lib.nfn_engine_create_layered(C.byref(cc), arr, device)

    def estimate_device_bytes(self) -> int:
        """Weights, page pools and activations of an engine with this configuration."""
        up = lambda v: (v + 15) // 16 * 16  # noqa: E731
        es, wp = (4 if self.dtype == "float32" else 2), up(self.width)
        rows = min(self.max_step_rows, max(self.max_seq, self.max_batch))
        pool = self.kv_tokens or self.max_batch * ((self.max_seq + KV_PAGE - 1) // KV_PAGE * KV_PAGE)
        weights, cache, widest, routed = wp * up(self.vocab) * (1 + self.untied_head) + self.vocab * self.n_layer * up(self.side_dim), 0, 0, 0
        for y in self.layers:
            dim, vdim = up(y.dim), up(y.vdim)
            q, v = y.heads * dim, y.heads * vdim
            if y.mixer == "delta":
                conv = 2 * y.kv_heads * dim + v
                n_in = conv + up(y.heads) + up(y.rank_decay) + up(y.rank_gate)
                own = q * up(y.rank_decay) + v * up(y.rank_gate)
                cache += self.max_batch * (4 * q * vdim + 2 * es * conv * (y.conv_taps - 1))
                widest = max(widest, n_in + conv + (4 // es) * (q + v) + 2 * v)
            elif y.mixer == "wkv":
                n_in, own = 4 * q, up(y.rank_decay) * (wp + 2 * q)
                cache += self.max_batch * 4 * (q * dim + 2 * wp)
                widest = max(widest, n_in + 5 * wp + v + (4 // es) * (2 * q + up(y.rank_decay)) + 2 * up(y.rank_decay))
            elif y.mixer == "latent":
                rank, rot = up(y.kv_rank), up(y.rot_dim)
                n_in, own = y.heads * (dim + rot) + (0 if y.kv_from >= 0 else rank + rot) + (v if y.out_gate else 0), y.heads * rank * (2 * dim + vdim)
                cache += 0 if y.kv_from >= 0 else (rank + rot) * pool * es
                short = rows if es == 4 else min(rows, 15 * self.max_batch)                # rows that attend to the latents, rows of the expansion
                cache += short * y.heads * (2 * rank + rot) * es + (0 if es == 4 else (rows + min(y.look or self.max_seq, self.max_seq) + 2 * KV_PAGE) * (rank + y.heads * (dim + vdim)) * es)
                widest = max(widest, n_in + v)
            elif y.mixer == "linear":
                n_in, own = 2 * (q + v), 0
                cache += 4 * q * vdim * self.max_batch + (0 if es == 4 or dim > 128 else min(y.heads * self.max_batch, 160) * 9 * 4 * dim * vdim // sum(z.mixer == "linear" for z in self.layers))
                widest = max(widest, n_in + v + (4 // es) * v)
            elif y.mixer == "gru":
                n_in, own = 3 * v, 0
                cache += 4 * v * self.max_batch
                widest = max(widest, n_in + v)
            else:
                kv = 0 if y.kv_from >= 0 else y.kv_heads * (dim + vdim)
                n_in, own = q + kv + (v if y.out_gate else 0) + (0 if self.chained else 2 * up(y.ff)), 0
                cache += kv * pool * es
                widest = max(widest, n_in + q + v + up(y.ff))
            cache += 2 * 2 * self.max_batch * max(self.input_taps - 1, 0) * wp * es
            if y.weights_of < 0:
                weights += wp * (n_in + v + up(y.ff) * (3 if self.chained else 1) + 2 * up(self.side_dim) + 2 * up(y.shared_ff)) + own + wp * (up(y.experts) + 3 * y.experts * up(y.expert_ff))
            routed = max(routed, (rows * y.top + 127 * y.experts) * es * (2 * wp + 3 * up(y.expert_ff)) if y.experts else 0)
        acts = rows * (es * ((4 if self.input_taps else 3) * wp + widest + up(self.side_dim)) + 4 * (wp * max(self.streams, 1) + up(self.side_dim))) + 4 * 2 * max(self.max_batch, 64) * up(self.vocab)
        chunks = (96 << 20) * sum(any(y.mixer == m for y in self.layers) for m in ("delta", "wkv")) if es == 2 else 0        # operands of the recurrences' prompt chunks
        return int(2 * weights + cache + acts + routed + chunks)


@dataclass(frozen=True)
class StepEntry:
    """The next tokens of one slot in a step; ``want``: places among them whose logits (and, with sampling, successors) are asked for."""
    slot: int
    tokens: Sequence[int]
    want: Sequence[int] = ()
    sampling: Sampling | None = None


@dataclass
class EngineConfig:
    family: int = 0                # 0 GPT-2 style, 1 Llama style
    n_layer: int = 12
    d_model: int = 768
    n_head: int = 12
    n_kv_head: int = 12
    head_dim: int = 64
    d_ff: int = 3072
    vocab: int = 50257
    padded_vocab: int = 50304
    max_seq: int = 1024
    max_batch: int = 8
    qk_norm: int = 0               # 0 none, 1 weightless, 2 weighted
    rope_hf: int = 1
    rope_theta: float = 10000.0
    norm_eps: float = 1e-5
    qk_norm_eps: float = 1e-6
    logit_softcap: float = 0.0
    tie_embeddings: int = 1
    window: int = 0
    global_every: int = 0
    embed_scale: float = 1.0
    use_cuda_graph: int = 1
    # Glimmer-style blocks (family 1): gated attention output, sandwich norms with (1 + w) scales,
    # weightless embedding norm, rotary embedding on sliding-window layers only, query scale,
    # logit multiplier
    gated_attention: int = 0
    sandwich_norms: int = 0
    centered_norms: int = 0
    embed_norm: int = 0
    rope_local_only: int = 0
    q_scale: float = 0.0
    output_multiplier: float = 0.0
    post_norm_eps: float = 0.0
    mlp_activation: int = 0       # GPT-2 family: epilogue id of the MLP activation (0 = tanh GELU); see MLP_ACTIVATION_IDS
    kv_cache_mode: int = 0        # 0: bf16 K / V rows; 1: TurboQuant 3.5-bit records (decode only: no verification blocks)

    MLP_ACTIVATION_IDS = {"gelu": 1, "silu": 3, "relu2": 4, "relu": 6}

    @classmethod
    def gpt2(cls, cfg, max_batch: int = 8, *, activation: str | None = None, **kw) -> "EngineConfig":
        """From a ``models.gpt2.GPT2Config``. ``activation``: the one a mixture-of-activations checkpoint selected
        (``checkpoint.dense.read_moa_sidecar``); default: the configuration's own."""
        kw.setdefault("mlp_activation", cls.MLP_ACTIVATION_IDS[activation or getattr(cfg, "mlp_activation", "gelu")])
        return cls(family=0, n_layer=cfg.n_layer, d_model=cfg.d_model, n_head=cfg.n_head, n_kv_head=cfg.n_head,
                   head_dim=cfg.head_dim, d_ff=cfg.mlp_mult * cfg.d_model, vocab=cfg.vocab_size, padded_vocab=cfg.padded_vocab,
                   max_seq=cfg.max_seq_len, max_batch=max_batch, qk_norm=1 if cfg.qk_norm else 0, norm_eps=cfg.ln_eps,
                   qk_norm_eps=cfg.qk_norm_eps, logit_softcap=cfg.logit_softcap, tie_embeddings=1, **kw)

    @classmethod
    def glimmer(cls, *, n_layer: int, d_model: int, n_head: int, n_kv_head: int, head_dim: int, d_ff: int, vocab: int, max_seq: int,
                window: int, max_batch: int = 8, logit_softcap: float = 20.0, **kw) -> "EngineConfig":
        """Muse-Glimmer block layout: every 4th layer global without position signal, the others
        sliding-window with rotary embedding (theta 5e5), weightless per-head QK norm with query scale
        3.87, gated attention, centered sandwich norms, output multiplier 0.19611613513818404."""
        base = dict(family=1, n_layer=n_layer, d_model=d_model, n_head=n_head, n_kv_head=n_kv_head, head_dim=head_dim, d_ff=d_ff,
                    vocab=vocab, padded_vocab=(vocab + 127) // 128 * 128, max_seq=max_seq, max_batch=max_batch, qk_norm=1, rope_hf=1,
                    rope_theta=5.0e5, norm_eps=1e-5, qk_norm_eps=1e-6, logit_softcap=logit_softcap, tie_embeddings=0, window=window,
                    global_every=4, gated_attention=1, sandwich_norms=1, centered_norms=1, embed_norm=1, rope_local_only=1,
                    q_scale=3.87, output_multiplier=0.19611613513818404, post_norm_eps=1e-8)
        base.update(kw)
        return cls(**base)

    def c(self) -> _CConfig:
        return _CConfig(*[getattr(self, f.name) for f in fields(self)])

    def create(self, lib, device: int):
        return lib.nfn_engine_create(C.byref(self.c()), device)


def _api():
    L = _lib.load()
    if getattr(L, "_engine_ready", False):
        return L
    vp, ip, ll, sp = C.c_void_p, C.c_int, C.c_longlong, C.POINTER(_CSampling)
    table = {
        "last_error": (C.c_char_p, []), "create": (vp, [C.POINTER(_CConfig), ip]), "create_layered": (vp, [C.POINTER(_CLayeredConfig), C.POINTER(_CLayer), ip]),
        "destroy": (None, [vp]), "set_tensor": (ip, [vp, C.c_char_p, vp, ll]), "set_tensor_kquant": (ip, [vp, C.c_char_p, ip, vp, ll, ll]),
        "expected_tensors": (ip, [vp, C.c_char_p, ip]), "load_dense_v5": (ip, [vp, C.c_char_p]), "finalize": (ip, [vp]), "set_turboquant": (ip, [vp, vp]),
        "device_bytes": (ll, [vp]), "prefill": (ip, [vp, ip, vp, ip, sp, vp]), "decode": (ip, [vp, vp, vp, sp, vp, vp]), "release": (ip, [vp, ip]),
        "step": (ip, [vp, vp, ip, vp, vp, ip, vp, vp, vp]), "free_tokens": (ll, [vp]), "stream": (vp, [vp]),
        "slot_length": (ip, [vp, ip]), "last_logits": (ip, [vp, ip, vp]), "launches": (ll, [vp]), "enable_verify": (ip, [vp, ip]),
        "verify": (ip, [vp, vp, vp, ip, vp]), "verify_logits": (ip, [vp, ip, ip, vp]), "commit": (ip, [vp, vp]), "truncate": (ip, [vp, ip, ip]),
        "fork": (ip, [vp, ip, ip, ip]), "prefill_rows": (ip, [vp, ip, vp, ip, ip, sp, vp]), "enable_taps": (ip, [vp, vp, ip]),
        "read_taps": (ip, [vp, ip, ip, ip, vp, ip]),
    }
    for name, (res, args) in table.items():
        fn = getattr(L, "nfn_engine_" + name, None)       # a library built for one kind of model has no creator for the other
        if fn is not None:
            fn.restype, fn.argtypes = res, args
    L._engine_ready = True
    return L


def resident_inference_abi_version() -> int:
    return int(_api().nfn_engine_abi_version())


def resident_inference_capabilities() -> dict:
    return {"abi_version": resident_inference_abi_version(), "families": ["gpt2", "llama", "layered"], "kv_cache": "bf16",
            # layer-list models: paged caches, steps of mixed prompt portions and single tokens, bf16 or true 32-bit
            "paged_kv_cache": ["layered"], "mixed_steps": ["layered"], "float32": ["layered"], "mixers": {"layered": sorted(LayerSpec.MIXER_IDS)},
            "recurrent_state": ["layered"], "routed_experts": ["layered"], "residual_streams": ["layered"],
            "hybrid_local_global": True, "qk_norm": True, "rope": ["hf", "legacy"], "continuous_batching": True,
            "cuda_graph_decode": True, "on_device_sampling": ["greedy", "temperature", "top_k", "top_p"],
            # projection weights may stay resident in K-quant blocks (``set_tensor_kquant``: quantised GEMV for up to eight rows,
            # decode-then-GEMM beyond); NF4 checkpoints are dequantised at load time; there is no int8-activation MMQ path
            "block_verification": True, "hidden_state_taps": True, "gpt2_mlp_activations": sorted(EngineConfig.MLP_ACTIVATION_IDS),
            "kv_cache_modes": ["bf16", "turboquant-3.5 (decode only)"], "quantized_weights": ["Q4_K", "Q5_K", "Q6_K"], "weight_dtypes": ["bf16", "k-quant projections (set_tensor_kquant)"],
            "dequantised_at_load": ["NF4"]}


class EngineError(RuntimeError):
    pass


class ResidentEngine:
    def __init__(self, config: "EngineConfig | LayeredEngineConfig", device: int = 0, *, turboquant_profile: str = "mse-3.5", turboquant_seed: int = 0) -> None:
        self.config = config
        self.device = int(device)
        self._L = _api()
        self._h = config.create(self._L, device)
        if not self._h:
            raise EngineError(self._err())
        self._finalized = False
        if config.kv_cache_mode == 1:
            self._set_turboquant(turboquant_profile, turboquant_seed)

    def _set_turboquant(self, profile: str, seed: int) -> None:
        """``kv_cache_mode`` 1: the codec of ``quant.turboquant`` (deterministic rotation / projection, Lloyd-Max centroids, the
        default outlier channel set) lives on the device for the engine's life; K / V are kept as its records."""
        from ..quant.turboquant import TurboQuantCodec, default_outlier_indices
        hd = self.config.head_dim
        self.turboquant = TurboQuantCodec(hd, profile=profile, seed=seed, outlier_indices=default_outlier_indices(hd))
        self._tq_tensors = t = self.turboquant.device_tables(torch.device("cuda", self.device))

        class _Tables(C.Structure):
            _fields_ = [("rotation", C.c_void_p), ("projection", C.c_void_p), ("centroids", C.c_void_p), ("key_fields", C.c_void_p),
                        ("value_fields", C.c_void_p), ("D", C.c_int), ("qjl", C.c_int), ("key_rec_bytes", C.c_int), ("value_rec_bytes", C.c_int)]
        self._tq_c = _Tables(t["rotation"].data_ptr(), t["projection"].data_ptr(), t["centroids"].data_ptr(), t["key_fields"].data_ptr(),
                             t["value_fields"].data_ptr(), hd, int(profile == "qjl-3.5"), self.turboquant.key_layout.record_bytes,
                             self.turboquant.value_layout.record_bytes)
        self._check(self._L.nfn_engine_set_turboquant(self._h, C.cast(C.byref(self._tq_c), C.c_void_p)))

    @property
    def kv_bytes_per_token(self) -> int:
        """Cache bytes one token occupies in a global (full-context) layer; in all layers together for a layer-list model."""
        c = self.config
        if c.family == 2:
            return sum(y.cache_row for y in c.layers) * (4 if c.dtype == "float32" else 2)
        if c.kv_cache_mode == 1:
            return c.n_kv_head * (self.turboquant.key_layout.record_bytes + self.turboquant.value_layout.record_bytes)
        return 2 * c.n_kv_head * c.head_dim * 2

    def _err(self) -> str:
        return (self._L.nfn_engine_last_error() or b"").decode("utf-8", "replace")

    def _check(self, rc: int) -> None:
        if rc < 0:
            raise EngineError(self._err())

    def close(self) -> None:
        if getattr(self, "_h", None):
            self._L.nfn_engine_destroy(self._h)
            self._h = None

    __del__ = close

    # ---- weights --------------------------------------------------------------------------
    def expected_tensors(self) -> dict[str, int]:
        n = self._L.nfn_engine_expected_tensors(self._h, None, 0)
        buf = C.create_string_buffer(n + 1)
        self._L.nfn_engine_expected_tensors(self._h, buf, n + 1)
        return {a: int(b) for a, b in (line.split() for line in buf.value.decode().splitlines())}

    def set_tensor(self, name: str, t: torch.Tensor) -> None:
        t = t.detach().to("cpu", torch.bfloat16).contiguous()
        self._check(self._L.nfn_engine_set_tensor(self._h, name.encode(), t.data_ptr(), t.numel()))

    QTYPES = {"Q4_K": 12, "Q5_K": 13, "Q6_K": 14}

    def set_tensor_kquant(self, name: str, qtype: int | str, blocks: torch.Tensor) -> None:
        """Keeps projection weight ``name`` resident in its K-quant blocks (uint8, rows of K / 256 super-blocks back to back - the
        GGUF layout). Decode-sized products (up to eight rows) read the blocks directly; larger ones decode the tensor into one
        shared bf16 scratch buffer first. Embeddings, norms and biases stay bf16.

        Reference counterpart: the K-quant resident weights of ``resident_glimmer_cuda.cpp`` (``weight_precision k-quant-*``)."""
        from ..ops.infer import quant_block_bytes
        q = self.QTYPES[qtype] if isinstance(qtype, str) else int(qtype)
        b = blocks.detach().to("cpu", torch.uint8).contiguous().reshape(-1)
        numel = b.numel() // quant_block_bytes(q) * 256
        self._check(self._L.nfn_engine_set_tensor_kquant(self._h, name.encode(), q, b.data_ptr(), b.numel(), numel))

    def load_named_tensors(self, tensors: dict[str, torch.Tensor], quantized: dict[str, tuple] | None = None) -> None:
        """``quantized``: name -> (qtype, uint8 blocks) for projection weights that stay in K-quant form; those names need no
        entry in ``tensors``."""
        quantized = quantized or {}
        for name, (qtype, blocks) in quantized.items():
            self.set_tensor_kquant(name, qtype, blocks)
        for name, numel in self.expected_tensors().items():
            if name in quantized:
                continue
            if name not in tensors:
                raise EngineError(f"missing tensor {name!r}")
            t = tensors[name]
            if name in ("wte", "tok_embeddings", "lm_head") and t.numel() < numel:  # pad the vocabulary rows
                pad = torch.zeros(numel // t.shape[1] - t.shape[0], t.shape[1], dtype=t.dtype)
                t = torch.cat([t.cpu(), pad])
            self.set_tensor(name, t)
        self.finalize()

    def load_dense_checkpoint(self, path) -> None:
        self._check(self._L.nfn_engine_load_dense_v5(self._h, str(path).encode()))
        self.finalize()

    def load_hf_llama_state_dict(self, sd: dict[str, torch.Tensor]) -> None:
        """Hugging Face Llama / Qwen3-style names -> the engine's fused layout (q|k|v rows
        concatenated, gate|up rows concatenated)."""
        c = self.config
        out = {"tok_embeddings": sd["model.embed_tokens.weight"], "norm": sd["model.norm.weight"]}
        if not c.tie_embeddings:
            out["lm_head"] = sd["lm_head.weight"]
        for l in range(c.n_layer):
            p = f"model.layers.{l}."
            out[f"layers.{l}.attn_norm"] = sd[p + "input_layernorm.weight"]
            out[f"layers.{l}.wqkv"] = torch.cat([sd[p + f"self_attn.{n}_proj.weight"] for n in "qkv"])
            if c.qk_norm == 2:
                out[f"layers.{l}.q_norm"] = sd[p + "self_attn.q_norm.weight"]
                out[f"layers.{l}.k_norm"] = sd[p + "self_attn.k_norm.weight"]
            out[f"layers.{l}.wo"] = sd[p + "self_attn.o_proj.weight"]
            out[f"layers.{l}.ffn_norm"] = sd[p + "post_attention_layernorm.weight"]
            out[f"layers.{l}.w_gate_up"] = torch.cat([sd[p + "mlp.gate_proj.weight"], sd[p + "mlp.up_proj.weight"]])
            out[f"layers.{l}.w_down"] = sd[p + "mlp.down_proj.weight"]
        self.load_named_tensors(out)

    def finalize(self) -> None:
        self._check(self._L.nfn_engine_finalize(self._h))
        self._finalized = True

    @property
    def device_bytes(self) -> int:
        return int(self._L.nfn_engine_device_bytes(self._h))

    @property
    def launches(self) -> int:
        return int(self._L.nfn_engine_launches(self._h))

    # ---- stepping --------------------------------------------------------------------------
    def prefill(self, slot: int, tokens: Sequence[int], sampling: Sampling | None = None) -> int:
        arr = (C.c_int32 * len(tokens))(*tokens)
        out = C.c_int32(0)
        s = (sampling or Sampling()).c()
        self._check(self._L.nfn_engine_prefill(self._h, slot, C.cast(arr, C.c_void_p), len(tokens), C.byref(s), C.cast(C.byref(out), C.c_void_p)))
        return int(out.value)

    def prefill_rows(self, slot: int, rows: torch.Tensor, sampling: Sampling | None = None) -> int:
        """Runs a prompt given as its layer-0 input rows (bf16 [n, d_model], host or this engine's device): token embeddings
        after the embedding norm, media placeholders replaced by projected media features (``serving.multimodal``)."""
        if rows.dim() != 2 or rows.shape[1] != self.config.d_model or rows.dtype != torch.bfloat16:
            raise EngineError("prefill_rows wants a bf16 [n, d_model] tensor")
        rows = rows.contiguous()
        out = C.c_int32(0)
        s = (sampling or Sampling()).c()
        self._check(self._L.nfn_engine_prefill_rows(self._h, slot, C.c_void_p(rows.data_ptr()), rows.shape[0], int(rows.is_cuda), C.byref(s),
                                                    C.cast(C.byref(out), C.c_void_p)))
        return int(out.value)

    def decode(self, tokens_in: dict[int, int], sampling: Sampling | None = None, per_slot: dict[int, Sampling] | None = None) -> dict[int, int]:
        B = self.config.max_batch
        tok = (C.c_int32 * B)()
        act = (C.c_uint8 * B)()
        for slot, t in tokens_in.items():
            tok[slot], act[slot] = t, 1
        s = (sampling or Sampling()).c()
        ps = None
        if per_slot:
            ps = (_CSampling * B)(*[(per_slot.get(b) or sampling or Sampling()).c() for b in range(B)])
        out = (C.c_int32 * B)()
        self._check(self._L.nfn_engine_decode(self._h, C.cast(tok, C.c_void_p), C.cast(act, C.c_void_p), C.byref(s),
                                              C.cast(ps, C.c_void_p) if ps is not None else None, C.cast(out, C.c_void_p)))
        return {slot: int(out[slot]) for slot in tokens_in}

    @property
    def stream(self) -> "torch.cuda.ExternalStream":
        """The stream the engine launches on, for events around its calls."""
        return torch.cuda.ExternalStream(self._L.nfn_engine_stream(self._h), device=self.device)

    # ---- steps of mixed batches (layer-list models) ----------------------------------------
    @property
    def has_steps(self) -> bool:
        return self.config.family == 2

    @property
    def has_verify(self) -> bool:
        """Block verification (speculative decoding) and truncation to any prefix."""
        return self.config.family != 2

    @property
    def free_tokens(self) -> int:
        """Tokens the cache pool still has whole pages for."""
        return int(self._L.nfn_engine_free_tokens(self._h))

    def step(self, entries: Sequence[StepEntry], *, logits: bool = False) -> tuple[list[list[int]], torch.Tensor | None]:
        """Runs the next tokens of several slots as one batch. Returns, per entry, the token drawn after each wanted place (greedy
        unless the entry has its own sampling), and with ``logits`` the fp32 rows [wanted places of all entries, vocab]."""
        tokens: list[int] = []
        want: list[int] = []
        sam: list[_CSampling] = []
        for e in entries:
            sampling = (e.sampling or Sampling()).c()
            for w in e.want:
                if not 0 <= w < len(e.tokens):
                    raise EngineError("a wanted place lies outside its entry")
                want.append(len(tokens) + w)
                sam.append(sampling)
            tokens.extend(int(t) for t in e.tokens)
        n, k = len(entries), len(want)
        ce = (_CEntry * n)(*[_CEntry(e.slot, len(e.tokens)) for e in entries])
        tok, wr, out, ps = (C.c_int32 * len(tokens))(*tokens), (C.c_int32 * k)(*want), (C.c_int32 * k)(), (_CSampling * k)(*sam)
        lg = torch.empty(k, self.config.vocab, dtype=torch.float32) if logits else None
        addr = lambda a: C.cast(a, C.c_void_p)  # noqa: E731
        self._check(self._L.nfn_engine_step(self._h, addr(ce), n, addr(tok), addr(wr), k, addr(ps), addr(out),
                                            C.c_void_p(lg.data_ptr()) if lg is not None and k else None))
        drawn = iter(out)
        return [[int(next(drawn)) for _ in e.want] for e in entries], lg

    def release(self, slot: int) -> None:
        self._check(self._L.nfn_engine_release(self._h, slot))

    def slot_length(self, slot: int) -> int:
        return int(self._L.nfn_engine_slot_length(self._h, slot))

    def last_logits(self, slot: int) -> torch.Tensor:
        out = torch.empty(self.config.vocab, dtype=torch.float32)
        self._check(self._L.nfn_engine_last_logits(self._h, slot, out.data_ptr()))
        return out

    # ---- hidden-state taps (context of a block-diffusion draft) ---------------------------------
    def enable_taps(self, layers: Sequence[int]) -> None:
        """Keep the residual stream after each listed layer (0-based) for every cached position. Call before the first decode step."""
        arr = (C.c_int32 * len(layers))(*[int(l) for l in layers])
        self._check(self._L.nfn_engine_enable_taps(self._h, C.cast(arr, C.c_void_p), len(layers)))
        self.tap_layers = tuple(int(l) for l in layers)

    def read_taps(self, slot: int, pos0: int, n: int, *, device: bool = True):
        """bf16 [n, taps * d_model] for positions [pos0, pos0 + n) of ``slot`` (a CUDA tensor, or a host tensor with ``device=False``)."""
        import torch
        width = len(getattr(self, "tap_layers", ())) * self.config.d_model
        if not width:
            raise RuntimeError("taps are not enabled on this engine")
        out = torch.empty(n, width, dtype=torch.bfloat16, device=torch.device("cuda", self.device) if device else "cpu")
        self._check(self._L.nfn_engine_read_taps(self._h, slot, pos0, n, C.c_void_p(out.data_ptr()), int(device)))
        return out

    # ---- block verification / session operations ----------------------------------------------
    def enable_verify(self, max_rows: int = 17) -> None:
        """Allocates the staging buffers for ``verify`` / ``commit`` (once)."""
        self._check(self._L.nfn_engine_enable_verify(self._h, max_rows))
        self._verify_rows = max(max_rows, getattr(self, "_verify_rows", 0))

    def verify(self, blocks: dict[int, Sequence[int]]) -> dict[int, list[int]]:
        """Runs each slot's token block at the slot's current position without touching its KV
        cache. Returns, per slot, the most likely successor after every block row."""
        if not getattr(self, "_verify_rows", 0):
            self.enable_verify()
        B = self.config.max_batch
        rows = max(len(v) for v in blocks.values())
        tok = (C.c_int32 * (B * rows))()
        live = (C.c_int32 * B)()
        for slot, ids in blocks.items():
            live[slot] = len(ids)
            for r, t in enumerate(ids):
                tok[slot * rows + r] = t
        out = (C.c_int32 * (B * rows))()
        self._check(self._L.nfn_engine_verify(self._h, C.cast(tok, C.c_void_p), C.cast(live, C.c_void_p), rows, C.cast(out, C.c_void_p)))
        self._last_verify_rows = rows
        return {slot: [int(out[slot * rows + r]) for r in range(len(ids))] for slot, ids in blocks.items()}

    def verify_logits(self, slot: int, row: int) -> torch.Tensor:
        out = torch.empty(self.config.vocab, dtype=torch.float32)
        self._check(self._L.nfn_engine_verify_logits(self._h, slot, row, out.data_ptr()))
        return out

    def commit(self, accepted: dict[int, int]) -> None:
        """Appends the first ``accepted[slot]`` rows of the last ``verify`` to the caches."""
        acc = (C.c_int32 * self.config.max_batch)()
        for slot, n in accepted.items():
            acc[slot] = n
        self._check(self._L.nfn_engine_commit(self._h, C.cast(acc, C.c_void_p)))

    def append(self, slot: int, tokens: Sequence[int], chunk: int | None = None) -> int:
        """Extends a slot that already holds tokens (``prefill`` only starts at position 0).
        Returns the most likely next token."""
        if self.has_steps:
            return self.step([StepEntry(slot, tokens, (len(tokens) - 1,))])[0][0][0]
        if not getattr(self, "_verify_rows", 0):
            self.enable_verify()
        chunk = min(chunk or self._verify_rows, self._verify_rows)
        nxt = -1
        for i in range(0, len(tokens), chunk):
            part = list(tokens[i:i + chunk])
            nxt = self.verify({slot: part})[slot][-1]
            self.commit({slot: len(part)})
        return nxt

    def truncate(self, slot: int, n: int) -> None:
        self._check(self._L.nfn_engine_truncate(self._h, slot, n))

    def fork(self, src_slot: int, dst_slot: int, n: int | None = None) -> None:
        self._check(self._L.nfn_engine_fork(self._h, src_slot, dst_slot, self.slot_length(src_slot) if n is None else n))

    def generate(self, prompts: Iterable[Sequence[int]], max_new_tokens: int = 32, sampling: Sampling | None = None,
                 eos_token: int | None = None) -> list[list[int]]:
        """Continuous batching over ``max_batch`` slots; returns the generated ids per prompt."""
        prompts = [list(p) for p in prompts]
        if self.has_steps:
            from .scheduler import StepScheduler
            sched = StepScheduler(self)
            ids = [sched.submit(p, max_new_tokens, sampling, eos_token) for p in prompts]
            done = sched.run()
            return [done[i] for i in ids]
        results: list[list[int]] = [[] for _ in prompts]
        pending = list(range(len(prompts)))[::-1]
        live: dict[int, int] = {}       # slot -> prompt index
        last: dict[int, int] = {}       # slot -> token to feed next
        free = list(range(self.config.max_batch))[::-1]
        sampling = sampling or Sampling()

        def finished(idx: int, tok: int) -> bool:
            return len(results[idx]) >= max_new_tokens or (eos_token is not None and tok == eos_token)

        while pending or live:
            while pending and free:
                idx, slot = pending.pop(), free.pop()
                tok = self.prefill(slot, prompts[idx], sampling)
                results[idx].append(tok)
                if finished(idx, tok) or len(prompts[idx]) + 1 >= self.config.max_seq:
                    self.release(slot)
                    free.append(slot)
                else:
                    live[slot], last[slot] = idx, tok
            if not live:
                continue
            nxt = self.decode({slot: last[slot] for slot in live}, sampling)
            for slot, tok in nxt.items():
                idx = live[slot]
                results[idx].append(tok)
                last[slot] = tok
                if finished(idx, tok) or self.slot_length(slot) + 1 >= self.config.max_seq:
                    self.release(slot)
                    free.append(slot)
                    del live[slot], last[slot]
        return results
