"""Prefill and decode throughput of Bulidra, Murilorn or Vopozen and, at equal size, of Glimmer blocks - the closest model the engine served before:
grouped heads, sliding windows, gated attention, gated feed-forward; of Kidolorn beside Vopozen. Random bf16 weights; one JSON line per model, size and
phase.

Murilorn at equal size: delta-rule and attention layers in turn with the same heads, the same active feed-forward width (four of thirty-two
experts), four residual streams. Vopozen at equal size: chunked attention, latent attention, time mixing and latent attention on the earlier layer's
cache in turn, the same heads, gated and routed feed-forwards in turn with the same active weights (four of thirty-two plain experts and a shared
one). Kidolorn at equal size: linear attention, latent attention, the gated recurrence (as wide as all heads together) and latent attention on the
earlier layer's cache in turn, without windows; dense and routed feed-forwards in turn (four of thirty-two gated experts).

``ms`` is device time (CUDA events on the engine's stream, median over repetitions of the public ``prefill`` / ``decode`` call,
including its host-to-device copy of tokens and the read-back of the drawn token); weights and caches are larger than L2. Beside it
stand the bytes (decode) or floating-point operations (prefill) the phase cannot avoid and the fraction of the measured peaks.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, ff=5632, window=1024, layers=8, vocab=32768),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, ff=14336, window=1024, layers=6, vocab=32768),
    "w4096_wide_window": dict(width=4096, heads=32, kv_heads=8, dim=128, ff=14336, window=4096, layers=6, vocab=32768),
}
SIDE_DIM = 256
EXPERTS, TOP, STREAMS, RANK, KEEP = 32, 4, 4, 128, 4
LATENT, ROT, DECAY = 512, 64, 64
VOPOZEN = ("attention", "latent", "wkv", "reader")
KIDOLORN = ("lightning", "latent", "mingru", "reader")
BESIDE = {"kidolorn": "vopozen"}                    # the closest model; others: Glimmer blocks


def _peaks() -> tuple[float, float]:
    path = os.path.join(os.path.dirname(__file__), "..", "..", "MEASURED_PEAKS.json")
    if os.path.exists(path):
        p = json.load(open(path))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


def _engine(kind: str, z: dict, max_batch: int, max_seq: int):
    from ..models.bulidra import BulidraConfig, BulidraLayer, engine_config
    from ..models import kidolorn as Q, murilorn as M, vopozen as V
    from ..serving import EngineConfig, ResidentEngine
    L = z["layers"]
    if kind == "murilorn":
        ex = dict(experts=EXPERTS, top=TOP, expert_ff=z["ff"] // TOP)
        pair = (M.MurilornLayer("channel_delta", z["heads"], z["heads"], z["dim"], z["dim"], conv=4, rank_decay=RANK, rank_gate=RANK, **ex),
                M.MurilornLayer("attention", z["heads"], z["kv_heads"], z["dim"], z["dim"], scale=z["dim"] ** -0.5, softcap=30.0, window=z["window"], keep_first=KEEP, **ex))
        cfg = M.engine_config(M.MurilornConfig(z["vocab"], z["width"], 1.0, 1e-5, STREAMS, None, 1.0, 30.0, (pair * L)[:L]), max_batch=max_batch, max_seq=max_seq,
                              max_step_rows=max_seq)
    elif kind == "vopozen":
        cfg = V.engine_config(V.VopozenConfig(z["vocab"], z["width"], 1e-5, 0.5, tuple(_vopozen_layers(z))), max_batch=max_batch, max_seq=max_seq, max_step_rows=max_seq)
    elif kind == "kidolorn":
        cfg = Q.engine_config(Q.KidolornConfig(z["vocab"], z["width"], 1e-5, 4, tuple(_kidolorn_layers(z))), max_batch=max_batch, max_seq=max_seq, max_step_rows=max_seq)
    elif kind == "bulidra":
        layers = tuple(BulidraLayer(z["heads"], z["kv_heads"], z["dim"], z["dim"], 4, z["dim"] ** -0.5, z["window"], 0.1, 1024, None, z["ff"]) for _ in range(L))
        cfg = engine_config(BulidraConfig(z["vocab"], z["width"], 1.0, 1e-5, SIDE_DIM, layers), max_batch=max_batch, max_seq=max_seq, max_step_rows=max_seq)
    else:
        cfg = EngineConfig.glimmer(n_layer=z["layers"], d_model=z["width"], n_head=z["heads"], n_kv_head=z["kv_heads"], head_dim=z["dim"], d_ff=z["ff"],
                                   vocab=z["vocab"], max_seq=max_seq, window=z["window"], max_batch=max_batch, global_every=0, tie_embeddings=1)
    eng = ResidentEngine(cfg)
    g = torch.Generator(device="cuda").manual_seed(0)
    for n, k in eng.expected_tensors().items():
        leaf = n.rsplit(".", 1)[-1]
        if leaf.startswith("hc"):
            t = torch.eye(STREAMS, device="cuda").flatten() if leaf.endswith("mix") else torch.full((k,), 1.0 / STREAMS if leaf.endswith("in") else 1.0, device="cuda")
        elif leaf in ("a_log", "dt_bias", "w0"):
            t = torch.full((k,), -1.0, device="cuda")
        elif "norm" in n:
            t = torch.full((k,), 0.0 if kind == "murilorn" and leaf != "out_norm" else 1.0, device="cuda")
        else:
            t = torch.randn(k, generator=g, device="cuda") * 0.02
        eng.set_tensor(n, t.bfloat16())
    eng.finalize()
    return eng


def _vopozen_layers(z: dict) -> list:
    """Chunks of 1.5 windows: the decode steps at a context of 4096 then see as many keys as with the window."""
    from ..models import vopozen as V
    L, rot = z["layers"], dict(rot_base=1e4, scale=z["dim"] ** -0.5)
    out: list = []
    for i in range(L):
        kind = VOPOZEN[i % 4]
        f = dict(ff=z["ff"]) if i % 2 == 0 else dict(experts=EXPERTS, top=TOP, expert_ff=z["ff"] // 4, shared_ff=z["ff"] // 2, groups=8, keep=4, route_scale=1.5)
        if kind == "attention":
            out.append(V.VopozenLayer("attention", z["heads"], z["kv_heads"], z["dim"], z["dim"], look=3 * z["window"] // 2, rot_dims=ROT, **rot, **f))
        elif kind == "wkv":
            out.append(V.VopozenLayer("wkv", z["heads"], z["heads"], z["dim"], z["dim"], rank_decay=DECAY, **f))
        else:
            out.append(V.VopozenLayer("latent_attention", z["heads"], 1, z["dim"], z["dim"], look=z["window"], rot_dims=ROT, rot_dim=ROT, kv_rank=LATENT, kv_from=i - 2 if kind == "reader" else -1,
                                      **rot, **f))
    return out


def _kidolorn_layers(z: dict) -> list:
    from ..models import kidolorn as Q
    out: list = []
    for i in range(z["layers"]):
        kind, H, d = KIDOLORN[i % 4], z["heads"], z["dim"]
        f = dict(ff=z["ff"], limit=7.0) if i % 2 == 0 else dict(experts=EXPERTS, top=TOP, expert_ff=z["ff"] // TOP, limit=7.0)
        if kind == "lightning":
            out.append(Q.KidolornLayer("lightning", H, d, d, decay=tuple(1 - 2.0 ** (-1 - 9 * h / H) for h in range(H)), **f))
        elif kind == "mingru":
            out.append(Q.KidolornLayer("mingru", vdim=H * d, **f))
        else:
            out.append(Q.KidolornLayer("latent_attention", H, d, d, scale=d ** -0.5, rot_dim=ROT, kv_rank=LATENT, kv_from=i - 2 if kind == "reader" else -1, **f))
    return out


def _time(eng, fn, n: int, warmup: int) -> float:
    for _ in range(warmup):
        fn()
    pairs = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(n)]
    with torch.cuda.stream(eng.stream):
        for a, b in pairs:
            a.record()
            fn()
            b.record()
    torch.cuda.synchronize()
    return statistics.median(a.elapsed_time(b) for a, b in pairs)


def _work(z: dict, kind: str, prompt: int, batch: int, context: int) -> tuple[float, float]:
    """(FLOPs of a prompt, bytes of a decode step): products and attention over visible keys; weights and visible cache rows."""
    w, q, kv = z["width"], z["heads"] * z["dim"], z["kv_heads"] * z["dim"]
    if kind == "murilorn":
        return _murilorn_work(z, prompt, batch, context)
    if kind == "vopozen":
        return _vopozen_work(z, prompt, batch, context)
    if kind == "kidolorn":
        return _kidolorn_work(z, prompt, batch, context)
    per = w * (q + 2 * kv + q + 2 * z["ff"]) + w * (q + z["ff"]) + (2 * w * SIDE_DIM if kind == "bulidra" else 0)
    win = min(z["window"], prompt)
    keys = win * (win + 1) / 2 + (prompt - win) * win
    flops = z["layers"] * (2.0 * per * prompt + 4.0 * q * keys)
    seen = min(z["window"], context)
    return flops, 2.0 * z["layers"] * (per + batch * seen * 2 * kv) + 2.0 * z["vocab"] * w


def _murilorn_work(z: dict, prompt: int, batch: int, context: int) -> tuple[float, float]:
    w, q, kv, L = z["width"], z["heads"] * z["dim"], z["kv_heads"] * z["dim"], z["layers"]
    n_delta = (L + 1) // 2
    n_att = L - n_delta
    delta = w * (3 * q + z["heads"] + 2 * RANK) + 2 * RANK * q + q * w
    att = w * (q + 2 * kv) + q * w
    expert = 3 * w * (z["ff"] // TOP)
    win = min(z["window"], prompt)
    keys = win * (win + 1) / 2 + (prompt - win) * win
    rule = 7.0 * q * z["dim"]                                   # decay, correction, write, read-out
    flops = n_delta * (2.0 * delta + rule) * prompt + n_att * (2.0 * att * prompt + 4.0 * q * keys) + L * 2.0 * (TOP * expert + EXPERTS * w) * prompt
    chosen = EXPERTS * (1 - (1 - TOP / EXPERTS) ** batch)       # experts a batch of uniform choices touches
    seen = min(z["window"] + KEEP, context)
    byts = 2.0 * (n_delta * delta + n_att * (att + batch * seen * 2 * kv) + L * (chosen * expert + EXPERTS * w)) + n_delta * batch * 8.0 * q * z["dim"] + 2.0 * z["vocab"] * w
    return flops, byts


def _vopozen_work(z: dict, prompt: int, batch: int, context: int) -> tuple[float, float]:
    w, q, kv = z["width"], z["heads"] * z["dim"], z["kv_heads"] * z["dim"]
    chosen = EXPERTS * (1 - (1 - TOP / EXPERTS) ** batch)       # experts a batch of uniform choices touches
    flops, byts = 0.0, 2.0 * z["vocab"] * w
    for y in _vopozen_layers(z):
        if y.type == "attention":
            per, n = w * (q + kv) + q * w, min(y.look, prompt)
            keys = prompt / n * n * (n + 1) / 2
            flops += 4.0 * q * keys
            byts += 2.0 * batch * min(context % y.look or y.look, context) * 2 * kv
        elif y.type == "wkv":
            per = w * (4 * q + DECAY) + DECAY * q + q * w
            flops += 5.0 * q * z["dim"] * prompt
            byts += batch * 8.0 * q * z["dim"]
        else:
            row = LATENT + ROT
            per, n = w * (z["heads"] * (z["dim"] + ROT) + (row if y.kv_from < 0 else 0)) + 2 * q * LATENT + q * w, min(y.look, prompt)
            keys = n * (n + 1) / 2 + (prompt - n) * n
            flops += 2.0 * z["heads"] * (2 * z["dim"] + ROT) * keys
            byts += 2.0 * batch * min(y.look, context) * row
        act, read = (3 * w * y.ff,) * 2 if y.ff else (w * (2 * TOP * y.expert_ff + 2 * y.shared_ff + EXPERTS), w * (2 * chosen * y.expert_ff + 2 * y.shared_ff + EXPERTS))
        flops += 2.0 * (per + act) * prompt
        byts += 2.0 * (per + read)
    return flops, byts


def _kidolorn_work(z: dict, prompt: int, batch: int, context: int) -> tuple[float, float]:
    w, q = z["width"], z["heads"] * z["dim"]
    chosen = EXPERTS * (1 - (1 - TOP / EXPERTS) ** batch)       # experts a batch of uniform choices touches
    flops, byts = 0.0, 2.0 * z["vocab"] * w
    for y in _kidolorn_layers(z):
        if y.type == "lightning":
            per = 5 * w * q
            flops += 5.0 * q * z["dim"] * prompt
            byts += batch * 8.0 * q * z["dim"]
        elif y.type == "mingru":
            per = 4 * w * q
            byts += batch * 8.0 * q
        else:
            row = LATENT + ROT
            per = w * (z["heads"] * (z["dim"] + ROT) + (row if y.kv_from < 0 else 0)) + 2 * q * LATENT + 2 * q * w
            flops += 2.0 * z["heads"] * (2 * z["dim"] + ROT) * prompt * (prompt + 1) / 2
            byts += 2.0 * batch * context * row
        act, read = (3 * w * y.ff,) * 2 if y.ff else (w * (3 * TOP * y.expert_ff + EXPERTS), w * (3 * chosen * y.expert_ff + EXPERTS))
        flops += 2.0 * (per + act) * prompt
        byts += 2.0 * (per + read)
    return flops, byts


def run(args, clock_sampler, sizes=None) -> None:
    hbm, tf = _peaks()
    for name in sizes or SIZES:
        z = SIZES[name]
        for kind in (BESIDE.get(args.serving, "glimmer"), args.serving):
            prompt, context = 8192, 4096
            eng = _engine(kind, z, 1, prompt + 64)
            g = torch.Generator().manual_seed(1)
            ids = torch.randint(0, z["vocab"], (prompt,), generator=g).tolist()
            with clock_sampler(0) as clocks:
                ms = _time(eng, lambda: eng.prefill(0, ids), max(args.steps // 2, 3), 3)
            flops, _ = _work(z, kind, prompt, 1, 0)
            print(json.dumps({"serving": kind, "size": name, "phase": "prefill", "prompt": prompt, "ms": round(ms, 3), "tokens_per_s": round(prompt / ms * 1e3),
                              "fraction_of_measured_bf16": round(flops / ms * 1e3 / tf, 3), "device_bytes": eng.device_bytes, "clocks": clocks.summary()}), flush=True)
            eng.close()
            del eng
            for batch in (1, 8, 32):
                eng = _engine(kind, z, batch, context + 128)
                last = {b: eng.prefill(b, ids[64 * b:64 * b + context]) for b in range(batch)}      # different tokens, different experts

                def step():
                    nonlocal last
                    last = eng.decode(last)

                with clock_sampler(0) as clocks:
                    ms = _time(eng, step, max(3 * args.steps, 30), 5)
                _, byts = _work(z, kind, 1, batch, context)
                print(json.dumps({"serving": kind, "size": name, "phase": "decode", "batch": batch, "context": context, "ms": round(ms, 4),
                                  "tokens_per_s": round(batch / ms * 1e3), "fraction_of_measured_hbm": round(byts / ms * 1e3 / hbm, 3),
                                  "clocks": clocks.summary()}), flush=True)
                eng.close()
                del eng
