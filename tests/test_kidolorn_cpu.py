"""Kidolorn without a GPU: configuration, tensor packing, how much every mistake would show in the reference's logits, the scheduler's room for pages
that stay, the architecture registry."""
import copy
import json

import pytest
import torch

import kidolorn_oracle as oracle
from kidolorn_cases import boost_needle, dense, lasting_memory, latent, lightning, mingru, model, moe, tokens_of
from neuralfn_b200.models.kidolorn import KidolornConfig, engine_config, expected_shapes, pack_tensors
from neuralfn_b200.models.layered_common import ModelConfigError
from neuralfn_b200.serving.architectures import architecture_of, is_model_directory


def rich():
    return model([latent(heads=3, dim=20, rot=6, vdim=24, rank=40, mlp=moe(ff=24)), lightning(heads=3, dim=24, vdim=40, mlp=dense(40)), mingru(width=56),
                  latent(heads=2, dim=24, rot=6, vdim=40, rank=40, kv_from=0, scale=0.3, mlp=moe(experts=5, top=2, limit=0.5)), mingru(width=40, mlp=dense(24, limit=0.7))], vocab=70, width=72, taps=4)


def test_configuration_round_trip_and_refusals():
    cfg, w = rich()
    c = KidolornConfig.from_dict(cfg)
    assert KidolornConfig.from_dict(c.to_dict()) == c
    loose = copy.deepcopy(cfg)
    loose["layers"][0]["surplus"] = loose["layers"][0]["mixer"]["kv_from"] = None                    # settings without a value are none
    assert KidolornConfig.from_dict(loose) == c
    e = engine_config(c, max_batch=3, max_seq=100)
    assert [y.mixer for y in e.layers] == ["latent", "linear", "gru", "latent", "gru"] and [y.kv_from for y in e.layers] == [-1, -1, -1, 0, -1]
    assert e.window == 0 and e.sandwich == 1 and e.scalar_norms == 1 and e.input_taps == 4 and e.estimate_device_bytes() > 0
    assert [y.cache_row for y in e.layers] == [46, 0, 0, 0, 0] and [y.ff_limit for y in e.layers] == [0.9, 1.1, 0.0, 0.5, 0.7]
    bad = [(0, "type", "conv"), (0, "mixer.heads", 2.5), (0, "mixer.rot.dims", 4), (0, "mixer.rot.base", 0.0), (0, "mixer.rot_dim", 5), (0, "mixer.kv_from", 0), (0, "mixer.mask", {"size": 4}),
           (0, "mlp.kind", "gated"), (0, "mlp.router.top", 9), (0, "mlp.router.scale", 2.0), (0, "mlp.expert.limit", 0.0), (0, "mlp.shared", {"ff": 4}), (1, "mixer.decay", [0.5, 0.5]), (1, "mixer.kv_heads", 3),
           (1, "mlp.limit", -1.0), (2, "mixer.width", 0), (2, "mixer.heads", 2), (3, "mixer.kv_from", 1), (3, "mixer.kv_from", 3), (3, "mixer.kv_rank", 24), (3, "mixer.rot.base", 7.0)]
    for at, path, value in bad:
        broken = copy.deepcopy(cfg)
        node = broken["layers"][at]
        *head, last = path.split(".")
        for k in head:
            node = node[k]
        node[last] = value
        with pytest.raises(ModelConfigError):
            KidolornConfig.from_dict(broken)
    for key, value in (("streams", 2), ("width", 0), ("layers", []), ("canon", {"taps": 0}), ("canon", {"taps": 3, "bias": True})):
        with pytest.raises(ModelConfigError):
            KidolornConfig.from_dict({**cfg, key: value})
    with pytest.raises(ValueError, match="decays"):
        from dataclasses import replace
        replace(e, layers=(replace(e.layers[1], decay=(0.5,)),)).create(None, 0)


def test_packed_tensors_compute_the_same_projections():
    cfg, w = rich()
    c = KidolornConfig.from_dict(cfg)
    assert set(expected_shapes(c)) == set(w)
    t = pack_tensors(c, w)
    D = lambda n: t[n].double()  # noqa: E731
    h = torch.randn(5, 72, dtype=torch.float64)
    hp = torch.zeros(5, 80, dtype=torch.float64)
    hp[:, :72] = h

    def same(got, ref, groups, pad):
        ref, got = ref.reshape(5, groups, -1), got.reshape(5, groups, pad)
        assert torch.allclose(got[..., :ref.shape[2]], ref) and not got[..., ref.shape[2]:].any()

    pairs = [0, 3, 1, 4, 2, 5]                                     # i and i + 3 turn together
    q, c1, kr, g = (hp @ D("layers.0.w_in").T).split([3 * 48, 48, 16, 3 * 32], 1)
    ref = (h @ w["l0.mix.q"].double().T).view(5, 3, 26)
    same(q.reshape(5, 3, 48)[..., :32], ref[..., :20], 3, 32)
    same(q.reshape(5, 3, 48)[..., 32:], ref[..., 20:][..., pairs], 3, 16)
    z = h @ w["l0.mix.dkv"].double().T
    same(c1, z[:, :40], 1, 48)
    same(kr, z[:, 40:][:, pairs], 1, 16)
    same(g, h @ w["l0.mix.g"].double().T, 3, 32)
    assert t["layers.3.w_in"].shape[0] == 2 * 48 + 2 * 48 and "layers.3.c_norm" not in t
    lat = torch.randn(5, 40, dtype=torch.float64)
    lp = torch.zeros(5, 48, dtype=torch.float64)
    lp[:, :40] = lat
    uk, uv = (lp @ D("layers.0.w_ukv").T).split([3 * 32, 3 * 32], 1)
    same(uk, lat @ w["l0.mix.uk"].double().T, 3, 32)
    same(uv, lat @ w["l0.mix.uv"].double().T, 3, 32)
    # queries through the transposed key projection score the latent as the keys would
    qa = torch.einsum("thd,hrd->thr", q.reshape(5, 3, 48)[..., :32], D("layers.0.w_uk_t").view(3, 48, 32))
    assert torch.allclose((qa * lp[:, None]).sum(-1), (q.reshape(5, 3, 48)[..., :32] * uk.view(5, 3, 32)).sum(-1))
    parts = (hp @ D("layers.1.w_in").T).split([3 * 32, 3 * 32, 3 * 48, 3 * 48], 1)
    for s, part, pad in zip("qkvg", parts, (32, 32, 48, 48)):
        same(part, h @ w[f"l1.mix.{s}"].double().T, 3, pad)
    assert torch.equal(t["layers.1.out_norm"].view(3, 48)[:, :40].flatten(), w["l1.mix.norm"])
    parts = (hp @ D("layers.2.w_in").T + D("layers.2.bias_in")).split(64, 1)
    for s, part in zip("zxg", parts):
        assert torch.allclose(part[:, :56], h @ w[f"l2.mix.{s}"].double().T + (w[f"l2.mix.{s}.b"].double() if s != "g" else 0)) and not part[:, 56:].any()
    assert torch.equal(t["layers.4.in_conv2"][:, :72], w["l4.canon2"].T) and not t["layers.4.in_conv2"][:, 72:].any()
    assert t["layers.4.norm2_b"].shape == (1,) and "layers.2.norm2" not in t
    up = (hp @ D("layers.4.w_gate_up").T + D("layers.4.bias_gate_up")).split(32, 1)
    for s, part in zip(("gate", "up"), up):
        same(part, h @ w[f"l4.mlp.{s}"].double().T + w[f"l4.mlp.{s}.b"].double(), 1, 32)
    for e in range(8):
        gate, part = (hp @ D("layers.0.w_gate_up")[e].T).split(32, 1)
        same(gate, h @ w[f"l0.mlp.e{e}.gate"].double().T, 1, 32)
        same(part, h @ w[f"l0.mlp.e{e}.up"].double().T, 1, 32)
        assert torch.equal(t["layers.0.w_down"][e, :72, :24], w[f"l0.mlp.e{e}.down"])
    assert pack_tensors(c, {**w, "l2.norm2": w["l0.norm2"], "l2.canon2": w["l0.canon2"]}).keys() == t.keys()      # of a feed-forward that is not there
    broken = dict(w)
    broken.pop("l0.mix.sink")
    with pytest.raises(ModelConfigError, match="l0.mix.sink"):
        pack_tensors(c, broken)


def _spread(a, b):
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (a - a.mean(-1, keepdim=True)).pow(2).mean().sqrt())


def _patched(name, fn):
    """A mistake in one of the reference's functions."""
    def plant(c, w, monkeypatch):
        monkeypatch.setattr(oracle, name, fn(getattr(oracle, name)))
    return plant


def _neighbours(f):
    def g(x, dims, base):
        """neighbours paired instead of halves"""
        order = [j for i in range(dims // 2) for j in (i, i + dims // 2)]
        inverse = torch.tensor(order).argsort().tolist()
        y = f(x[..., inverse], dims, base)
        return y[..., order]
    return g


def _read_first(f):
    def g(q, k, v, decay):
        S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), torch.zeros_like(v)
        for t in range(q.shape[0]):
            out[t] = (S * q[t][:, :, None]).sum(1)
            S = torch.tensor(decay, dtype=q.dtype)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        return out
    return g


def _per_head_norm(f):
    def g(h, W, p, m, eps):
        T, H = h.shape[0], m["heads"]
        q, k, v = (oracle.silu(h @ W[p + n].T).view(T, H, -1) for n in "qkv")
        o = oracle.rms(oracle.linear_rule(q, k, v, m["decay"]), eps).reshape(T, -1)
        return (o * W[p + "norm"] * oracle.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T
    return g


def _sigmoid_weights(f):
    def g(z, top):
        """(a common factor of a token's weights would not show: the norm behind the sublayer takes it out again)"""
        e, _ = f(z, top)
        return e, oracle.sigmoid(z[e])
    return g


MISTAKES = {
    "no convolution on a mixer's input": lambda c, w, m: w["l1.canon1"].zero_(),
    "no convolution on a feed-forward's input": lambda c, w, m: w["l0.canon2"].zero_(),
    "taps turned round": lambda c, w, m: w.update({"l2.canon1": w["l2.canon1"].flip(1)}),
    "convolution instead of its sum with the row": _patched("sublayer_input", lambda f: lambda x, W, p, which, eps: oracle.short_conv(oracle.rms(x, eps) * W[f"{p}norm{which}"], W[f"{p}canon{which}"])),
    "norm in front": lambda c, w, m: w["l2.norm1"].fill_(1.2),
    "norm behind": lambda c, w, m: w["l1.norm1b"].fill_(1.0),
    "norm behind a feed-forward": lambda c, w, m: w["l4.norm2b"].fill_(0.9),
    "norm epsilon": lambda c, w, m: c["norm"].update(eps=0.05),
    "decays": lambda c, w, m: c["layers"][1]["mixer"].update(decay=[0.7, 0.97, 0.995]),
    "read before writing": _patched("linear_rule", _read_first),
    "a norm per head": _patched("lightning_mixer", _per_head_norm),
    "weights of the lightning norm": lambda c, w, m: w["l1.mix.norm"].fill_(1.0),
    "lightning gate": lambda c, w, m: w["l1.mix.g"].zero_(),
    "share without bias": lambda c, w, m: w["l2.mix.z.b"].zero_(),
    "candidate without bias": lambda c, w, m: w["l4.mix.x.b"].zero_(),
    "candidate is linear": _patched("candidate", lambda f: lambda u: u + 0.5),
    "candidate is a sigmoid": _patched("candidate", lambda f: oracle.sigmoid),
    "gate of the gated recurrence": lambda c, w, m: w["l2.mix.g"].zero_(),
    "share and rest swapped": _patched("gated_rule", lambda f: lambda z, cand: f(1 - z, cand)),
    "sinks left out": lambda c, w, m: w["l0.mix.sink"].fill_(-60.0),
    "sinks of zero": lambda c, w, m: w["l3.mix.sink"].zero_(),
    "scaled sinks": lambda c, w, m: w.update({"l0.mix.sink": w["l0.mix.sink"] * 0.4}),
    "latent norm": lambda c, w, m: w["l0.mix.dkv.norm"].fill_(1.0),
    "output gate": lambda c, w, m: w["l3.mix.g"].zero_(),
    "rotation base": lambda c, w, m: [c["layers"][i]["mixer"]["rot"].update(base=400.0) for i in (0, 3)],
    "rotation of neighbours": _patched("rotate_half", _neighbours),
    "score scale": lambda c, w, m: c["layers"][3]["mixer"].update(scale=0.28),
    "gate's limit": lambda c, w, m: c["layers"][1]["mlp"].update(limit=1.3),
    "an expert's limit": lambda c, w, m: c["layers"][3]["mlp"]["expert"].update(limit=0.6),
    "no one added to up": _patched("clamped_gate", lambda f: lambda g, u, limit: f(g, u, limit) - f(g, torch.zeros_like(u), limit)),
    "no lower limit of up": _patched("clamped_gate", lambda f: lambda g, u, limit: (lambda a: a * oracle.sigmoid(1.702 * a) * (torch.clamp(u, max=limit) + 1))(torch.clamp(g, max=limit))),
    "a lower limit of the gate": _patched("clamped_gate", lambda f: lambda g, u, limit: f(torch.clamp(g, min=-limit), u, limit)),
    "plain SiLU": _patched("clamped_gate", lambda f: lambda g, u, limit: oracle.silu(torch.clamp(g, max=limit)) * (torch.clamp(u, -limit, limit) + 1)),
    "feed-forward without bias": lambda c, w, m: w["l1.mlp.up.b"].zero_(),
    "output without bias": lambda c, w, m: w["l4.mlp.down.b"].zero_(),
    "sigmoids as weights": _patched("route", _sigmoid_weights),
    "fewer experts": lambda c, w, m: c["layers"][3]["mlp"]["router"].update(top=1),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_a_planted_mistake_shows(name, monkeypatch):
    """Every mistake moves some logit row by far more than the tolerance the GPU tests use in 32-bit (3e-5)."""
    cfg, w = rich()
    ids = tokens_of(cfg, 60, seed=2)
    good, _ = oracle.forward(cfg, w, ids)
    cfg2, w2 = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    MISTAKES[name](cfg2, w2, monkeypatch)
    assert _spread(good, oracle.forward(cfg2, w2, ids)[0]) > 1e-3


def test_needles_and_memories_show_in_bf16_terms():
    cfg, w = model([latent(heads=5, dim=32, rot=16, vdim=32, rank=64)], vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    ids = tokens_of(cfg, 300, seed=1, below=62)
    ids[-1] = 62
    a = oracle.forward(cfg, w, ids)[0][-1:]
    ids[4] = 63
    assert _spread(a, oracle.forward(cfg, w, ids)[0][-1:]) > 0.3
    for layer in (lightning(heads=3, dim=32, vdim=32, decay=[1.0, 0.999, 1.0]), mingru(width=48)):
        cfg, w = model([layer], vocab=40)
        lasting_memory(cfg, w, write=38, read=39)
        ids = tokens_of(cfg, 150, seed=3, below=38)
        ids[-1] = 39
        a = oracle.forward(cfg, w, ids)[0][-1:]
        ids[4] = 38
        assert _spread(a, oracle.forward(cfg, w, ids)[0][-1:]) > 0.3


def test_sharp_routing_is_never_close_and_uses_many_experts(monkeypatch):
    cfg, w = model([mingru(mlp=moe(experts=12, top=3)), lightning(mlp=moe())], width=96)
    gaps, chosen = [], set()
    orig = oracle.route
    monkeypatch.setattr(oracle, "route", lambda *a: (lambda r: (chosen.update(r[0].tolist()), r)[1])(orig(*a)))
    oracle.forward(cfg, w, tokens_of(cfg, 150, seed=7), gaps=gaps)
    assert len(gaps) == 300 and min(gaps) > 0.05 and len(chosen) >= 6


def test_scheduler_counts_every_page_of_a_sequence():
    from neuralfn_b200.serving.engine import Sampling
    from neuralfn_b200.serving.scheduler import StepRequest, StepScheduler
    cfg, _ = model([latent(), lightning(), mingru()])
    limits = engine_config(KidolornConfig.from_dict(cfg), max_batch=2, max_seq=4096, kv_tokens=4096, max_step_rows=64)
    eng = type("E", (), dict(config=limits, has_steps=True, free_tokens=4096))()
    assert StepScheduler(eng)._pages_for(StepRequest(0, [1] * 2000, 500, Sampling(), None)) == (2500 + 63) // 64


def test_registry_knows_the_design(tmp_path):
    cfg, _ = rich()
    a = architecture_of(cfg)
    assert a.family == "kidolorn" and a.component == "layered" and a.dtypes == ("bfloat16", "float32") and a.steps
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert is_model_directory(tmp_path)
