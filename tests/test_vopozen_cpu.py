"""Vopozen without a GPU: configuration, tensor packing, how much every mistake would show in the reference's logits, the scheduler's room for
chunks, the architecture registry."""
import copy
import json

import pytest
import torch

import vopozen_oracle as oracle
from neuralfn_b200.models.layered_common import ModelConfigError
from neuralfn_b200.models.vopozen import VopozenConfig, engine_config, expected_shapes, pack_tensors
from neuralfn_b200.serving.architectures import architecture_of, is_model_directory
from vopozen_cases import attention, boost_needle, dense, lasting_memory, latent, model, moe, tokens_of, wkv


def rich():
    return model([attention(heads=6, kv_heads=3, dim=24, rot=10, chunk=13, mlp=dense(40)), latent(heads=3, dim=20, rot=6, vdim=24, rank=40, window=9, mlp=moe(ff=24)),
                  wkv(heads=3, dim=24, rank=5, mlp=None), latent(heads=2, dim=24, rot=6, vdim=40, rank=40, window=17, kv_from=1, mlp=moe(experts=5, groups=None, top=2, shared=0))],
                 vocab=70, width=72)


def test_configuration_round_trip_and_refusals():
    cfg, w = rich()
    c = VopozenConfig.from_dict(cfg, w)
    assert VopozenConfig.from_dict(c.to_dict()) == c == VopozenConfig.from_dict(cfg)
    bare = copy.deepcopy(cfg)
    for y in bare["layers"]:
        y["mixer"].pop("rank_decay", None)
        y["surplus"] = None                                      # settings without a value are none
    assert VopozenConfig.from_dict(bare, w) == c                 # the tensors give the inner size
    e = engine_config(c, max_batch=3, max_seq=100)
    assert [y.mixer for y in e.layers] == ["attention", "latent", "wkv", "latent"] and [y.kv_from for y in e.layers] == [-1, -1, -1, 1]
    assert e.window == 17 and e.post_norm == 1 and e.residual_mult == 0.7 and e.estimate_device_bytes() > 0
    assert [y.cache_row for y in e.layers] == [3 * 48, 46, 0, 0]
    assert engine_config(VopozenConfig.from_dict({**cfg, "layers": cfg["layers"][:1]}), max_seq=100).window == 13
    bad = [(0, "type", "conv"), (0, "mixer.kv_heads", 4), (0, "mixer.vdim", 32), (0, "mixer.rot.dims", 26), (0, "mixer.rot.dims", 5), (0, "mixer.mask.size", 0), (0, "mixer.surprise", 1),
           (0, "mlp.kind", "gated"), (0, "mixer.heads", 2.5), (1, "mixer.rot.dims", 4), (1, "mixer.kv_from", 0), (3, "mixer.kv_from", 2), (3, "mixer.kv_rank", 24), (3, "mixer.rot.base", 7.0),
           (1, "mlp.router.top", 9), (1, "mlp.router.top", 5), (1, "mlp.router.groups.count", 3), (1, "mlp.router.groups.keep", 5), (1, "mlp.expert.act", "relu"), (2, "mixer.kv_heads", 3)]
    for at, path, value in bad:
        broken = copy.deepcopy(cfg)
        node = broken["layers"][at]
        *head, last = path.split(".")
        for k in head:
            node = node[k]
        node[last] = value
        with pytest.raises(ModelConfigError):
            VopozenConfig.from_dict(broken)
    for key, value in (("streams", 2), ("width", 0), ("layers", [])):
        with pytest.raises(ModelConfigError):
            VopozenConfig.from_dict({**cfg, key: value})


def test_packed_tensors_compute_the_same_projections():
    cfg, w = rich()
    c = VopozenConfig.from_dict(cfg, w)
    assert set(expected_shapes(c)) == set(w)
    t = pack_tensors(c, w)
    D = lambda n: t[n].double()  # noqa: E731
    h = torch.randn(5, 72, dtype=torch.float64)
    hp = torch.zeros(5, 80, dtype=torch.float64)
    hp[:, :72] = h

    def same(got, ref, groups, pad):
        ref, got = ref.reshape(5, groups, -1), got.reshape(5, groups, pad)
        assert torch.allclose(got[..., :ref.shape[2]], ref) and not got[..., ref.shape[2]:].any()

    q, k = (hp @ D("layers.0.w_in").T).split([6 * 32, 3 * 32], 1)
    same(q, h @ w["l0.mix.q"].double().T, 6, 32)
    same(k, h @ w["l0.mix.k"].double().T, 3, 32)
    y = hp @ D("layers.1.w_in").T
    q, c1, kr = y.split([3 * 48, 48, 16], 1)
    ref = (h @ w["l1.mix.q"].double().T).view(5, 3, 26)
    same(q.reshape(5, 3, 48)[..., :32], ref[..., :20], 3, 32)
    same(q.reshape(5, 3, 48)[..., 32:], ref[..., 20:], 3, 16)
    z = h @ w["l1.mix.dkv"].double().T
    same(c1, z[:, :40], 1, 48)
    same(kr, z[:, 40:], 1, 16)
    assert t["layers.3.w_in"].shape[0] == 2 * 48 and "layers.3.c_norm" not in t
    lat = torch.randn(5, 40, dtype=torch.float64)
    lp = torch.zeros(5, 48, dtype=torch.float64)
    lp[:, :40] = lat
    uk, uv = (lp @ D("layers.1.w_ukv").T).split([3 * 32, 3 * 32], 1)
    same(uk, lat @ w["l1.mix.uk"].double().T, 3, 32)
    same(uv, lat @ w["l1.mix.uv"].double().T, 3, 32)
    # queries through the transposed key projection score the latent as the keys would
    qa = torch.einsum("thd,hrd->thr", q.reshape(5, 3, 48)[..., :32], D("layers.1.w_uk_t").view(3, 48, 32))
    assert torch.allclose((qa * lp[:, None]).sum(-1), (q.reshape(5, 3, 48)[..., :32] * uk.view(5, 3, 32)).sum(-1))
    for i, s in enumerate("rkvg"):
        same((hp @ D("layers.2.w_in").T).split(3 * 32, 1)[i], h @ w[f"l2.mix.{s}"].double().T, 3, 32)
    low = torch.randn(5, 5, dtype=torch.float64)
    both = torch.cat([torch.nn.functional.pad(0.75 * low, (0, 11)), torch.nn.functional.pad(0.25 * low, (0, 11))], 1)
    same(both @ D("layers.2.w2").T, low @ w["l2.mix.w2"].double().T, 3, 32)
    assert t["layers.2.mu"].shape == (5, 80) and torch.equal(t["layers.2.mu"][4, :72], w["l2.mix.mu.w"])
    for e in range(8):
        same(hp @ D("layers.1.w_gate_up")[e].T, h @ w[f"l1.mlp.e{e}.up"].double().T, 1, 32)
        assert torch.equal(t["layers.1.w_down"][e, :72, :24], w[f"l1.mlp.e{e}.down"])
    assert "layers.1.w_shared_up" in t and "layers.3.w_shared_up" not in t
    assert pack_tensors(c, {**w, "l2.norm2": w["l1.norm2"]}).keys() == t.keys()                       # of a feed-forward that is not there
    broken = dict(w)
    broken.pop("l1.mix.dkv.norm")
    with pytest.raises(ModelConfigError, match="l1.mix.dkv.norm"):
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


def _half_turn(f):
    def g(x, first, dims, base):
        """halves paired instead of neighbours"""
        order = [j for i in range(dims // 2) for j in (i, i + dims // 2)]
        y = f(x[..., order + list(range(dims, x.shape[-1]))], first, dims, base)
        out = y.clone()
        out[..., order] = y[..., :dims]
        return out
    return g


def _values_after_norm(f):
    def g(h, W, p, m, eps):
        T, H, d = h.shape[0], m["heads"], m["dim"]
        q, v = (h @ W[p + "q"].T).view(T, H, d), (h @ W[p + "k"].T).view(T, m["kv_heads"], d)
        q, k = oracle.norm(q, W[p + "q.norm"], eps), oracle.norm(v, W[p + "k.norm"], eps)
        v = k
        q, k = (oracle.rotate(t, 0, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
        mask = oracle.seen(T, oracle.in_chunk, oracle.size_of(m))
        n = H // m["kv_heads"]
        out = torch.stack([oracle.attend(q[:, x] @ k[:, x // n].T * m["scale"], mask, v[:, x // n]) for x in range(H)], 1)
        return out.reshape(T, -1) @ W[p + "o"].T
    return g


def _rule(bonus=True, late=False):
    def make(f):
        def g(r, k, v, w, u):
            S, out = torch.zeros(r.shape[1], r.shape[2], r.shape[2], dtype=r.dtype), torch.zeros_like(r)
            for t in range(r.shape[0]):
                kv = k[t][:, :, None] * v[t][:, None, :]
                if late:
                    S = w[t][:, :, None] * S
                out[t] = ((S + (u[:, :, None] * kv if bonus else 0)) * r[t][:, :, None]).sum(1)
                S = (S if late else w[t][:, :, None] * S) + kv
            return out
        return g
    return make


MISTAKES = {
    "chunk one larger": lambda c, w, m: c["layers"][0]["mixer"]["mask"].update(size=14),
    "chunk as a window": _patched("in_chunk", lambda f: oracle.in_window),
    "window one wider": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(size=10),
    "window one narrower": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(size=8),
    "reader with the owner's window": lambda c, w, m: c["layers"][3]["mixer"]["mask"].update(size=9),
    "query norm": lambda c, w, m: w["l0.mix.q.norm"].fill_(1.0),
    "key norm": lambda c, w, m: w["l0.mix.k.norm"].fill_(1.0),
    "latent norm": lambda c, w, m: w["l1.mix.dkv.norm"].fill_(1.0),
    "normed values": _patched("attention_mixer", _values_after_norm),
    "rotation base": lambda c, w, m: c["layers"][0]["mixer"]["rot"].update(base=900.0),
    "rotation size": lambda c, w, m: c["layers"][0]["mixer"]["rot"].update(dims=8),
    "latent rotation base": lambda c, w, m: [c["layers"][i]["mixer"]["rot"].update(base=400.0) for i in (1, 3)],
    "rotation of halves": _patched("rotate", _half_turn),
    "positions from one": _patched("rotate", lambda f: lambda x, first, dims, base: f(x, 1, dims, base) if x.shape[1] > 3 else f(x, 0, dims, base)),
    "score scale": lambda c, w, m: c["layers"][0]["mixer"].update(scale=0.28),
    "latent score scale": lambda c, w, m: c["layers"][3]["mixer"].update(scale=0.38),
    "no shift": lambda c, w, m: w["l2.mix.mu.k"].zero_(),
    "no bonus": _patched("wkv_rule", _rule(bonus=False)),
    "read after decay": _patched("wkv_rule", _rule(late=True)),
    "decay bias": lambda c, w, m: w["l2.mix.w0"].zero_(),
    "decay input": lambda c, w, m: w["l2.mix.w1"].zero_(),
    "gate": lambda c, w, m: w["l2.mix.g"].zero_(),
    "output weights": lambda c, w, m: w["l2.mix.norm"].fill_(1.0),
    "no correction": lambda c, w, m: w["l1.mlp.correction"].zero_(),
    "no groups": lambda c, w, m: c["layers"][1]["mlp"]["router"].pop("groups"),
    "one group more": lambda c, w, m: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3),
    "excluded scores as zero": _patched("closed", lambda f: lambda choice, ok: choice.masked_fill(~ok, 0.0)),
    "fewer experts": lambda c, w, m: c["layers"][3]["mlp"]["router"].update(top=1),
    "router scale": lambda c, w, m: c["layers"][1]["mlp"]["router"].update(scale=1.6),
    "no shared expert": lambda c, w, m: c["layers"][1]["mlp"].pop("shared"),
    "expert activation": _patched("relu_squared", lambda f: lambda z: torch.clamp(z, min=0)),
    "feed-forward activation": _patched("silu", lambda f: lambda z: torch.clamp(z, min=0)),
    "residual factor": lambda c, w, m: c.update(residual_mult=0.68),
    "norm epsilon": lambda c, w, m: c["norm"].update(eps=0.05),
    "output norm": lambda c, w, m: w["l3.norm2"].fill_(1.0),
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
    for layer, near, far in ((attention(heads=4, kv_heads=2, dim=32, rot=16, chunk=50, scale=0.45), 100, 99), (latent(heads=5, dim=32, rot=16, vdim=32, rank=64, window=50), 70, 69)):
        cfg, w = model([layer], vocab=64)
        boost_needle(cfg, w, query=62, key=63)
        rows = {}
        for place in (None, near, far):
            ids = tokens_of(cfg, 120, seed=1, below=62)
            ids[-1] = 62
            if place is not None:
                ids[place] = 63
            rows[place] = oracle.forward(cfg, w, ids)[0][-1:]
        assert _spread(rows[None], rows[near]) > 0.3 and _spread(rows[None], rows[far]) < 1e-9      # seen, and just out of sight
    cfg, w = model([wkv(heads=3, dim=32)], vocab=40)
    lasting_memory(cfg, w, write=38, read=39)
    ids = tokens_of(cfg, 150, seed=3, below=38)
    ids[-1] = 39
    a = oracle.forward(cfg, w, ids)[0][-1:]
    ids[4] = 38
    assert _spread(a, oracle.forward(cfg, w, ids)[0][-1:]) > 0.3


def test_sharp_routing_is_never_close_and_uses_many_experts(monkeypatch):
    cfg, w = model([wkv(mlp=moe(experts=12, groups=(4, 2), top=3)), attention(chunk=20, mlp=moe(groups=None))], width=96)
    gaps, chosen = [], set()
    orig = oracle.route
    monkeypatch.setattr(oracle, "route", lambda *a: (lambda r: (chosen.update(r[0].tolist()), r)[1])(orig(*a)))
    oracle.forward(cfg, w, tokens_of(cfg, 150, seed=7), gaps=gaps)
    assert len(gaps) == 300 and min(gaps) > 0.01 and len(chosen) >= 6


def test_scheduler_counts_chunk_pages():
    from neuralfn_b200.serving.engine import Sampling
    from neuralfn_b200.serving.scheduler import StepRequest, StepScheduler
    cfg, _ = model([attention(chunk=100), latent(window=70), wkv()])
    limits = engine_config(VopozenConfig.from_dict(cfg), max_batch=2, max_seq=4096, kv_tokens=4096, max_step_rows=64)
    eng = type("E", (), dict(config=limits, has_steps=True, free_tokens=4096))()
    need = StepScheduler(eng)._pages_for(StepRequest(0, [1] * 2000, 500, Sampling(), None))
    assert need == (100 + 64 + 64 + 63) // 64                    # chunk, one pass, the page at hand


def test_registry_knows_the_design(tmp_path):
    cfg, _ = rich()
    a = architecture_of(cfg)
    assert a.family == "vopozen" and a.component == "layered" and a.dtypes == ("bfloat16", "float32") and a.steps
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert is_model_directory(tmp_path)
