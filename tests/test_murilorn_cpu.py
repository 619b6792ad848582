"""Murilorn without a GPU: configuration, tensor packing, how much every mistake would show in the reference's logits, the scheduler's room
for kept first tokens, the architecture registry."""
import copy
import json

import pytest
import torch

import murilorn_oracle as oracle
from murilorn_cases import attention, boost_needle, delta, lasting_memory, model, sharp_routing, tokens_of
from neuralfn_b200.models.layered_common import ModelConfigError
from neuralfn_b200.models.murilorn import MurilornConfig, engine_config, expected_shapes, layer_order, pack_tensors
from neuralfn_b200.serving.architectures import architecture_of, is_model_directory


def rich():
    return model([delta(heads=6, kv_heads=3, dim=24, vdim=40, ff=40, experts=5, top=2), attention(heads=6, kv_heads=2, dim=24, vdim=40, window=9, keep=2),
                  delta(heads=3, kv_heads=3, dim=40, vdim=24, conv=2, experts=0), attention(experts=3, top=1)],
                 vocab=70, width=72, streams=3, loop=(1, 3, 2))


def test_configuration_round_trip_and_refusals():
    cfg, w = rich()
    c = MurilornConfig.from_dict(cfg, w)
    assert MurilornConfig.from_dict(c.to_dict()) == c == MurilornConfig.from_dict(cfg)
    bare = copy.deepcopy(cfg)
    for y in bare["layers"]:
        y["mixer"].pop("rank_decay", None), y["mixer"].pop("rank_gate", None)
        y["surplus"] = None                                      # settings without a value are none
    assert MurilornConfig.from_dict(bare, w) == c                # the tensors give the inner sizes
    assert layer_order(c) == oracle.layer_order(cfg) == [0, 1, 2, 1, 2, 3]
    e = engine_config(c, max_batch=3, max_seq=100)
    assert [y.weights_of for y in e.layers] == [-1, -1, -1, 1, 2, -1] and [y.mixer for y in e.layers] == ["delta", "attention"] * 3
    assert e.window == 0 and e.streams == 3 and e.untied_head == 1 and e.norm_offset == 1.0 and e.estimate_device_bytes() > 0
    no_wide = engine_config(MurilornConfig.from_dict({**cfg, "layers": cfg["layers"][:3]}), max_seq=100)
    assert no_wide.window == 9 + 64                              # the page of the kept tokens stays too
    bad = [("type", "recurrent"), ("mixer.kv_heads", 4), ("mixer.conv", 0), ("mixer.surprise", 1), ("mlp.kind", "dense"), ("mlp.router.top", 6), ("mlp.router.top", 0),
           ("mlp.expert.act", "relu"), ("mixer.heads", 2.5)]
    for path, value in bad:
        broken = copy.deepcopy(cfg)
        node = broken["layers"][0]
        *head, last = path.split(".")
        for k in head:
            node = node[k]
        node[last] = value
        with pytest.raises(ModelConfigError):
            MurilornConfig.from_dict(broken)
    for key, value in (("loop", {"start": 2, "stop": 9, "times": 1}), ("loop", {"start": 0, "stop": 1, "times": 0}), ("rotation", 1), ("streams", -1)):
        with pytest.raises(ModelConfigError):
            MurilornConfig.from_dict({**cfg, key: value})


def test_packed_tensors_compute_the_same_projections():
    cfg, w = rich()
    c = MurilornConfig.from_dict(cfg, w)
    assert set(expected_shapes(c)) == set(w)
    t = pack_tensors(c, w)
    h = torch.randn(5, 72, dtype=torch.float64)
    hp = torch.zeros(5, 80, dtype=torch.float64)
    hp[:, :72] = h

    def same(got, name, groups, pad, bias=None):
        ref = (h @ w[name].double().T + (0 if bias is None else w[bias].double())).view(5, groups, -1)
        got = got.reshape(5, groups, pad)
        assert torch.allclose(got[..., :ref.shape[2]], ref) and not got[..., ref.shape[2]:].any()

    y = hp @ t["layers.0.w_in"].double().T
    q, k, v, b, a1, g1 = y.split([3 * 32, 3 * 32, 6 * 48, 16, 16, 32], 1)
    for got, n, groups, pad in ((q, "q", 3, 32), (k, "k", 3, 32), (v, "v", 6, 48), (b, "b", 1, 16), (a1, "a1", 1, 16), (g1, "g1", 1, 32)):
        same(got, f"l0.mix.{n}", groups, pad)
    assert torch.allclose((a1 @ t["layers.0.w_a2"].double().T).view(5, 6, 32)[..., :24].reshape(5, -1), (h @ w["l0.mix.a1"].double().T) @ w["l0.mix.a2"].double().T)
    assert torch.allclose((g1 @ t["layers.0.w_g2"].double().T).view(5, 6, 48)[..., :40].reshape(5, -1), (h @ w["l0.mix.g1"].double().T) @ w["l0.mix.g2"].double().T)
    assert torch.equal(t["layers.0.conv"][:, 32:56].T, w["l0.mix.q.conv"][24:48])
    y = hp @ t["layers.1.w_in"].double().T + t["layers.1.bias_in"].double()
    for got, n, groups, pad in zip(y.split([6 * 32, 2 * 32, 2 * 48], 1), "qkv", (6, 2, 2), (32, 32, 48)):
        same(got, f"l1.mix.{n}", groups, pad, f"l1.mix.{n}.b")
    for e in range(5):
        up2 = hp @ t["layers.0.w_gate_up"][e].double().T
        same(up2[:, :48], f"l0.mlp.e{e}.gate", 1, 48)
        same(up2[:, 48:], f"l0.mlp.e{e}.up", 1, 48)
        assert torch.equal(t["layers.0.w_down"][e, :72, :40], w[f"l0.mlp.e{e}.down"])
    assert not any(n.startswith(("layers.3", "layers.4")) for n in t) and "layers.5.w_in" in t      # the loop's later passes own no tensors
    assert "layers.2.hc1_mix" in t and "layers.2.hc2_mix" not in t
    assert pack_tensors(c, {**w, "l2.norm2": w["l1.norm2"]}).keys() == t.keys()                       # of a feed-forward that is not there
    broken = dict(w)
    broken.pop("l1.mix.q.b")
    with pytest.raises(ModelConfigError, match="l1.mix.q.b"):
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


def _early_read(rule):
    def f(q, k, v, g, beta):
        S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), torch.zeros_like(v)
        for t in range(q.shape[0]):
            S = g[t][:, :, None] * S
            out[t] = (S * q[t][:, :, None]).sum(1)
            S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1)))[:, None]
        return out
    return f


MISTAKES = {
    "window one wider": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(size=10),
    "window one narrower": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(size=8),
    "one kept token too many": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(keep_first=3),
    "one kept token too few": lambda c, w, m: c["layers"][1]["mixer"]["mask"].update(keep_first=1),
    "no soft cap": lambda c, w, m: c["layers"][3]["mixer"].pop("softcap"),
    "score scale": lambda c, w, m: c["layers"][3]["mixer"].update(scale=0.38),
    "key bias": lambda c, w, m: w["l1.mix.k.b"].zero_(),
    "value bias": lambda c, w, m: w["l1.mix.v.b"].zero_(),
    "no sink": _patched("softmax_with_sink", lambda f: lambda s: torch.softmax(s, -1)),
    "loop once less": lambda c, w, m: c["loop"].update(times=1),
    "norm epsilon": lambda c, w, m: c["norm"].update(eps=0.1),
    "embedding scale": lambda c, w, m: c["embedding"].update(scale=1.9),
    "logit scale": lambda c, w, m: c.update(logit_scale=1.4),
    "no logit cap": lambda c, w, m: c.pop("logit_softcap"),
    "fewer experts": lambda c, w, m: c["layers"][0]["mlp"]["router"].update(top=1),
    "history dropped": lambda c, w, m: w["l0.mix.k.conv"][:, 0].zero_(),
    "value convolution": lambda c, w, m: w["l0.mix.v.conv"][:, 1].zero_(),
    "decay rate": lambda c, w, m: w["l0.mix.A_log"].add_(0.2),
    "decay bias": lambda c, w, m: w["l0.mix.dt_bias"].zero_(),
    "step size": lambda c, w, m: w["l0.mix.b"].zero_(),
    "output gate": lambda c, w, m: w["l0.mix.g2"].zero_(),
    "output norm": lambda c, w, m: w["l0.mix.norm"].fill_(1.0),
    "stream mix transposed": lambda c, w, m: w.update({n: t.T.contiguous() for n, t in w.items() if n.endswith("hc1.mix")}),
    "stream output": lambda c, w, m: w["l1.hc2.out"].fill_(1.0),
    "stream input": lambda c, w, m: w["l1.hc1.in"].fill_(0.3),
    "norm around one": _patched("centred_norm", lambda f: lambda x, w, eps: f(x, w - 1, eps)),
    "read before write": _patched("delta_rule", _early_read),
    "weight on the output": _patched("silu", lambda f: lambda z: z),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_a_planted_mistake_shows(name, monkeypatch):
    """Every mistake moves some logit row by far more than the tolerance the GPU tests use in 32-bit (3e-5)."""
    cfg, w = rich()
    ids = tokens_of(cfg, 40, seed=2)
    good, _ = oracle.forward(cfg, w, ids)
    cfg2, w2 = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    MISTAKES[name](cfg2, w2, monkeypatch)
    assert _spread(good, oracle.forward(cfg2, w2, ids)[0]) > 1e-3


def test_needles_and_memories_show_in_bf16_terms():
    cfg, w = model([attention(heads=4, kv_heads=2, dim=32, vdim=32, window=50, keep=3, experts=0)], streams=0, vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    for place, mask in ((119 - 49, {"size": 49, "keep_first": 3}), (119 - 50, {"size": 51, "keep_first": 3}), (2, {"size": 50, "keep_first": 2}),
                        (3, {"size": 50, "keep_first": 4})):
        ids = tokens_of(cfg, 120, seed=1, below=62)
        ids[-1], ids[place] = 62, 63
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"] = mask
        a, b = oracle.forward(cfg, w, ids)[0][-1:], oracle.forward(other, w, ids)[0][-1:]
        assert _spread(a, b) > 0.3, place
    cfg, w = model([delta(conv=2, experts=0)], streams=0, vocab=40, width=64)
    lasting_memory(cfg, w, write=38, read=39)
    ids = tokens_of(cfg, 150, seed=3, below=38)
    ids[-1] = 39
    a = oracle.forward(cfg, w, ids)[0][-1:]
    ids[4] = 38
    assert _spread(a, oracle.forward(cfg, w, ids)[0][-1:]) > 0.3


def test_sharp_routing_is_never_close():
    cfg, w = model([delta(experts=9, top=1), attention(experts=12, top=3, window=20)], streams=3, vocab=96, width=96)
    sharp_routing(cfg, w)
    gaps = []
    oracle.forward(cfg, w, tokens_of(cfg, 150, seed=7), gaps=gaps)
    assert len(gaps) == 2 and min(gaps) > 0.02
    chosen = set()
    orig = oracle.torch.topk
    try:
        oracle.torch.topk = lambda *a, **k: (lambda r: (chosen.update(r.indices.tolist()), r)[1])(orig(*a, **k))
        oracle.forward(cfg, w, tokens_of(cfg, 60, seed=8))
    finally:
        oracle.torch.topk = orig
    assert len(chosen) >= 5


def test_scheduler_counts_kept_pages():
    from neuralfn_b200.serving.scheduler import StepRequest, StepScheduler
    from neuralfn_b200.serving.engine import Sampling
    cfg, w = model([attention(window=70, keep=65, experts=0)], streams=0)
    limits = engine_config(MurilornConfig.from_dict(cfg), max_batch=2, max_seq=4096, kv_tokens=4096, max_step_rows=64)
    eng = type("E", (), dict(config=limits, has_steps=True, free_tokens=4096))()
    need = StepScheduler(eng)._pages_for(StepRequest(0, [1] * 2000, 500, Sampling(), None))
    assert need == (70 + 128 + 64 + 64 + 63) // 64                # window, two kept pages, one pass, the page at hand


def test_registry_knows_the_design(tmp_path):
    cfg, _ = rich()
    a = architecture_of(cfg)
    assert a.family == "murilorn" and a.component == "layered" and a.dtypes == ("bfloat16", "float32") and a.steps
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert is_model_directory(tmp_path)
