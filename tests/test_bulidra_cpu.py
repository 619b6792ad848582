"""Bulidra without a GPU: configuration, tensor packing, how much every mistake would show in the reference's logits, the step scheduler
and the trace replay on a stand-in engine, the architecture registry."""
import copy
import io
import json

import pytest
import torch

import bulidra_oracle as oracle
from bulidra_cases import boost_needle, layer, model, tokens_of
from neuralfn_b200.models.bulidra import BulidraConfig, BulidraError, engine_config, expected_shapes, pack_tensors
from neuralfn_b200.serving import StepEntry, trace
from neuralfn_b200.serving.architectures import ArchitectureError, architecture_of, is_model_directory
from neuralfn_b200.serving.scheduler import StepScheduler


def rich():
    return model([layer(heads=6, kv_heads=2, dim=24, vdim=40, window=9, temp=(0.7, 5), ff=40), layer(heads=6, kv_heads=2, dim=24, vdim=40, kv_from=0, window=14, ff=0),
                  layer(conv=1)], vocab=70, width=72, side=12)


def test_configuration_round_trip_and_refusals():
    cfg, _ = rich()
    c = BulidraConfig.from_dict(cfg)
    assert BulidraConfig.from_dict(c.to_dict()) == c
    e = engine_config(c, max_batch=3, max_seq=100)
    assert [y.kv_from for y in e.layers] == [-1, 0, -1] and [y.window for y in e.layers] == [9, 14, 0] and e.window == 0
    assert e.layers[0].alibi == 8.0 and e.layers[0].q_temp_every == 5 and e.layers[1].ff == 0 and e.estimate_device_bytes() > 0
    bad = [("type", "recurrent"), ("mixer.kv_heads", 4), ("mixer.mask", {"size": 0}), ("mixer.surprise", 1), ("mlp", {"kind": "experts", "ff": 8}),
           ("mixer.kv_from", 0), ("mixer.q_temp", {"coef": 1.0, "every": 2.5})]
    for path, value in bad:
        broken = copy.deepcopy(cfg)
        node, *rest = [broken["layers"][0]], *path.split(".")
        node = node[0]
        for k in rest[:-1]:
            node = node[k]
        node[rest[-1]] = value
        with pytest.raises(BulidraError):
            BulidraConfig.from_dict(broken)


def test_packed_tensors_compute_the_same_projections():
    cfg, w = rich()
    c = BulidraConfig.from_dict(cfg)
    assert set(expected_shapes(c)) == set(w)
    t = pack_tensors(c, w)
    h = torch.randn(5, 72, dtype=torch.float64)
    hp = torch.zeros(5, 80, dtype=torch.float64)
    hp[:, :72] = h
    y = hp @ t["layers.0.w_in"].double().T
    dp, vp, fp = 32, 48, 48
    q, k, v, g, gate, up = y.split([6 * dp, 2 * dp, 2 * vp, 6 * vp, fp, fp], 1)
    for got, n, heads, pad in ((q, "mix.q", 6, dp), (k, "mix.k", 2, dp), (v, "mix.v", 2, vp), (g, "mix.g", 6, vp), (gate, "mlp.gate", 1, fp), (up, "mlp.up", 1, fp)):
        ref = (h @ w["l0." + n].double().T).view(5, heads, -1)
        got = got.reshape(5, heads, pad)
        assert torch.allclose(got[..., :ref.shape[2]], ref) and not got[..., ref.shape[2]:].any()
    a, f = torch.randn(5, 6, 40, dtype=torch.float64), torch.randn(5, 40, dtype=torch.float64)
    cat = torch.zeros(5, 6 * vp + fp, dtype=torch.float64)
    cat[:, :6 * vp].view(5, 6, vp)[..., :40] = a
    cat[:, 6 * vp:6 * vp + 40] = f
    ref = a.reshape(5, -1) @ w["l0.mix.o"].double().T + f @ w["l0.mlp.down"].double().T
    assert torch.allclose((cat @ t["layers.0.w_out"].double().T)[:, :72], ref)
    assert t["layers.0.conv"].shape == (3, 6 * dp + 2 * dp + 2 * vp) and t["layers.2.conv"].shape[0] == 1
    assert torch.equal(t["layers.0.conv"][:, 32:56].T, w["l0.mix.q.conv"][24:48])
    se = t["side_embed"].view(70, 3, 16)
    assert torch.equal(se[..., :12], w["side.embed"].view(70, 3, 12)) and not se[..., 12:].any()
    assert t["layers.1.w_in"].shape[0] == 6 * dp + 6 * vp and t["layers.1.w_out"].shape == (80, 6 * vp)
    broken = dict(w)
    broken.pop("l1.mix.q")
    with pytest.raises(BulidraError, match="l1.mix.q"):
        pack_tensors(c, broken)


def _spread(a, b):
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / (a - a.mean(-1, keepdim=True)).pow(2).mean().sqrt())


MISTAKES = {
    "window one wider": lambda c, w: c["layers"][0]["mixer"]["mask"].update(size=10),
    "window one narrower": lambda c, w: c["layers"][0]["mixer"]["mask"].update(size=8),
    "reader keeps the owner's window": lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=9),
    "no temperature": lambda c, w: c["layers"][0]["mixer"].pop("q_temp"),
    "temperature period": lambda c, w: c["layers"][0]["mixer"]["q_temp"].update(every=6),
    "score scale": lambda c, w: c["layers"][2]["mixer"].update(scale=0.38),
    "norm epsilon": lambda c, w: c["norm"].update(eps=0.1),
    "embedding scale": lambda c, w: c["embedding"].update(scale=4.0),
    "no token input": lambda c, w: c.pop("token_side"),
    "no feed-forward": lambda c, w: c["layers"][0].update(mlp=None),
    "history dropped": lambda c, w: w["l0.mix.k.conv"][:, 0].zero_(),
    "value convolution": lambda c, w: w["l0.mix.v.conv"][:, 1].zero_(),
    "one-tap convolution": lambda c, w: w["l2.mix.k.conv"].fill_(1.0),
    "output gate": lambda c, w: w["l0.mix.g"].zero_(),
    "final norm": lambda c, w: w["final.norm"].fill_(1.0),
}


@pytest.mark.parametrize("name", list(MISTAKES))
def test_a_planted_mistake_shows(name):
    """Every mistake moves some logit row by far more than the tolerance the GPU tests use in 32-bit (3e-5)."""
    cfg, w = rich()
    ids = tokens_of(cfg, 40, seed=2)
    good, _ = oracle.forward(cfg, w, ids)
    cfg2, w2 = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    MISTAKES[name](cfg2, w2)
    assert _spread(good, oracle.forward(cfg2, w2, ids)[0]) > 2e-3


def test_a_needle_shows_in_bf16_terms():
    cfg, w = model([layer(heads=4, kv_heads=2, dim=32, vdim=32, window=50, conv=1, ff=0)], side=0, vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    for dist, size in ((49, 49), (50, 51)):
        ids = tokens_of(cfg, 120, seed=1, below=62)
        ids[-1], ids[119 - dist] = 62, 63
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = size
        a, b = oracle.forward(cfg, w, ids)[0][-1:], oracle.forward(other, w, ids)[0][-1:]
        assert _spread(a, b) > 0.3


class FakeEngine:
    """Counts tokens per slot; the successor of a sequence is its length modulo 50."""

    def __init__(self, max_batch, pool, max_seq=64, window=0):
        self.config = type("C", (), dict(max_batch=max_batch, max_seq=max_seq, max_step_rows=32, vocab=50, window=window))
        self.pool, self.has_steps, self.held, self.batches = pool, True, {}, []

    @property
    def free_tokens(self):
        return self.pool - sum((n + 63) // 64 * 64 for n in self.held.values())

    def release(self, slot):
        self.held.pop(slot, None)

    def step(self, entries, logits=False):
        self.batches.append([(e.slot, len(e.tokens)) for e in entries])
        out, rows = [], []
        for e in entries:
            base = self.held.get(e.slot, 0)
            self.held[e.slot] = base + len(e.tokens)
            assert self.held[e.slot] <= self.config.max_seq
            out.append([(base + w + 1) % 50 for w in e.want])
            rows += [torch.full((50,), float(base + w)) for w in e.want]
        assert self.free_tokens >= 0, "pool overrun"
        return out, torch.stack(rows) if logits and rows else None


def test_scheduler_mixes_portions_with_decoding_and_respects_the_pool():
    eng = FakeEngine(max_batch=3, pool=128)
    sched = StepScheduler(eng, step_rows=8)
    want = {}
    for n, new in ((20, 5), (3, 9), (40, 4), (1, 1), (30, 3)):
        rid = sched.submit(list(range(n)), new)
        want[rid] = [(n + i) % 50 for i in range(new)]
    assert sched.run() == want
    assert all(sum(n for _, n in b) <= 8 for b in eng.batches)
    assert any(len(b) > 1 and {n for _, n in b} != {1} and 1 in {n for _, n in b} for b in eng.batches), "no step mixed a portion with a token"
    assert max(len(b) for b in eng.batches) == 2          # the pool holds two sequences, not three
    with pytest.raises(ValueError, match="pool"):
        StepScheduler(FakeEngine(2, 64, max_seq=200)).submit([1] * 100, 10)
    eos = StepScheduler(FakeEngine(2, 128))
    rid = eos.submit([1, 2, 3], 20, eos_token=6)
    assert eos.run()[rid] == [3, 4, 5, 6]
    with pytest.raises(ValueError, match="prompt"):
        eos.submit([], 3)


def test_trace_replay_keeps_names_apart_and_orders_rows():
    eng = FakeEngine(max_batch=2, pool=256)
    r = trace.TraceReplay(eng)
    out = r.run({"step": 0, "entries": [{"id": "x", "tokens": [1, 2, 3, 4], "want": [3, 1]}, {"id": "y", "tokens": [9], "want": [0]}], "end": ["y"]})
    assert out[:, 0].tolist() == [3.0, 1.0, 0.0]
    assert r.run({"step": 1, "entries": [{"id": "z", "tokens": [5, 6], "want": []}], "end": []}) is None
    out = r.run({"step": 2, "entries": [{"id": "x", "tokens": [7], "want": [0]}, {"id": "z", "tokens": [7], "want": [0]}], "end": ["x", "z"]})
    assert out[:, 0].tolist() == [4.0, 2.0] and eng.held == {}
    with pytest.raises(ValueError, match="slots"):
        r.run({"entries": [{"id": str(i), "tokens": [1], "want": []} for i in range(3)]})


def test_registry_and_unsupported_formats(tmp_path):
    cfg, _ = rich()
    assert architecture_of(cfg).family == "bulidra" and architecture_of({"architectures": ["LlamaForCausalLM"]}).dtypes == ("bfloat16",)
    with pytest.raises(ArchitectureError, match="Nothing"):
        architecture_of({"architecture": "Nothing"})
    assert not is_model_directory(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["LlamaForCausalLM"]}))
    assert is_model_directory(tmp_path)
    rc = trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"], io.StringIO(""), io.StringIO())
    assert rc == trace.EXIT_UNSUPPORTED


def test_component_sources_exist():
    from neuralfn_b200.ops import _build
    for name, files in _build.COMPONENTS.items():
        assert len(_build._sources(name)) == len(files)


def test_step_entries_are_checked_before_the_engine_sees_them():
    from neuralfn_b200.serving.engine import EngineError, ResidentEngine
    eng = ResidentEngine.__new__(ResidentEngine)
    with pytest.raises(EngineError, match="wanted place"):
        eng.step([StepEntry(0, [1, 2], (2,))])
