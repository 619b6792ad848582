"""Bulidra on the layer-list engine against the plain reference: every mechanism alone and together, whole prompts, token by token, cut
prompts, mixed batches, reused pages and slots, window and page edges, greedy generation through the scheduler - in bf16 and in
32-bit."""
import copy

import pytest
import torch

import bulidra_oracle as oracle
from bulidra_cases import boost_needle, layer, model, tokens_of
from step_helpers import repeat_cuts, run_cuts, run_mixed, worst

pytestmark = pytest.mark.gpu

TOL = {"bfloat16": 0.03, "float32": 3e-5}      # root mean square over the vocabulary, relative to the logits' spread


def make_engine(cfg, weights, dtype="float32", **kw):
    from neuralfn_b200.models.bulidra import BulidraConfig, engine_config, pack_tensors
    from neuralfn_b200.serving import ResidentEngine
    c = BulidraConfig.from_dict(cfg)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq", 1024)
    eng = ResidentEngine(engine_config(c, dtype=dtype, **kw))
    eng.load_named_tensors(pack_tensors(c, weights))
    return eng


def sizes_grid():
    return {
        "plain": model([layer()], side=0),
        "one_head": model([layer(heads=1, kv_heads=1, dim=16, vdim=16)], side=0),
        "no_mlp": model([layer(ff=0), layer(ff=0)], side=0),
        "mlp": model([layer(ff=40)], side=0),
        "conv1": model([layer(conv=1)], side=0),
        "conv2": model([layer(conv=2), layer(conv=2)], side=0),
        "conv5": model([layer(conv=5), layer(conv=4)], side=0),
        "temperature": model([layer(temp=(0.9, 7))], side=0),
        "window": model([layer(window=5), layer(window=33)], side=0),
        "window1": model([layer(window=1)], side=0),
        "window64": model([layer(window=64), layer(window=65), layer(window=63)], side=0),
        "side": model([layer(), layer(ff=0)], side=24),
        "shared": model([layer(window=20), layer(kv_from=0, window=90), layer(), layer(kv_from=2, window=3), layer(kv_from=0, window=6)], side=0),
        "odd_sizes": model([layer(heads=6, kv_heads=2, dim=40, vdim=24, ff=56, window=50), layer(heads=5, kv_heads=5, dim=24, vdim=56, ff=72)],
                           vocab=203, width=136, side=20),
        "wide_heads": model([layer(heads=4, kv_heads=1, dim=160, vdim=144, window=70, ff=32)], side=0),
        "many_groups": model([layer(heads=24, kv_heads=2, dim=32, vdim=32, ff=32, window=100)], side=0),
        "huge_head": model([layer(heads=2, kv_heads=1, dim=272, vdim=288, ff=32, window=40)], side=0),
        "constants": model([layer(scale=0.05, temp=(2.0, 3)), layer(scale=0.6, window=77)], side=8, embed_scale=0.5, eps=0.03),
        "all": model([layer(temp=(0.5, 32), window=48, ff=96), layer(ff=64, conv=4, window=100), layer(kv_from=1, window=130, ff=0, temp=(0.3, 50)),
                      layer(heads=8, kv_heads=4, dim=64, vdim=48, ff=80)], side=16),
    }


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(sizes_grid()))
def test_mechanism_prompt_decode_and_portions(case, dtype):
    cfg, w = sizes_grid()[case]
    T = 150
    ids = tokens_of(cfg, T, seed=3)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([T], [1] * T, repeat_cuts(T, [2]), repeat_cuts(T, [17, 1, 40, 3]), [64, 64, 22], [63, 2, 85]):
        assert worst(run_cuts(eng, 1, ids, cuts), want) < TOL[dtype], cuts[:4]
    eng.close()


def test_paths_agree_with_the_plain_kernels_in_bf16():
    """The tensor-core attention kernels against 32-bit mode with bf16-sized tolerance, over head sizes that select every variant."""
    for h, g, d, v in ((8, 2, 128, 128), (16, 1, 64, 96), (3, 3, 48, 80), (4, 2, 256, 256), (12, 4, 96, 16), (32, 2, 16, 128), (130, 1, 16, 16)):
        cfg, w = model([layer(heads=h, kv_heads=g, dim=d, vdim=v, window=90, ff=32, scale=d ** -0.5)], side=0)
        ids = tokens_of(cfg, 260, seed=h)
        ref = run_cuts(make_engine(cfg, w, "float32"), 0, ids, [260]).double()
        eng = make_engine(cfg, w, "bfloat16")
        for cuts in ([260], [200] + [1] * 60, repeat_cuts(260, [30, 15, 70])):
            assert worst(run_cuts(eng, 0, ids, cuts), ref) < TOL["bfloat16"], (h, g, d, v, cuts[:3])
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [1, 2, 31, 64, 65, 200])
def test_window_edges_and_far_keys(window, dtype):
    """A key whose score towers over the others, exactly at and around the window's far edge, in prompts and in decoding, at places
    before, on and after page borders."""
    cfg, w = model([layer(heads=4, kv_heads=2, dim=32, vdim=32, window=window, conv=1, ff=0)], side=0, vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    eng = make_engine(cfg, w, dtype)
    for end in (210, 255, 256, 257):
        for dist in sorted({0, 1, window - 1, window, window + 1, end}):
            if dist < 0 or dist > end or dist == 0:
                continue
            ids = tokens_of(cfg, end + 1, seed=end, below=62)
            ids[end] = 62
            ids[end - dist] = 63
            want, _ = oracle.forward(cfg, w, ids)
            for cuts in ([end + 1], [end, 1], [end - 1, 2], repeat_cuts(end + 1, [50])):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (end, dist, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(dtype):
    cfg, w = sizes_grid()["all"]
    eng = make_engine(cfg, w, dtype)
    for n in (1, 2, 3, 5):
        ids = tokens_of(cfg, n, seed=n)
        want, _ = oracle.forward(cfg, w, ids)
        for cuts in ([n], [1] * n):
            assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reuse(dtype):
    """Unequal requests together, some fed by portions and some by single tokens, left out of steps, ended and replaced, in a pool that
    holds only what is live: every logit equals the request's own."""
    cfg, w = sizes_grid()["all"]
    lengths = [190, 70, 3, 128, 64, 41, 150, 2]
    seqs = [tokens_of(cfg, n, seed=100 + i) for i, n in enumerate(lengths)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    eng = make_engine(cfg, w, dtype, max_batch=3, max_seq=256, kv_tokens=192 + 128 + 64)
    room = eng.free_tokens
    got = run_mixed(eng, seqs, slots=3, room=384, seed=5)
    for i in range(len(seqs)):
        assert worst(got[i], want[i]) < TOL[dtype], i
    assert eng.free_tokens == room
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_pages_given_back(dtype):
    cfg, w = model([layer(window=70, scale=0.2), layer(window=20, kv_from=0, scale=0.2), layer(window=40, ff=48, scale=0.2)], side=8, seed=10)
    ids = tokens_of(cfg, 420, seed=9)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype, max_batch=2, max_seq=512, max_step_rows=64)
    room, low = eng.free_tokens, 10 ** 9
    from neuralfn_b200.serving import StepEntry
    out = [eng.step([StepEntry(0, ids[:200], range(200))], logits=True)[1]]      # longer than one pass
    for t in range(200, 420):
        out.append(eng.step([StepEntry(0, [ids[t]], (0,))], logits=True)[1])
        low = min(low, eng.free_tokens)
    assert worst(torch.cat(out), want) < TOL[dtype]
    assert room - low <= 70 + 2 * 64, "pages behind the window stay held"
    eng.release(0)
    assert eng.free_tokens == room
    eng.close()


def test_pool_limits_are_errors():
    from neuralfn_b200.serving import EngineError, StepEntry
    cfg, w = sizes_grid()["plain"]
    eng = make_engine(cfg, w, max_batch=2, max_seq=512, kv_tokens=128)
    eng.step([StepEntry(0, tokens_of(cfg, 65, seed=1))])
    with pytest.raises(EngineError, match="pool is full"):
        eng.step([StepEntry(1, tokens_of(cfg, 1, seed=1))])
    with pytest.raises(EngineError, match="vocabulary"):
        eng.step([StepEntry(0, [cfg["vocab"]])])
    with pytest.raises(EngineError, match="slot"):
        eng.step([StepEntry(0, [1]), StepEntry(0, [2])])
    assert eng.slot_length(0) == 65
    eng.release(0)
    eng.step([StepEntry(1, tokens_of(cfg, 128, seed=1))])
    with pytest.raises(EngineError, match="not available"):
        eng.enable_verify(4)
    eng.close()


def greedy(cfg, w, ids, n):
    ids, gap = list(ids), []
    for _ in range(n):
        row = oracle.forward(cfg, w, ids)[0][-1]
        top = torch.topk(row, 2).values
        gap.append(float(top[0] - top[1]))
        ids.append(int(row.argmax()))
    return ids[-n:], min(gap)


def test_greedy_generation_through_the_scheduler():
    cfg, w = sizes_grid()["all"]
    prompts = [tokens_of(cfg, n, seed=n) for n in (5, 90, 33, 1, 66)]
    want = [greedy(cfg, w, p, 8) for p in prompts]
    assert min(g for _, g in want) > 1e-3      # no near ties
    from neuralfn_b200.serving.scheduler import StepScheduler
    eng = make_engine(cfg, w, "float32", max_batch=2, max_seq=256, kv_tokens=256)
    assert eng.generate(prompts, max_new_tokens=8) == [t for t, _ in want]
    sched = StepScheduler(eng, step_rows=7)      # prompts in portions of a few rows
    ids = [sched.submit(p, 8) for p in prompts]
    done = sched.run()
    assert [done[i] for i in ids] == [t for t, _ in want]
    assert eng.prefill(0, prompts[1]) == want[1][0][0]      # the one-sequence calls of every engine
    nxt = [want[1][0][0]]
    for _ in range(7):
        nxt.append(eng.decode({0: nxt[-1]})[0])
    assert nxt == want[1][0]
    assert torch.argmax(eng.last_logits(0)) == nxt[-1]
    assert eng.launches > 0
    eng.close()


def test_fork_copies_pages_and_history():
    cfg, w = sizes_grid()["all"]
    ids = tokens_of(cfg, 130, seed=4)
    want, _ = oracle.forward(cfg, w, ids)
    from neuralfn_b200.serving import EngineError, StepEntry
    eng = make_engine(cfg, w)
    run_cuts(eng, 0, ids[:100], [100])
    eng.fork(0, 2)
    eng.step([StepEntry(0, tokens_of(cfg, 40, seed=8))])
    eng.release(0)
    got = torch.cat([eng.step([StepEntry(2, [t], (0,))], logits=True)[1] for t in ids[100:]])
    assert worst(got, want[100:]) < TOL["float32"]
    with pytest.raises(EngineError, match="run again"):
        eng.truncate(2, 50)
    eng.close()


def test_directory_session_and_command_line(tmp_path, capsys):
    """The model directory through the registry: sessions (prefill, decode, truncate, fork) and ``nfn infer``."""
    import json
    from neuralfn_b200.checkpoint.safetensors_io import write_safetensors
    from neuralfn_b200.cli.nfn import main
    from neuralfn_b200.serving import GenerationConfig, NativeInferenceModel, NativeModelLoadConfig
    cfg, w = sizes_grid()["all"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", w)
    ids = tokens_of(cfg, 20, seed=6)
    w16 = {k: v.to(torch.bfloat16) for k, v in w.items()}
    want, gap = greedy(cfg, w16, ids, 4)
    assert main(["infer", "--checkpoint", str(tmp_path), "--prompt-tokens", ",".join(map(str, ids)), "--max-new-tokens", "4", "--dtype", "float32"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["token_ids"] == want
    with NativeInferenceModel.load(tmp_path, NativeModelLoadConfig(session_count=2, context_tokens=256, dtype="float32")) as m:
        s = m.create_session()
        s.prefill(ids[:12])
        s.prefill(ids[12:])
        r = s.decode(GenerationConfig(max_new_tokens=4, temperature=0.0))
        assert list(r.token_ids) == want
        child = m.fork_session(s, 15)
        s.truncate(20)
        assert list(s.decode(GenerationConfig(max_new_tokens=4, temperature=0.0)).token_ids) == want
        tail = greedy(cfg, w16, ids[:15], 2)[0]
        assert list(child.decode(GenerationConfig(max_new_tokens=2, temperature=0.0)).token_ids) == tail


def test_trace_replay_writes_wanted_rows(tmp_path):
    import io
    import json
    import numpy as np
    from neuralfn_b200.checkpoint.safetensors_io import write_safetensors
    from neuralfn_b200.serving import trace
    cfg, w = sizes_grid()["all"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", w)
    a, b = tokens_of(cfg, 70, seed=1), tokens_of(cfg, 9, seed=2)
    la, lb = oracle.forward(cfg, w, a)[0], oracle.forward(cfg, w, b)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [65, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[66:67], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "b2", "tokens": b, "want": [8]}, {"id": "a", "tokens": a[67:], "want": [2]}], "end": ["a", "b2"]}]
    (tmp_path / "o").mkdir()
    text = io.StringIO()
    rc = trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "192"],
                    io.StringIO("\n".join(map(json.dumps, steps)) + "\n"), text)
    assert rc == 0 and text.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    rows = {0: [la[65], la[2]], 1: [la[66]], 2: [lb[8], la[69]]}
    for n, want in rows.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", "<f4").copy()).view(len(want), -1)
        assert worst(got, torch.stack(want)) < TOL["float32"]


def test_oracle_weights_are_left_alone():
    cfg, w = sizes_grid()["all"]
    before = copy.deepcopy(w)
    oracle.forward(cfg, w, [1, 2, 3])
    assert all(torch.equal(before[k], w[k]) for k in w)
