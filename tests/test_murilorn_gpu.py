"""Murilorn on the layer-list engine against the plain reference: every mechanism alone and together, whole prompts, token by token, cut
prompts, mixed batches, reused pages and slots, edges of windows, kept tokens, pages and chunks, greedy generation through the scheduler -
in bf16 and in 32-bit."""
import json

import pytest
import torch

import murilorn_oracle as oracle
from murilorn_cases import attention, boost_needle, delta, lasting_memory, model, sharp_routing, tokens_of
from step_helpers import repeat_cuts, run_cuts, run_mixed, worst

pytestmark = pytest.mark.gpu

TOL = {"bfloat16": 0.03, "float32": 3e-5}      # root mean square over the vocabulary, relative to the logits' spread


def make_engine(cfg, weights, dtype="float32", **kw):
    from neuralfn_b200.models.murilorn import MurilornConfig, engine_config, pack_tensors
    from neuralfn_b200.serving import ResidentEngine
    c = MurilornConfig.from_dict(cfg, weights)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq", 1024)
    eng = ResidentEngine(engine_config(c, dtype=dtype, **kw))
    eng.load_named_tensors(pack_tensors(c, weights))
    return eng


def routed(layers, **kw):
    cfg, w = model(layers, **kw)
    sharp_routing(cfg, w)
    return cfg, w


def everything(routing=True, **kw):
    n = dict(experts=10, top=2) if routing else {}
    return (routed if routing else model)(
        [delta(heads=6, kv_heads=3, dim=48, vdim=32, conv=4, **n), attention(heads=6, kv_heads=2, dim=32, vdim=48, window=48, keep=5, **n),
         delta(heads=2, kv_heads=2, dim=32, vdim=64, conv=2, **n), attention(window=100, keep=70, experts=0)], streams=3, loop=(1, 3, 2), width=96, **kw)


def grid():
    none = dict(experts=0)
    return {
        "attention": model([attention(**none)], streams=0),
        "attention_no_cap": model([attention(softcap=0, scale=0.2, **none)], streams=0),
        "window": model([attention(window=5, **none), attention(window=33, **none)], streams=0),
        "window1": model([attention(window=1, keep=1, **none)], streams=0),
        "kept": model([attention(window=7, keep=1, **none), attention(window=20, keep=90, **none), attention(window=64, keep=64, **none)], streams=0),
        "one_head": model([attention(heads=1, kv_heads=1, dim=16, vdim=16, window=9, keep=3, **none)], streams=0),
        "wide_heads": model([attention(heads=4, kv_heads=1, dim=160, vdim=144, window=70, keep=4, scale=0.1, **none)], streams=0),
        "many_groups": model([attention(heads=24, kv_heads=2, dim=32, vdim=32, window=70, keep=4, **none)], streams=0),
        "huge_head": model([attention(heads=2, kv_heads=1, dim=272, vdim=288, window=40, keep=2, scale=0.05, **none)], streams=0),
        "delta": model([delta(**none)], streams=0),
        "delta_one_head": model([delta(heads=1, kv_heads=1, dim=16, vdim=16, **none)], streams=0),
        "delta_conv1": model([delta(conv=1, **none), delta(conv=2, **none)], streams=0),
        "delta_conv5": model([delta(conv=5, **none), delta(conv=4, **none)], streams=0),
        "delta_groups": model([delta(heads=8, kv_heads=2, dim=24, vdim=40, **none), delta(heads=3, kv_heads=3, dim=64, vdim=16, **none)], streams=0),
        "delta_wide": model([delta(heads=2, kv_heads=1, dim=144, vdim=136, **none)], streams=0),
        "delta_wider": model([delta(heads=2, kv_heads=2, dim=320, vdim=48, **none)], streams=0),
        "delta_ranks": model([delta(rank_decay=40, rank_gate=4, **none)], streams=0),
        "experts": model([attention(window=40, experts=3, top=3)], streams=0),
        "one_expert": model([delta(experts=1, top=1, ff=48)], streams=0),
        "routed": routed([attention(window=40, experts=6, top=1), delta(experts=12, top=3, ff=24)], streams=0),
        "streams1": model([attention(window=40), delta()], streams=1),
        "streams2": model([attention(window=40), delta(**none)], streams=2),
        "streams5": model([attention(window=40), delta()], streams=5),
        "streams9": model([delta(), attention(window=12, **none)], streams=9),
        "loop": model([delta(), attention(window=30, keep=2, **none), delta(**none)], loop=(0, 2, 3)),
        "loop_of_all": model([attention(window=50, keep=3)], loop=(0, 1, 4)),
        "odd_sizes": model([delta(heads=3, kv_heads=1, dim=40, vdim=24, ff=56), attention(heads=5, kv_heads=5, dim=24, vdim=56, window=50, keep=9, ff=72)], vocab=203, width=136),
        "constants": model([attention(scale=0.05, softcap=3.0, window=77), delta()], embed_scale=0.7, eps=0.03, logit_scale=0.4, logit_softcap=2.0),
        "no_logit_cap": model([delta()], logit_scale=1.0, logit_softcap=0),
        "all": everything(),
    }


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(grid()))
def test_mechanism_prompt_decode_and_portions(case, dtype):
    cfg, w = grid()[case]
    T = 150
    ids, gaps = tokens_of(cfg, T, seed=3), []
    want, _ = oracle.forward(cfg, w, ids, gaps=gaps)
    assert min(gaps, default=1.0) > 0.02                 # no close choices
    eng = make_engine(cfg, w, dtype)
    for cuts in ([T], [1] * T, repeat_cuts(T, [2]), repeat_cuts(T, [17, 1, 40, 3]), repeat_cuts(T, [16, 31]), [64, 64, 22], [63, 2, 85]):
        assert worst(run_cuts(eng, 1, ids, cuts), want) < TOL[dtype], cuts[:4]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,keep", [(1, 0), (2, 1), (31, 6), (64, 64), (65, 33), (130, 3)])
def test_window_and_kept_edges_with_far_keys(window, keep, dtype):
    """A key whose score towers over the others, exactly at and around the window's far edge and the last kept token, in prompts and in
    decoding, at places before, on and after page borders."""
    cfg, w = model([attention(heads=4, kv_heads=2, dim=32, vdim=32, window=window, keep=keep, experts=0)], streams=0, vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    eng = make_engine(cfg, w, dtype)
    for end in (210, 255, 256):
        places = {end - d for d in (1, window - 1, window, window + 1)} | {0, keep - 1, keep, keep + 1}
        for place in sorted(p for p in places if 0 <= p < end):
            ids = tokens_of(cfg, end + 1, seed=end, below=62)
            ids[end], ids[place] = 62, 63
            want, _ = oracle.forward(cfg, w, ids)
            for cuts in ([end + 1], [end, 1], [end - 1, 2], repeat_cuts(end + 1, [50])):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (end, place, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_the_state_holds_arrives_later(dtype):
    """One token is written, all others leave the state alone; it is read back at every kind of distance and cut."""
    cfg, w = model([delta(heads=4, kv_heads=2, dim=32, vdim=32, conv=2, experts=0)], streams=0, vocab=40)
    lasting_memory(cfg, w, write=38, read=39)
    eng = make_engine(cfg, w, dtype)
    base = tokens_of(cfg, 300, seed=5, below=38)
    for place in (0, 1, 14, 15, 16, 17, 63, 64, 100):
        for dist in (1, 2, 15, 16, 17, 48, 150):
            ids = base[:place + dist] + [39]
            ids[place] = 38
            want, _ = oracle.forward(cfg, w, ids)
            n = len(ids)
            for cuts in ([n], [n - 1, 1], repeat_cuts(n, [33, 2]), repeat_cuts(n, [16]), [place + 1, n - place - 1]):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (place, dist, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rate,bias", [(4.0, 3.0), (-14.0, 0.0), (2.0, -2.0)])
def test_extreme_decays(rate, bias, dtype):
    """States that forget within a token, never, or both within one head."""
    cfg, w = model([delta(dim=48, experts=0), delta(conv=1, experts=0)], streams=0)
    for i in range(2):
        w[f"l{i}.mix.A_log"].fill_(rate)
        w[f"l{i}.mix.dt_bias"].fill_(bias)
        if rate == 2.0:
            w[f"l{i}.mix.dt_bias"][::2] = -12.0
    ids = tokens_of(cfg, 200, seed=11)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([200], repeat_cuts(200, [40, 1, 17]), [150] + [1] * 50):
        assert worst(run_cuts(eng, 2, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens(dtype):
    cfg, w = everything()
    eng = make_engine(cfg, w, dtype)
    for n in (1, 2, 3, 5, 16, 17):
        ids = tokens_of(cfg, n, seed=n)
        want, _ = oracle.forward(cfg, w, ids)
        for cuts in ([n], [1] * n):
            assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reuse(dtype):
    """Every logit of a mixed batch equals the request's own, in pages and slots that held other requests before."""
    cfg, w = everything()
    lengths = [190, 70, 3, 128, 64, 41, 150, 2]
    seqs = [tokens_of(cfg, n, seed=100 + i) for i, n in enumerate(lengths)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    eng = make_engine(cfg, w, dtype, max_batch=3, max_seq=256, kv_tokens=384)
    room = eng.free_tokens
    got = run_mixed(eng, seqs, slots=3, room=384, seed=5)
    for i in range(len(seqs)):
        assert worst(got[i], want[i]) < TOL[dtype], i
    assert eng.free_tokens == room
    eng.close()


def test_batch_of_single_tokens_leaves_idle_slots_alone():
    """A slot that is left out of decode steps keeps its state; padded rows of the replayed graph touch nothing."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = everything()
    eng = make_engine(cfg, w, "float32", max_batch=4)
    ids = [tokens_of(cfg, 40, seed=20 + s) for s in range(4)]
    want = [oracle.forward(cfg, w, s)[0] for s in ids]
    at, got = [0] * 4, [[] for _ in ids]
    for n in range(60):
        who = [s for s in range(4) if (n + s) % (s + 2) != 0 and at[s] < 40]
        if not who:
            continue
        rows = eng.step([StepEntry(s, [ids[s][at[s]]], (0,)) for s in who], logits=True)[1]
        for k, s in enumerate(who):
            got[s].append(rows[k:k + 1])
            at[s] += 1
    for s in range(4):
        assert worst(torch.cat(got[s]), want[s][:at[s]]) < TOL["float32"], s
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_pages_given_back(dtype):
    cfg, w = model([attention(window=70, keep=5, scale=0.2), delta(), attention(window=20, keep=66, scale=0.2, experts=0)], seed=10)
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
    assert room - low <= 70 + 3 * 64, "pages behind the window stay held"
    eng.release(0)
    assert eng.free_tokens == room
    eng.close()


def test_models_without_pages_count_tokens_all_the_same():
    from neuralfn_b200.serving import EngineError, StepEntry
    cfg, w = model([delta()], streams=0)
    eng = make_engine(cfg, w, max_batch=2, max_seq=512, kv_tokens=128)
    eng.step([StepEntry(0, tokens_of(cfg, 65, seed=1))])
    with pytest.raises(EngineError, match="pool is full"):
        eng.step([StepEntry(1, tokens_of(cfg, 1, seed=1))])
    eng.release(0)
    assert eng.free_tokens == 128
    prompts = [tokens_of(cfg, n, seed=n) for n in (9, 40)]
    want = [greedy(cfg, w, p, 5) for p in prompts]
    assert min(g for _, g in want) > 1e-3
    assert eng.generate(prompts, max_new_tokens=5) == [t for t, _ in want]
    with pytest.raises(EngineError, match="run again"):
        eng.step([StepEntry(0, [1, 2, 3])])
        eng.truncate(0, 2)
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
    cfg, w = everything()
    prompts = [tokens_of(cfg, n, seed=n) for n in (5, 90, 33, 1, 66)]
    want = [greedy(cfg, w, p, 8) for p in prompts]
    assert min(g for _, g in want) > 1e-3      # no near ties
    from neuralfn_b200.serving.scheduler import StepScheduler
    eng = make_engine(cfg, w, "float32", max_batch=2, max_seq=256, kv_tokens=512)
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
    eng.close()


def test_fork_copies_pages_history_and_state():
    cfg, w = everything()
    ids = tokens_of(cfg, 190, seed=4)
    want, _ = oracle.forward(cfg, w, ids)
    from neuralfn_b200.serving import EngineError, StepEntry
    eng = make_engine(cfg, w)
    room = eng.free_tokens
    run_cuts(eng, 0, ids[:160], [160])
    eng.fork(0, 2)
    eng.step([StepEntry(0, tokens_of(cfg, 40, seed=8))])
    eng.release(0)
    got = torch.cat([eng.step([StepEntry(2, [t], (0,))], logits=True)[1] for t in ids[160:]])
    assert worst(got, want[160:]) < TOL["float32"]
    with pytest.raises(EngineError, match="run again"):
        eng.truncate(2, 50)
    eng.release(2)
    assert eng.free_tokens == room
    eng.close()


def _directory(tmp_path, cfg, w):
    from neuralfn_b200.checkpoint.safetensors_io import write_safetensors
    for y in cfg["layers"]:                      # the tensors' shapes say these
        y["mixer"].pop("rank_decay", None), y["mixer"].pop("rank_gate", None)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", w)


def test_directory_session_and_command_line(tmp_path, capsys):
    """The model directory through the registry: sessions (prefill, decode, truncate, fork) and ``nfn infer``."""
    from neuralfn_b200.cli.nfn import main
    from neuralfn_b200.serving import GenerationConfig, NativeInferenceModel, NativeModelLoadConfig
    cfg, w = everything()
    _directory(tmp_path, cfg, w)
    ids = tokens_of(cfg, 20, seed=6)
    want, gap = greedy(cfg, w, ids, 4)
    assert gap > 1e-3
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
        assert list(child.decode(GenerationConfig(max_new_tokens=2, temperature=0.0)).token_ids) == greedy(cfg, w, ids[:15], 2)[0]


def test_trace_replay_writes_wanted_rows(tmp_path):
    import io
    import numpy as np
    from neuralfn_b200.serving import trace
    cfg, w = everything()
    _directory(tmp_path, cfg, w)
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
    for n, want in {0: [la[65], la[2]], 1: [la[66]], 2: [lb[8], la[69]]}.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", "<f4").copy()).view(len(want), -1)
        assert worst(got, torch.stack(want)) < TOL["float32"]
