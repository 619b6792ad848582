"""Kidolorn on the layer-list engine against the plain reference: every mechanism alone and together, whole prompts, token by token, cut prompts, mixed
batches, reused pages and slots, far keys, what a state holds, first tokens, long decoding, greedy generation through the scheduler - in bf16 and
in 32-bit."""
import json

import pytest
import torch

import kidolorn_oracle as oracle
from kidolorn_cases import boost_needle, dense, lasting_memory, latent, lightning, mingru, model, moe, tokens_of
from step_helpers import repeat_cuts, run_cuts, run_mixed, worst

pytestmark = pytest.mark.gpu

TOL = {"bfloat16": 0.045, "float32": 3e-5}      # root mean square over the vocabulary, relative to the logits' spread


def make_engine(cfg, weights, dtype="float32", **kw):
    from neuralfn_b200.models.kidolorn import KidolornConfig, engine_config, pack_tensors
    from neuralfn_b200.serving import ResidentEngine
    c = KidolornConfig.from_dict(cfg)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq", 1024)
    eng = ResidentEngine(engine_config(c, dtype=dtype, **kw))
    eng.load_named_tensors(pack_tensors(c, weights))
    return eng


def everything(**kw):
    return model([lightning(heads=5, dim=24, vdim=40, mlp=moe()), latent(heads=6, dim=40, rot=24, vdim=24, mlp=dense(72)), mingru(width=88, mlp=moe(experts=6, top=1)),
                  latent(heads=3, dim=24, rot=24, vdim=56, kv_from=1, scale=0.3, mlp=moe(experts=5, top=5, ff=40)), lightning(heads=2, dim=48, vdim=16), mingru(width=40, mlp=dense(40))],
                 width=96, vocab=203, taps=4, **kw)


def grid():
    return {
        "latent": model([latent()]),
        "latent_shared": model([latent(), latent(kv_from=0), latent(heads=2, dim=56, vdim=16, kv_from=0, scale=0.2)]),
        "latent_one_head": model([latent(heads=1, dim=16, rot=2, vdim=16, rank=16)]),
        "latent_odd": model([latent(heads=7, dim=20, rot=10, vdim=36, rank=37)]),
        "latent_many_heads": model([latent(heads=20, dim=16, vdim=16), latent(heads=37, dim=16, vdim=32, kv_from=0)]),
        "latent_wide": model([latent(heads=3, dim=128, rot=64, vdim=128, rank=512, scale=0.08)]),
        "latent_wide_rotation": model([latent(heads=18, dim=72, rot=80, vdim=72, rank=200, scale=0.1)]),
        "latent_wider": model([latent(heads=2, dim=32, rot=16, vdim=272, rank=528, scale=0.2)]),
        "lightning": model([lightning()]),
        "lightning_one_head": model([lightning(heads=1, dim=16, vdim=16)]),
        "lightning_64": model([lightning(heads=2, dim=64, vdim=64), lightning(heads=3, dim=56, vdim=128)]),
        "lightning_128": model([lightning(heads=2, dim=128, vdim=128), lightning(heads=5, dim=80, vdim=48)]),
        "lightning_wide": model([lightning(heads=2, dim=144, vdim=80), lightning(heads=1, dim=320, vdim=16)]),
        "lightning_wide_values": model([lightning(heads=2, dim=16, vdim=208), lightning(heads=1, dim=48, vdim=528)]),
        "lightning_decays": model([lightning(heads=4, decay=[1.0, 0.9999, 0.01, 0.0])]),
        "mingru": model([mingru()]),
        "mingru_narrow": model([mingru(width=5), mingru(width=16)]),
        "mingru_wide": model([mingru(width=300)]),
        "taps1": model([mingru(mlp=dense()), latent(mlp=moe())], taps=1),
        "taps2": model([lightning(mlp=dense()), latent()], taps=2),
        "taps7": model([mingru(mlp=moe()), latent(mlp=dense())], taps=7),
        "dense": model([lightning(mlp=dense(56)), latent(mlp=dense(24, limit=0.4))]),
        "experts": model([latent(mlp=moe())]),
        "experts_all": model([mingru(mlp=moe(experts=3, top=3)), latent(mlp=moe(experts=1, top=1, ff=24))]),
        "experts_many": model([lightning(mlp=moe(experts=40, top=6, limit=2.5))], width=96),
        "constants": model([latent(scale=0.05), mingru(mlp=dense(limit=7.0)), lightning()], eps=0.03),
        "odd_sizes": model([latent(heads=5, rank=24, mlp=moe(ff=72)), mingru(width=52, mlp=dense(88)), lightning(heads=5, dim=40, vdim=24)], vocab=203, width=136),
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
def test_far_keys_at_page_borders(dtype):
    """A key whose score towers over the others, at the start, around page borders and next to the query."""
    cfg, w = model([latent(heads=5, dim=32, rot=16, vdim=32, rank=64)], vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    eng = make_engine(cfg, w, dtype)
    for end in (190, 191, 192, 500):
        for place in (0, 1, 63, 64, 65, 127, 128, end - 65, end - 64, end - 2, end - 1):
            ids = tokens_of(cfg, end + 1, seed=end, below=62)
            ids[end], ids[place] = 62, 63
            want, _ = oracle.forward(cfg, w, ids)
            for cuts in ([end + 1], [end, 1], [end - 1, 2], repeat_cuts(end + 1, [50])):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (end, place, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sink", [9.0, -20.0])
def test_sinks_against_few_and_many_keys(sink, dtype):
    """A sink that takes most of every row's weight, and one that takes none, from the first token on."""
    cfg, w = model([latent(heads=5, rank=64)])
    w["l0.mix.sink"].fill_(sink)
    ids = tokens_of(cfg, 400, seed=6)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([400], [1] * 40 + [360], [300] + [1] * 100, repeat_cuts(400, [33, 2])):
        assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["lightning", "mingru"])
def test_what_the_state_holds_arrives_later(kind, dtype):
    """One token is written, all others leave the state alone; it is read back at every kind of distance and cut."""
    cfg, w = model([lightning(heads=3, dim=32, vdim=32, decay=[1.0, 0.999, 0.98]) if kind == "lightning" else mingru(width=48)], vocab=40)
    lasting_memory(cfg, w, write=38, read=39)
    eng = make_engine(cfg, w, dtype)
    base = tokens_of(cfg, 400, seed=5, below=38)
    for place in (0, 1, 7, 8, 15, 16, 62, 63, 64, 100):
        for dist in (1, 2, 16, 17, 64, 150, 270):
            ids = base[:place + dist] + [39]
            ids[place] = 38
            want, _ = oracle.forward(cfg, w, ids)
            n = len(ids)
            for cuts in ([n], [n - 1, 1], repeat_cuts(n, [33, 2]), repeat_cuts(n, [16]), [place + 1, n - place - 1]):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (place, dist, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [2, 4, 6])
def test_only_the_oldest_tap_counts(taps, dtype):
    """Every sublayer reads the token taps - 1 before: the history is right at portion borders and empty at the start."""
    cfg, w = model([mingru(mlp=dense()), lightning(mlp=dense()), latent()], taps=taps)
    for n in w:
        if ".canon" in n:
            w[n].zero_()
            w[n][:, 0] = 3.0
    ids = tokens_of(cfg, 120, seed=2)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([120], [1] * 120, repeat_cuts(120, [2]), repeat_cuts(120, [3, 1]), repeat_cuts(120, [16, 1, 17]), repeat_cuts(120, [33])):
        assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


@pytest.mark.parametrize("bias", [-14.0, 9.0])
def test_shares_near_zero_and_one(bias):
    """States that hardly move for thousands of tokens, and ones that are replaced by every token; in 32-bit the former may not drift."""
    cfg, w = model([mingru(width=96)])
    w["l0.mix.z.b"].fill_(bias)
    ids = tokens_of(cfg, 3000, seed=4)
    want, _ = oracle.forward(cfg, w, ids)
    for dtype in ("float32", "bfloat16"):
        eng = make_engine(cfg, w, dtype, max_seq=3072)
        for cuts in ([3000], [2900] + [1] * 100, repeat_cuts(3000, [700, 15])):
            assert worst(run_cuts(eng, 2, ids, cuts), want) < TOL[dtype], cuts[:3]
        eng.close()


def test_long_prompts_in_segments():
    """A lightning prompt long enough that its segments run side by side, alone and with others of unequal length."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = model([lightning(heads=2, dim=64, vdim=80, decay=[0.9995, 0.9])])
    seqs = [tokens_of(cfg, n, seed=n) for n in (1500, 70, 900)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    eng = make_engine(cfg, w, "bfloat16", max_seq=1600, max_step_rows=4096)
    for cuts in ([1500], [777, 723], repeat_cuts(1500, [600, 1, 30])):
        assert worst(run_cuts(eng, 3, seqs[0], cuts), want[0]) < TOL["bfloat16"]
    eng.release(3)
    got = eng.step([StepEntry(i, s, range(len(s))) for i, s in enumerate(seqs)], logits=True)[1].split([len(s) for s in seqs])
    for i in range(3):
        assert worst(got[i], want[i]) < TOL["bfloat16"], i
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


def test_several_long_portions_share_or_split_an_expansion():
    """Portions of many requests in one step: their latents fill the expansion's rows more than once."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = model([latent(mlp=dense()), latent(kv_from=0)], vocab=64)
    seqs = [tokens_of(cfg, n, seed=n) for n in (190, 60, 250, 130)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    eng = make_engine(cfg, w, "bfloat16", max_batch=4, max_seq=256, max_step_rows=200)
    half = [eng.step([StepEntry(i, s[:len(s) // 2], range(len(s) // 2)) for i, s in enumerate(seqs)], logits=True)[1],
            eng.step([StepEntry(i, s[len(s) // 2:], range(len(s) - len(s) // 2)) for i, s in enumerate(seqs)], logits=True)[1]]
    a, b = half[0].split([len(s) // 2 for s in seqs]), half[1].split([len(s) - len(s) // 2 for s in seqs])
    for i in range(4):
        assert worst(torch.cat([a[i], b[i]]), want[i]) < TOL["bfloat16"], i
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
def test_wide_batches_of_single_tokens(dtype):
    """More rows than the eight-column products take at a time."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = model([latent(mlp=moe()), mingru(), lightning(heads=8, dim=16, vdim=16, mlp=dense())], vocab=64, width=96)
    n = 75
    ids = [tokens_of(cfg, 12, seed=s) for s in range(n)]
    want = [oracle.forward(cfg, w, s)[0] for s in ids]
    eng = make_engine(cfg, w, dtype, max_batch=n, max_seq=64)
    got = [eng.step([StepEntry(s, [ids[s][t]], (0,)) for s in range(n)], logits=True)[1] for t in range(12)]
    for s in range(n):
        assert worst(torch.stack([g[s] for g in got]), want[s]) < TOL[dtype], s
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    cfg, w = model([latent(mlp=dense()), lightning(), mingru(mlp=dense()), latent(kv_from=0)], seed=10)
    ids = tokens_of(cfg, 420, seed=9)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype, max_batch=2, max_seq=512, max_step_rows=64)
    room = eng.free_tokens
    from neuralfn_b200.serving import StepEntry
    out = [eng.step([StepEntry(0, ids[:150], range(150))], logits=True)[1]]      # longer than one pass
    out += [eng.step([StepEntry(0, [t], (0,))], logits=True)[1] for t in ids[150:]]
    assert worst(torch.cat(out), want) < TOL[dtype]
    assert room - eng.free_tokens == 448
    eng.release(0)
    assert eng.free_tokens == room
    eng.close()


def test_models_without_pages_count_tokens_all_the_same():
    from neuralfn_b200.serving import EngineError, StepEntry
    cfg, w = model([mingru(mlp=dense()), lightning()])
    eng = make_engine(cfg, w, max_batch=2, max_seq=512, kv_tokens=128)
    eng.step([StepEntry(0, tokens_of(cfg, 65, seed=1))])
    with pytest.raises(EngineError, match="pool is full"):
        eng.step([StepEntry(1, tokens_of(cfg, 1, seed=1))])
    eng.release(0)
    assert eng.free_tokens == 128
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


def test_fork_copies_pages_histories_and_states():
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
