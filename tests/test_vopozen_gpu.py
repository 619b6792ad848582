"""Vopozen on the layer-list engine against the plain reference: every mechanism alone and together, whole prompts, token by token, cut prompts, mixed
batches, reused pages and slots, edges of chunks, windows and pages, what a state holds, greedy generation through the scheduler - in bf16 and
in 32-bit."""
import json

import pytest
import torch

import vopozen_oracle as oracle
from step_helpers import repeat_cuts, run_cuts, run_mixed, worst
from vopozen_cases import attention, boost_needle, dense, lasting_memory, latent, model, moe, tokens_of, wkv

pytestmark = pytest.mark.gpu

TOL = {"bfloat16": 0.03, "float32": 3e-5}      # root mean square over the vocabulary, relative to the logits' spread


def make_engine(cfg, weights, dtype="float32", **kw):
    from neuralfn_b200.models.vopozen import VopozenConfig, engine_config, pack_tensors
    from neuralfn_b200.serving import ResidentEngine
    c = VopozenConfig.from_dict(cfg, weights)
    kw.setdefault("max_batch", 4)
    kw.setdefault("max_seq", 1024)
    eng = ResidentEngine(engine_config(c, dtype=dtype, **kw))
    eng.load_named_tensors(pack_tensors(c, weights))
    return eng


def everything(**kw):
    return model([attention(heads=6, kv_heads=3, dim=40, rot=24, chunk=50, mlp=dense(72)), latent(window=37, mlp=moe()), wkv(heads=4, dim=24, mlp=moe(groups=None, shared=0)),
                  latent(heads=3, dim=40, vdim=24, window=90, kv_from=1, mlp=dense(40)), attention(chunk=130, mlp=moe(experts=6, top=1, groups=(3, 1))), wkv(heads=2, dim=48)],
                 width=96, vocab=203, mult=0.45, **kw)


def grid():
    return {
        "attention": model([attention()]),
        "chunks": model([attention(chunk=5), attention(chunk=33), attention(chunk=128)]),
        "chunk1": model([attention(chunk=1), attention(chunk=2)]),
        "rotate_all": model([attention(rot=32, base=77.5)]),
        "rotate_none": model([attention(rot=0)]),
        "rotate_two": model([attention(rot=2, chunk=70)]),
        "one_head": model([attention(heads=1, kv_heads=1, dim=16, rot=8, chunk=40)]),
        "odd_heads": model([attention(heads=5, kv_heads=5, dim=24, rot=6, chunk=90), attention(heads=6, kv_heads=1, dim=56, rot=50)]),
        "wide_heads": model([attention(heads=4, kv_heads=2, dim=160, rot=100, scale=0.08, chunk=75)]),
        "huge_head": model([attention(heads=2, kv_heads=1, dim=272, rot=150, scale=0.06, chunk=75)]),
        "many_groups": model([attention(heads=24, kv_heads=2, dim=32, chunk=80)]),
        "latent": model([latent()]),
        "latent_windows": model([latent(window=1), latent(window=5), latent(window=64), latent(window=65)]),
        "latent_shared": model([latent(window=9), latent(window=70, kv_from=0), latent(heads=2, dim=56, vdim=16, window=3, kv_from=0), latent(kv_from=0)]),
        "latent_one_head": model([latent(heads=1, dim=16, rot=2, vdim=16, rank=16, window=30)]),
        "latent_odd": model([latent(heads=7, dim=20, rot=10, vdim=36, rank=37, window=50)]),
        "latent_many_heads": model([latent(heads=20, dim=16, vdim=16, window=60), latent(heads=37, dim=16, vdim=32, kv_from=0)]),
        "latent_wide": model([latent(heads=3, dim=128, rot=64, vdim=128, rank=512, scale=0.08, window=100)]),
        "latent_wide_rotation": model([latent(heads=18, dim=72, rot=80, vdim=72, rank=200, scale=0.1, window=100)]),
        "latent_wider": model([latent(heads=2, dim=32, rot=16, vdim=272, rank=528, scale=0.2)]),
        "wkv": model([wkv()]),
        "wkv_one_head": model([wkv(heads=1, dim=16, rank=1)]),
        "wkv_64": model([wkv(heads=2, dim=64, rank=40), wkv(heads=3, dim=56, rank=16)]),
        "wkv_128": model([wkv(heads=2, dim=128), wkv(heads=1, dim=80)]),
        "wkv_wide": model([wkv(heads=2, dim=144)]),
        "wkv_wider": model([wkv(heads=1, dim=320)]),
        "dense": model([wkv(mlp=dense(56)), attention(chunk=40, mlp=dense(24))]),
        "experts": model([attention(chunk=40, mlp=moe())]),
        "experts_no_groups": model([latent(window=40, mlp=moe(groups=None, experts=5, top=2))]),
        "experts_one_group_kept": model([wkv(mlp=moe(experts=12, groups=(3, 1), top=4, ff=24, shared=0))]),
        "experts_single_groups": model([wkv(mlp=moe(experts=6, groups=(6, 2), top=2))]),
        "experts_all": model([wkv(mlp=moe(experts=3, groups=None, top=3, shared=100)), attention(chunk=30, mlp=moe(experts=1, groups=None, top=1, scale=0.6))]),
        "experts_many": model([attention(chunk=40, mlp=moe(experts=40, groups=(8, 3), top=6))], width=96),
        "constants": model([attention(scale=0.05, chunk=77), latent(scale=0.9, window=33), wkv()], eps=0.03, mult=1.3),
        "mult1": model([attention(chunk=64, mlp=dense()), wkv()], mult=1.0),
        "odd_sizes": model([attention(heads=3, kv_heads=3, dim=40, rot=18, chunk=50, mlp=moe(ff=72)), latent(heads=5, rank=24, window=50, mlp=dense(88)), wkv(heads=5, dim=40)], vocab=203, width=136),
        "all": everything(),
    }


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(grid()))
def test_mechanism_prompt_decode_and_portions(case, dtype):
    cfg, w = grid()[case]
    T = 150
    ids, gaps = tokens_of(cfg, T, seed=3), []
    want, _ = oracle.forward(cfg, w, ids, gaps=gaps)
    assert min(gaps, default=1.0) > 0.01                 # no close choices
    eng = make_engine(cfg, w, dtype)
    for cuts in ([T], [1] * T, repeat_cuts(T, [2]), repeat_cuts(T, [17, 1, 40, 3]), repeat_cuts(T, [16, 31]), [64, 64, 22], [63, 2, 85]):
        assert worst(run_cuts(eng, 1, ids, cuts), want) < TOL[dtype], cuts[:4]
    eng.close()


def needle_edges(layer, size, dtype, places_of, ends):
    """A key whose score towers over the others, exactly at and around an edge of what the last position sees."""
    cfg, w = model([layer], vocab=64)
    boost_needle(cfg, w, query=62, key=63)
    eng = make_engine(cfg, w, dtype)
    for end in ends:
        for place in sorted(p for p in places_of(end) if 0 <= p < end):
            ids = tokens_of(cfg, end + 1, seed=end, below=62)
            ids[end], ids[place] = 62, 63
            want, _ = oracle.forward(cfg, w, ids)
            for cuts in ([end + 1], [end, 1], [end - 1, 2], repeat_cuts(end + 1, [50])):
                assert worst(run_cuts(eng, 0, ids, cuts)[-1:], want[-1:]) < 2 * TOL[dtype], (end, place, cuts[:3])
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [2, 31, 64, 65, 130])
def test_chunk_edges_with_far_keys(size, dtype):
    """The first position of a query's chunk and the last of the one before; queries first, in the middle and last in their chunk."""
    def places(end):
        start = end // size * size
        return {start - 1, start, start + 1, end - 1, 0}
    k = 256 // size
    needle_edges(attention(heads=4, kv_heads=2, dim=32, rot=16, chunk=size, scale=0.45), size, dtype, places, {k * size, k * size - 1, k * size + size // 2, 257})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [1, 2, 31, 64, 65, 130])
def test_window_edges_with_far_keys(size, dtype):
    """Around the window's far edge, at places before, on and after page borders."""
    needle_edges(latent(heads=5, dim=32, rot=16, vdim=32, rank=64, window=size), size, dtype, lambda end: {end - d for d in (1, size - 1, size, size + 1)} | {0}, (210, 255, 256))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_reader_of_another_cache_looks_further_back(dtype):
    """The owner's window is narrower than the reader's: the pages stay as long as the reader needs them."""
    cfg, w = model([latent(window=3), latent(window=150, kv_from=0, dim=32, vdim=32)], vocab=64)
    for n in ("q", "uk", "uv"):
        w["l1.mix." + n] = (w["l1.mix." + n].float() * 1.5).to(torch.bfloat16)
    ids = tokens_of(cfg, 400, seed=8)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype, max_batch=2, max_seq=448, max_step_rows=128)
    for cuts in ([400], [100, 100] + [1] * 200, repeat_cuts(400, [31])):
        assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_the_state_holds_arrives_later(dtype):
    """One token is written, all others leave the state alone; it is read back at every kind of distance and cut."""
    cfg, w = model([wkv(heads=3, dim=32)], vocab=40)
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
def test_only_the_previous_token_counts(dtype):
    """Every input of the time mixing is the previous token's: the shift is right at portion and chunk borders and zero at the start."""
    cfg, w = model([wkv(heads=2, dim=32)], vocab=64)
    for s in "rkvgw":
        w[f"l0.mix.mu.{s}"].fill_(1.0)
    ids = tokens_of(cfg, 120, seed=2)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([120], [1] * 120, repeat_cuts(120, [2]), repeat_cuts(120, [16, 1, 17]), repeat_cuts(120, [33])):
        assert worst(run_cuts(eng, 0, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("w0", [5.0, -14.0, 1.5, "both"])
def test_extreme_decays(w0, dtype):
    """States that forget within a token, never, or both within one head."""
    cfg, w = model([wkv(dim=48), wkv(dim=64)])
    for i in range(2):
        w[f"l{i}.mix.w0"].fill_(0.0 if w0 == "both" else w0)
        if w0 == "both":
            w[f"l{i}.mix.w0"][::2], w[f"l{i}.mix.w0"][1::2] = 4.0, -12.0
    ids = tokens_of(cfg, 200, seed=11)
    want, _ = oracle.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype)
    for cuts in ([200], repeat_cuts(200, [40, 1, 17]), [150] + [1] * 50):
        assert worst(run_cuts(eng, 2, ids, cuts), want) < TOL[dtype], cuts[:3]
    eng.close()


def test_a_channel_that_forgets_at_once_and_then_remembers():
    """Decays that jump between tokens of one chunk: what came before the fast token is gone, what comes after it stays."""
    cfg, w = model([wkv(heads=2, dim=32, rank=1)], vocab=40)
    w["l0.mix.w1"] = (30 * torch.stack([torch.linalg.lstsq(w["embed"].double(), torch.where(torch.arange(40) < 3, 1.0, -1.0).double()[:, None]).solution[:, 0]])).to(torch.bfloat16)
    w["l0.mix.w2"].fill_(8.0)
    w["l0.mix.w0"].fill_(-4.0)                           # z = 4 for tokens 0 .. 2, -12 for the others
    w["l0.mix.mu.w"].zero_()
    ids = tokens_of(cfg, 200, seed=13)
    want, _ = oracle.forward(cfg, w, ids)
    for dtype in ("bfloat16", "float32"):
        eng = make_engine(cfg, w, dtype)
        for cuts in ([200], repeat_cuts(200, [40, 1, 17])):
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


def test_several_long_portions_share_or_split_an_expansion():
    """Portions of many requests in one step: their latents fill the expansion's rows more than once."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = model([latent(window=40, mlp=dense()), latent(kv_from=0)], vocab=64)
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
    """More rows than the fused decode steps and the eight-column products take at a time."""
    from neuralfn_b200.serving import StepEntry
    cfg, w = model([attention(chunk=20, mlp=moe()), latent(window=17), wkv(heads=8, dim=16, mlp=dense())], vocab=64, width=96)
    n = 75
    ids = [tokens_of(cfg, 12, seed=s) for s in range(n)]
    want = [oracle.forward(cfg, w, s)[0] for s in ids]
    eng = make_engine(cfg, w, dtype, max_batch=n, max_seq=64)
    got = [eng.step([StepEntry(s, [ids[s][t]], (0,)) for s in range(n)], logits=True)[1] for t in range(12)]
    for s in range(n):
        assert worst(torch.stack([g[s] for g in got]), want[s]) < TOL[dtype], s
    eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_pages_given_back(dtype):
    cfg, w = model([attention(chunk=90, mlp=dense()), latent(window=70), wkv(), latent(window=20, kv_from=1)], seed=10)
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
    assert room - low <= 90 + 2 * 64, "pages behind the chunk or window stay held"
    eng.release(0)
    assert eng.free_tokens == room
    eng.close()


def test_models_without_pages_count_tokens_all_the_same():
    from neuralfn_b200.serving import EngineError, StepEntry
    cfg, w = model([wkv(mlp=dense())])
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


def test_fork_copies_pages_previous_input_and_state():
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
    for y in cfg["layers"]:                      # the tensors' shapes say this
        y["mixer"].pop("rank_decay", None)
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
