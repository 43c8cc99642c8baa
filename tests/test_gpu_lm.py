"""Layered models end to end: the library's step function, scheduler, generation and programs against the plain
restatement, in both number formats and on configurations whose sizes differ everywhere they can."""
import ctypes as C
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

import lm_util
from lm_util import TOL, cut, error

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
LATENT = ["latent", "latent_odd", "latent_wide", "latent_full"]
STREAMS = ["streams", "streams_odd", "streams_wide", "streams_full"]
LOOPS = ["loops", "loops_odd", "loops_wide", "loops_full"]
NAMES = ["mixed", "odd", "wide", "plain"] + LATENT + STREAMS + LOOPS
DTYPES = [6, 0]                      # bfloat16, float32


@pytest.fixture
def load(pkg, torch_dev):
    made = []

    def f(folder, dtype, **kw):
        made.append(pkg.LanguageModel(folder, dtype, **kw))
        return made[-1]
    yield f
    for m in made:
        m.close()


def prompt(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def feed(m, seq, tokens, sizes):
    return np.concatenate([m.step([(seq, tokens[a:b], None)])[0] for a, b in cut(len(tokens), sizes)])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    t = prompt(cfg, 150)
    m = load(folder, dtype)
    s = m.open()
    assert error(feed(m, s, t, [150]), lm_util.reference(cfg, w, t)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 17], [16], [64, 5], [70, 2, 1, 1, 31], [33, 100]])
def test_portions(synth, tmp_path, load, name, dtype, sizes):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    t = prompt(cfg, 140)
    m = load(folder, dtype)
    assert error(feed(m, m.open(), t, sizes), lm_util.reference(cfg, w, t)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_first_tokens(synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m = load(folder, dtype)
    for n in (1, 2, 3):
        t = prompt(cfg, n, seed=n)
        for sizes in ([n], [1]):
            s = m.open()
            assert error(feed(m, s, t, sizes), lm_util.reference(cfg, w, t)) < TOL[dtype]
            m.end(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "latent", "latent_odd", "latent_wide", "streams", "streams_odd", "streams_full", *LOOPS])
def test_unequal_requests_in_one_batch_with_blocks_used_again(pkg, synth, tmp_path, load, name, dtype):
    """Random schedules over a pool that is too small for all requests together: requests come and go, pause,
    take portions beside single tokens, and sit on blocks and slots that others have used."""
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    r = np.random.default_rng(8)
    m = load(folder, dtype, max_tokens=512, max_sequences=4, max_step_rows=256)
    todo = [prompt(cfg, int(n), seed=50 + i) for i, n in enumerate(r.choice([1, 5, 16, 17, 48, 63, 64, 65, 100, 120], 14))]
    want, live, got = [lm_util.reference(cfg, w, t) for t in todo], {}, [[] for _ in todo]
    nxt = 0
    while nxt < len(todo) or live:
        while nxt < len(todo) and len(live) < 4:
            live[nxt] = [m.open(), 0]
            nxt += 1
        entries, who = [], []
        for i, (s, at) in live.items():
            k = min(int(r.choice([0, 1, 1, 1, 2, 7, 16, 40, 64])), len(todo[i]) - at)
            if k:
                entries.append((s, todo[i][at:at + k], None))
                who.append((i, k))
        if not entries:
            continue
        order = r.permutation(len(entries))
        out = m.step([entries[o] for o in order])
        for o, lg in zip(order, out):
            i, k = who[o]
            got[i].append(lg)
            live[i][1] += k
            if live[i][1] == len(todo[i]):
                m.end(live.pop(i)[0])
    for g, x in zip(got, want):
        assert error(np.concatenate(g), x) < TOL[dtype]
    lib = pkg.lib
    assert lib.cml_lm_blocks_free(m.h) == lib.cml_lm_blocks_total(m.h)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["wide", "latent", "latent_wide", "streams", "streams_wide", "loops", "loops_wide"])
def test_batch_does_not_change_a_request(synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m = load(folder, dtype, max_sequences=8)
    t = [prompt(cfg, 60, seed=i) for i in range(8)]
    alone = []
    for x in t:
        s = m.open()
        alone.append(np.concatenate([m.step([(s, x[:50], None)])[0]] + [m.step([(s, x[k:k + 1], None)])[0] for k in range(50, 60)]))
        m.end(s)
    seqs = [m.open() for _ in t]
    both = [[y] for y in m.step([(s, x[:50], None) for s, x in zip(seqs, t)])]
    for k in range(50, 60):
        for b, y in zip(both, m.step([(s, x[k:k + 1], None) for s, x in zip(seqs, t)])):
            b.append(y)
    for a, b in zip(alone, both):
        assert error(np.concatenate(b), a) < TOL[dtype] / 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "latent_odd", "streams", "streams_odd", "loops_windows"])
def test_long_decoding(pkg, synth, tmp_path, load, name, dtype):
    """Hundreds of decoded tokens, over many blocks; windows let blocks go on the way, so the sequence outgrows what
    the pool could hold of it at once."""
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    t = prompt(cfg, 420)
    m = load(folder, dtype, max_tokens=160, max_sequences=2)
    s = m.open()
    got = feed(m, s, t, [20] + [1] * 400)
    assert error(got, lm_util.reference(cfg, w, t)) < TOL[dtype]
    lib = pkg.lib
    assert lib.cml_lm_sequence_length(m.h, s) == 420 and lib.cml_lm_blocks_total(m.h) - lib.cml_lm_blocks_free(m.h) <= 9      # the longest window is 70, and up to 33 first tokens are kept


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["latent", "loops", "loops_full"])
def test_long_decoding_with_everything_in_sight(synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    t = prompt(cfg, 420)
    m = load(folder, dtype, max_tokens=432, max_sequences=2)
    assert error(feed(m, m.open(), t, [23] + [1] * 397), lm_util.reference(cfg, w, t)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_of_closed_sequences_start_over(synth, tmp_path, load, dtype):
    """A sequence in a slot that another one left in the middle of things finds no trace of it: states, rings, blocks."""
    cfg, w, folder = lm_util.build(synth, tmp_path, "loops")
    m = load(folder, dtype, max_tokens=128, max_sequences=1)
    for n, sizes in ((90, [90]), (1, [1]), (70, [1]), (2, [2]), (33, [2]), (3, [1, 2]), (128, [64])):
        t = prompt(cfg, n, seed=n)
        s = m.open()
        assert error(feed(m, s, t, sizes), lm_util.reference(cfg, w, t)) < TOL[dtype]
        m.end(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_shared_weights_and_a_missing_feed_forward(synth, tmp_path, load, dtype):
    """What config.json says is what runs: changing one thing in it moves the restatement by more than the tolerance."""
    cfg, w, folder = lm_util.build(synth, tmp_path, "mixed")
    t = prompt(cfg, 60)
    m = load(folder, dtype)
    got = feed(m, m.open(), t, [37, 1, 1, 21])
    assert error(got, lm_util.reference(cfg, w, t)) < TOL[dtype]
    for change in (lambda c: c["layers"].pop(2), lambda c: c["layers"][0]["mixer"]["mask"].update(size=18), lambda c: c["norm"].update(eps=1e-1),
                   lambda c: c["layers"][3]["mixer"]["q_temp"].update(every=49), lambda c: c["layers"][1]["mixer"]["q_temp"].update(coef=0.8)):
        other = json.loads(json.dumps(cfg))
        change(other)
        if len(other["layers"]) == 3:
            w2 = {k.replace("l3.", "l2."): v for k, v in w.items()}
        else:
            w2 = w
        assert error(lm_util.reference(other, w2, t), lm_util.reference(cfg, w, t)) > 100 * TOL[0]


# ---- greedy decoding, scheduler, generation ----------------------------------------------------------------
def greedy_reference(cfg, w, tokens, steps):
    """(ids, margins): the restatement's own greedy continuation and the gap between its best two logits at each step."""
    m = lm_util.model(cfg, w)
    st = m.new_state()
    lg, out, gap = m.forward(tokens, st)[-1], [], []
    for _ in range(steps):
        top = np.sort(lg)[-2:]
        out.append(int(lg.argmax()))
        gap.append(float((top[1] - top[0]) / lg.std()))
        lg = m.forward([out[-1]], st)[-1]
    return out, gap


def same_until_a_tie(got, want, gap, eps=0.05):
    for g, x, d in zip(got, want, gap):
        if g != x:
            return d < eps
    return True


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_loop_on_the_device(synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m = load(folder, dtype)
    prompts = [prompt(cfg, n, seed=n) for n in (5, 40, 33)]
    refs = [greedy_reference(cfg, w, p, 41) for p in prompts]
    seqs = [m.open() for _ in prompts]
    first = [int(x[0]) for x in m.step([(s, p, [len(p) - 1]) for s, p in zip(seqs, prompts)], greedy=True)]
    ids, ms = m.decode_greedy(seqs, first, 40)
    assert ms > 0
    for k, (want, gap) in enumerate(refs):
        assert same_until_a_tie([first[k]] + ids[:, k].tolist(), want, gap)
    # the sequences stand behind what was decoded: one more step fits the replayed history
    hist = [np.concatenate([p, [f], ids[:-1, k]]) for k, (p, f) in enumerate(zip(prompts, first))]
    nxt = m.step([(s, [int(ids[-1, k])], None) for k, s in enumerate(seqs)])
    for k, h in enumerate(hist):
        assert error(nxt[k], lm_util.reference(cfg, w, np.concatenate([h, [ids[-1, k]]]))[-1:]) < TOL[dtype] * 1.5


def serve(pkg, m, prompts, lengths, batch, gen=None):
    lib = pkg.lib
    sc = lib.cml_serving_default_config()
    sc.max_batch_size = batch
    ctx = lib.cml_serving_create(C.byref(sc))
    ids, out, status = [], {}, {}
    for p, n in zip(prompts, lengths):
        p = np.ascontiguousarray(p, np.int32)
        ids.append(lib.cml_serving_submit(ctx, pkg.np_ptr(p), len(p), n))

    def done(r, _):
        q = r.contents
        out[q.request_id] = [q.generated_tokens[i] for i in range(q.num_generated)]
        status[q.request_id] = q.status
    cb = pkg.FinishFn(done)
    steps = lib.cml_serving_run_lm(ctx, m.h, C.byref(gen) if gen else None, 0, cb, None)
    lib.cml_serving_free(ctx)
    return steps, [out.get(i) for i in ids], [status.get(i) for i in ids]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["wide", "latent", "streams", "loops"])
def test_scheduler_serves_more_requests_than_fit(pkg, synth, tmp_path, load, name, dtype):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m = load(folder, dtype, max_tokens=256, max_sequences=3, max_step_rows=48)       # prompts are cut, requests wait
    lens, new = [70, 3, 120, 33, 1, 64, 90], [9, 30, 12, 1, 25, 20, 7]
    prompts = [prompt(cfg, n, seed=n) for n in lens]
    steps, got, _ = serve(pkg, m, prompts, new, 3)
    assert steps > 0 and [len(g) for g in got] == new
    for p, n, g in zip(prompts, new, got):
        want, gap = greedy_reference(cfg, w, p, n)
        assert same_until_a_tie(g, want, gap)
    assert pkg.lib.cml_lm_blocks_free(m.h) == pkg.lib.cml_lm_blocks_total(m.h)
    # a request the pool can never hold, and one with an unknown token, end with an error; the others run
    never = prompt(cfg, 1000 if name == "streams" else 250)                          # windows in every layer: only its block table bounds a sequence
    _, got, status = serve(pkg, m, [prompts[0], never, [1, cfg["vocab"]], prompts[1]], [4, 50, 3, 5], 2)
    assert [len(g) for g in got] == [4, 0, 0, 5] and status[1] == status[2] == 4


@pytest.mark.parametrize("name", ["plain", "latent", "streams", "loops"])
def test_generation_and_sampling(pkg, synth, tmp_path, load, name):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m, lib = load(folder, 0), pkg.lib
    p = np.ascontiguousarray(prompt(cfg, 21), np.int32)
    want, gap = greedy_reference(cfg, w, p, 12)

    def run(gen):
        res = lib.cml_lm_generate(m.h, pkg.np_ptr(p), len(p), C.byref(gen))
        ids = [res.contents.token_ids[i] for i in range(res.contents.num_tokens)]
        lib.cml_generation_result_free(C.cast(res, C.c_void_p))
        assert ids[:21] == p.tolist()
        return ids[21:]
    got = run(pkg.GenerationConfig(0.8, 0.9, 40, 12, -1, False))
    assert len(got) == 12 and same_until_a_tie(got, want, gap)
    stop = got[3]
    assert run(pkg.GenerationConfig(0.8, 0.9, 40, 12, stop, False)) == got[:got.index(stop) + 1]
    assert run(pkg.GenerationConfig(0.7, 0.9, 1, 12, -1, True)) == got                # one candidate: sampling is greedy
    libc = C.CDLL(None)
    draws = []
    for _ in range(2):
        libc.srand(5)
        draws.append(run(pkg.GenerationConfig(1.5, 1.0, 0, 12, -1, True)))
    assert draws[0] == draws[1] and draws[0] != got


def test_step_refusals_change_nothing(pkg, synth, tmp_path, load):
    cfg, w, folder = lm_util.build(synth, tmp_path, "wide")
    m = load(folder, 0, max_tokens=96, max_sequences=2, max_step_rows=64)
    t = prompt(cfg, 90)
    a = m.open()
    parts = [m.step([(a, t[:60], None)])[0]]
    b = m.open()
    bad = [[(a, [cfg["vocab"]], None)], [(a, [-1], None)], [(a, t[:3], [3])], [(a, [1], None), (a, [2], None)], [(7, [1], None)], [(b, t[:65], None)],
           [(b, t[:50], None)], [(a, [], None)]]
    for e in bad:
        with pytest.raises(pkg.CmlB200Error):
            m.step(e)
    with pytest.raises(pkg.CmlB200Error):
        m.open()
    m.end(b)
    with pytest.raises(pkg.CmlB200Error):
        m.step([(b, [1], None)])
    parts.append(m.step([(a, t[60:90], None)])[0])
    assert error(np.concatenate(parts), lm_util.reference(cfg, w, t)) < TOL[0]


@pytest.mark.parametrize("name", ["odd", "latent_odd", "streams_odd", "loops_odd"])
def test_wanted_places_only_and_many_of_them(synth, tmp_path, load, name):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    m = load(folder, 6, max_tokens=2048 if name == "loops_odd" else 1024)    # one of its layers sees everything, so no block is let go
    t = prompt(cfg, 600)
    want = lm_util.reference(cfg, w, t)
    s, u = m.open(), m.open()
    some, none, last = [0, 1, 63, 64, 299], [], [299]
    out = m.step([(s, t[:300], some), (u, t[:300], none)])
    assert len(out[1]) == 0 and error(out[0], want[some]) < TOL[6]
    out = m.step([(u, t[300:600], None), (s, t[300:600], last)])        # 301 rows of logits: more than one pass of the head
    assert error(out[0], want[300:]) < TOL[6] and error(out[1], want[599:]) < TOL[6]
    picks = m.step([(s, t[:290], None)], greedy=True)[0]
    assert len(picks) == 290


# ---- the registry's other class, and the programs ------------------------------------------------------------
def test_llama_behind_the_same_interface(pkg, tmp_path, load):
    import __graft_entry__ as entry
    import llama_util
    cfg, path = llama_util.TINY, tmp_path / "tiny.gguf"
    # the hyper-parameters the loader asks for
    meta = [(f"llama.{k}", 4, v) for k, v in (("block_count", cfg["layers"]), ("embedding_length", cfg["hidden"]), ("attention.head_count", cfg["heads"]),
                                              ("attention.head_count_kv", cfg["kv_heads"]), ("feed_forward_length", cfg["inter"]),
                                              ("context_length", cfg["max_seq"]))]
    store = llama_util.build(entry, np.random.default_rng(4), cfg, path, metadata=meta)
    ref = llama_util.OracleLlama(entry, cfg, store, rope_all_heads=1, mask_absolute=1)
    t = np.random.default_rng(6).integers(0, cfg["vocab"], 20)
    want = ref.forward(t)
    m = load(path, 0, max_tokens=96, max_sequences=3)
    assert pkg.lib.cml_lm_architecture(m.h) == b"llama" and m.vocab == cfg["vocab"]
    a, b = m.open(), m.open()
    x = m.step([(b, t[:9], [8])])[0]
    assert np.abs(x - want[8]).max() < 1e-2 * np.abs(want).max()
    y = m.step([(a, t[:13], [12]), (b, t[9:10], [0])])                  # a prompt beside a decoded token
    assert np.abs(y[0] - want[12]).max() < 1e-2 * np.abs(want).max() and np.abs(y[1] - want[9]).max() < 1e-2 * np.abs(want).max()
    z = m.step([(a, t[13:14], [0])])[0]                                 # the other sequence stands still meanwhile
    z2 = m.step([(b, t[10:11], [0])])[0]
    assert np.abs(z - want[13]).max() < 1e-2 * np.abs(want).max() and np.abs(z2 - want[10]).max() < 1e-2 * np.abs(want).max()
    m.end(a), m.end(b)
    _, got, _ = serve(pkg, m, [t[:7], t[:12]], [5, 8], 2)
    assert [len(g) for g in got] == [5, 8] and got[0][0] == int(want[6].argmax())


@pytest.mark.parametrize("name", ["mixed", "latent", "streams", "loops"])
def test_trace_run_replays(synth, tmp_path, torch_dev, name):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    t = {"a": prompt(cfg, 90, 1), "b": prompt(cfg, 50, 2), "c": prompt(cfg, 30, 3)}
    want = {k: lm_util.reference(cfg, w, v) for k, v in t.items()}
    plan = [[("a", 40), ("b", 1)], [("b", 48), ("a", 1)], [("a", 2)], [("b", 1), ("a", 20)], [("c", 30), ("a", 27)]]
    for dtype, code in (("bfloat16", 6), ("float32", 0)):
        out = tmp_path / dtype
        out.mkdir()
        at, lines, rows = dict.fromkeys(t, 0), [], []
        for n, step in enumerate(plan):
            entries, end, mine = [], [], []
            for k, c in step:
                wanted = list(range(c)) if n != 2 else []
                entries.append({"id": k, "tokens": t[k][at[k]:at[k] + c].tolist(), "want": wanted})
                mine += [want[k][at[k] + j] for j in wanted]
                at[k] += c
                if at[k] == len(t[k]):
                    end.append(k)
            lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
            rows.append(mine)
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:-1] == [f"done {n}" for n in range(len(plan))]
        assert not (out / "2.f32").exists()
        for n, mine in enumerate(rows):
            if mine:
                got = np.fromfile(out / f"{n}.f32", np.float32).reshape(len(mine), cfg["vocab"])
                assert error(got, np.array(mine)) < TOL[code]


@pytest.mark.parametrize("name", ["plain", "latent_odd", "streams_odd", "loops_odd"])
def test_cml_generate_program(pkg, synth, tmp_path, load, name):
    cfg, w, folder = lm_util.build(synth, tmp_path, name)
    prompts = [prompt(cfg, 9, 1).tolist(), prompt(cfg, 30, 2).tolist()]
    args = sum((["--tokens", ",".join(map(str, p))] for p in prompts), [])
    r = subprocess.run([str(ROOT / "bin" / "cml_generate"), "--model", str(folder), "--dtype", "float32", "--max-new", "11", *args],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    got = [[int(x) for x in line.split()] for line in r.stdout.splitlines()]
    _, want, _ = serve(pkg, load(folder, 0), prompts, [11, 11], 2)
    assert got == want
