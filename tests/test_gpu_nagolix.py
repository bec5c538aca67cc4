"""Layered decoders on the GPU (executor.DecoderSession, the Nagolix loader) against the plain float64 statement of the
design: each mechanism alone, prompts whole and in portions, token by token, in batches, over freed pages and slots, long
decoding, greedy generation through the engine, and the command lines.  Two kernel paths: f32 arithmetic throughout, and
the path that serves (bfloat16 products, binary16 attention operands for prompt chunks)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import nagolix_models as nm
import nagolix_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PATHS = [nm.F32, nm.AUTO]


@pytest.fixture(scope="module")
def ex():
    from llama_rust_b200 import Executor
    with Executor(0) as e:
        yield e


@pytest.fixture(scope="module")
def stock(tmp_path_factory):
    """name, path -> (config, weights, folder, plain logits of a token list)"""
    made, known = {}, {}

    def get(name, path=nm.F32):
        if (name, path) not in made:
            cfg, buckets = nm.MODELS[name]
            w = nm.weights(cfg, 11, buckets, nm.SHARP[path])
            made[name, path] = (cfg, w, nm.write(tmp_path_factory.mktemp("m"), cfg, w))
        cfg, w, folder = made[name, path]

        def logits(toks):
            key = (name, path, tuple(toks))
            if key not in known:
                known[key] = plain.forward(cfg, w, toks)
            return known[key]
        return cfg, w, folder, logits
    return get


def _open(ex, folder, path=nm.F32, **kw):
    from llama_rust_b200 import models
    ex.set_path(path)
    return models.load(ex, folder, **kw)


def _feed(s, seq, toks, cuts):
    """All logits of toks, fed in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(s.forward([(seq, toks[at:at + n])], [list(range(n))]))
        at, i = at + n, i + 1
    return np.concatenate(out)


def _close(got, want, path, what=""):
    e = nm.error(got, want)
    assert e.max() <= nm.TOLERANCE[path], f"{what}: position {int(e.argmax())} of {len(e)} off by {e.max():.2e}"


# ---- each mechanism alone ------------------------------------------------------------------------------------------
ALONE = {
    "attention": ([nm.attention(4, 2, 24, 40, 10, 3, 20)], 0),
    "attention, one head": ([nm.attention(1, 1, 64, 16, 7, 1, 9)], 0),
    "attention, many heads per key": ([nm.attention(20, 2, 16, 24, 12, 2, 30)], 0),
    "attention, nothing kept": ([nm.attention(2, 2, 32, 32, 8, 0, 20)], 0),
    "attention, itself only": ([nm.attention(2, 1, 32, 8, 1, 0, 20)], 0),
    "latent": ([nm.latent(5, 16, 24, 48, 10)], 0),
    "latent, itself only": ([nm.latent(3, 16, 8, 64, 1)], 0),
    "latent, many heads": ([nm.latent(19, 8, 16, 104, 14)], 0),
    "latents of an earlier layer": ([nm.latent(2, 16, 8, 40, 5), nm.latent(6, 24, 16, 40, 13, kv_from=0)], 0),
    "attention and feed-forward": ([nm.attention(2, 1, 24, 24, 9, 2, 20)], 200),
    "latent and feed-forward": ([nm.latent(2, 16, 16, 32, 9)], 40),
}


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(ALONE))
def test_one_mechanism(ex, tmp_path, name, path):
    layers, ff = ALONE[name]
    cfg = nm.config(80, 120, layers, ff, limit=0.8)
    w = nm.weights(cfg, 5, 10, nm.SHARP[path])
    toks, stream = nm.tokens(90, cfg, 4), []
    want = plain.forward(cfg, w, toks, stream)
    s = _open(ex, nm.write(tmp_path / "m", cfg, w), path)
    got = s.forward([(0, toks)], [list(range(len(toks)))])
    x = s.residual(len(toks))
    assert np.abs(x - stream[-1]).max() <= nm.TOLERANCE[path] * np.abs(stream[-1]).max()
    _close(got, want, path, name)
    s.reset()
    _close(_feed(s, 0, toks, [20, 1]), want, path, name + ", decoded")
    s.free()


def test_residual_stream_layer_by_layer(ex, stock, tmp_path):
    """The first k layers of a model as models of their own: the residual stream after each layer."""
    cfg, w, _, _ = stock("mix")
    toks, stream = nm.tokens(50, cfg, 8), []
    plain.forward(cfg, w, toks, stream)
    for k in range(1, len(cfg["layers"]) + 1):
        sub = dict(cfg, layers=cfg["layers"][:k])
        sw = {n: a for n, a in w.items() if not n.startswith("l") or int(n[1:n.index(".")]) < k}
        s = _open(ex, nm.write(tmp_path / str(k), sub, sw), nm.F32)
        s.forward([(0, toks)], [[]])
        assert np.abs(s.residual(len(toks)) - stream[k - 1]).max() <= 1e-4 * np.abs(stream[k - 1]).max(), k
        s.free()


# ---- prompts, portions, decoding ---------------------------------------------------------------------------------------
CUTS = {"whole": [10 ** 6], "one by one": [1], "twos": [2], "sevens": [7], "sixteens": [16], "37": [37], "changing": [5, 64, 1, 1, 2, 90, 3, 17, 1, 40],
        "most, then one by one": [140, 1]}


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(nm.MODELS))
def test_portions(ex, stock, name, path):
    """Every way of cutting a prompt gives the plain logits at every position: windows, kept tokens and page borders (blocks
    of five positions) fall inside, before and behind the cuts."""
    cfg, _, folder, logits = stock(name, path)
    toks = nm.tokens(190, cfg, 6)
    want = logits(toks)
    s = _open(ex, folder, path, n_seq=2, block_tokens=5)
    for cut, sizes in CUTS.items():
        s.seq_reset(1)
        _close(_feed(s, 1, toks, sizes), want, path, f"{name}, {cut}")
    s.free()


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_f32_results_do_not_depend_on_the_cut(ex, stock, name):
    """With f32 arithmetic a position's logits have the same bits however its prompt was cut."""
    cfg, _, folder, _ = stock(name)
    toks = nm.tokens(80, cfg, 9)
    s = _open(ex, folder, nm.F32)
    ref = _feed(s, 0, toks, [10 ** 6])
    for sizes in ([1], [2], [9], [33, 1]):
        s.reset()
        assert np.array_equal(_feed(s, 0, toks, sizes).view(np.uint32), ref.view(np.uint32)), sizes
    s.free()


@pytest.mark.parametrize("n", [1, 2, 3])
def test_the_first_tokens(ex, stock, n):
    for name in nm.MODELS:
        for path in PATHS:
            cfg, _, folder, logits = stock(name, path)
            toks = nm.tokens(n, cfg, 30 + n)
            s = _open(ex, folder, path)
            _close(_feed(s, 0, toks, [n]), logits(toks), path, name)
            s.free()


@pytest.mark.parametrize("path", PATHS)
def test_long_decoding(ex, stock, path):
    """Several windows' worth of tokens decoded one by one behind a short prompt."""
    cfg, _, folder, logits = stock("groups", path)
    toks = nm.tokens(260, cfg, 12)
    s = _open(ex, folder, path, block_tokens=16)
    _close(_feed(s, 0, toks, [8, 1]), logits(toks), path)
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_prompt_longer_than_a_batch(ex, stock, path):
    cfg, _, folder, logits = stock("tiles", path)
    toks = nm.tokens(600, cfg, 13)
    s = _open(ex, folder, path)
    assert s.max_batch == 512
    _close(_feed(s, 0, toks, [10 ** 6]), logits(toks), path)
    s.free()


def _one_key_model(heads_cfg, key_at, cfg_tokens):
    """A one-layer attention model in which the token id 1 at any position draws all attention it can get: embeddings are
    zero but for a marker direction, keys answer to it, and its value is large."""
    cfg = nm.config(64, 40, [heads_cfg], 0, scale=1.0)
    w = nm.weights(cfg, 3, 8, sharp=1.0)
    w["pos"] = w["pos"] * 0
    e = w["embed"] * 0.25
    e[:, 0] = 0
    e[1, 0] = 4.0                          # the marker
    w["embed"] = e
    m = heads_cfg["mixer"]
    G, d = m["kv_heads"], m["dim"]
    k = w["l0.mix.k"] * 0.05
    k[::d, 0] = 8.0                        # first component of every key head: the marker
    w["l0.mix.k"] = k
    q = w["l0.mix.q"] * 0.05
    w["l0.mix.q"], w["l0.mix.q.b"] = q, w["l0.mix.q.b"] * 0
    w["l0.mix.q.b"][::d] = 8.0             # every query asks for it
    w["l0.mix.k.b"] = w["l0.mix.k.b"] * 0
    w["l0.mix.rel"] = w["l0.mix.rel"] * 0.1
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = np.full_like(w["l0.mix.q.norm"], 2.0), np.ones_like(w["l0.mix.k.norm"])
    rng = np.random.default_rng(0)
    toks = (2 + rng.integers(0, 38, cfg_tokens)).tolist()
    toks[key_at] = 1
    return cfg, {n: plain.bf16_to_f64(plain.f32_to_bf16(a).tobytes()).reshape(a.shape) for n, a in w.items()}, toks


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("key_at,window,keep", [(40, 50, 0), (0, 30, 1), (3, 30, 4), (4, 30, 4), (47, 64, 2), (48, 64, 2), (63, 17, 0), (64, 16, 3)])
def test_one_key_among_hundreds(ex, tmp_path, key_at, window, keep, path):
    """One key outweighs all others: the positions that see it and the first that does not -- window - 1 and window tokens
    further on, or the kept first tokens for ever -- differ at once, in prompts and in decoding, at page borders (blocks of
    sixteen) and inside."""
    cfg, w, toks = _one_key_model(nm.attention(4, 2, 16, 24, window, keep, 24), key_at, 200)
    want = plain.forward(cfg, w, toks)
    # in the plain statement itself, the key's appearance and disappearance stand out
    drop = key_at + window
    without = list(toks)
    without[key_at] = 2
    gap = nm.error(plain.forward(cfg, w, without), want)
    assert gap[key_at:drop].min() > 0.1 and (gap[drop:].min() > 0.1 if key_at < keep else gap[drop:].max() < 1e-9)
    s = _open(ex, nm.write(tmp_path / "m", cfg, w), path, block_tokens=16)
    for sizes in ([200], [drop - 1, 1], [key_at + 1, 1], [17], [drop, 100]):
        s.reset()
        _close(_feed(s, 0, toks, sizes), want, path, str(sizes))
    s.free()


# ---- batches, slots, pages ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["mix", "tiles"])
def test_batches_of_unequal_requests(ex, stock, name, path):
    """Requests of different lengths interleaved in ragged batches -- long prompts beside single tokens -- against the plain
    logits of each alone."""
    cfg, _, folder, logits = stock(name, path)
    reqs = [nm.tokens(n, cfg, 40 + n) for n in (150, 3, 77, 41)]
    s = _open(ex, folder, path, n_seq=5, block_tokens=4)
    got, at = [[] for _ in reqs], [0] * len(reqs)
    slots, rng = [3, 0, 4, 1], np.random.default_rng(2)
    while any(a < len(r) for a, r in zip(at, reqs)):
        live = [i for i in range(len(reqs)) if at[i] < len(reqs[i]) and rng.random() < 0.8]
        if not live:
            continue
        rng.shuffle(live)
        take = {i: min(int(rng.choice([1, 2, 5, 19, 64])), len(reqs[i]) - at[i]) for i in live}
        out = s.forward([(slots[i], reqs[i][at[i]:at[i] + take[i]]) for i in live], [list(range(take[i])) for i in live])
        k = 0
        for i in live:
            got[i].append(out[k:k + take[i]])
            k += take[i]
            at[i] += take[i]
    for i, r in enumerate(reqs):
        _close(np.concatenate(got[i]), logits(r), path, f"request {i}")
    s.free()


def test_f32_rows_do_not_depend_on_their_batch(ex, stock):
    cfg, _, folder, _ = stock("mix")
    a, b = nm.tokens(40, cfg, 50), nm.tokens(23, cfg, 51)
    s = _open(ex, folder, nm.F32, n_seq=2)
    alone = [_feed(s, q, t, [10 ** 6]) for q, t in ((0, a), (1, b))]
    s.reset()
    both = s.forward([(1, b), (0, a)], [list(range(23)), list(range(40))])
    assert np.array_equal(both[:23].view(np.uint32), alone[1].view(np.uint32)) and np.array_equal(both[23:].view(np.uint32), alone[0].view(np.uint32))
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_pages_and_slots_that_are_used_again(ex, stock, path):
    """A pool that holds one long request: what earlier requests left in pages and slots must not be seen."""
    cfg, _, folder, logits = stock("mix", path)
    s = _open(ex, folder, path, n_seq=3, kv_blocks=30, block_tokens=4)  # 120 positions
    for rnd, (slot, n) in enumerate([(0, 110), (2, 97), (1, 120), (0, 30)]):
        toks = nm.tokens(n, cfg, 60 + rnd)
        _close(_feed(s, slot, toks, [50, 1, 1, 30]), logits(toks), path, f"use {rnd}")
        if rnd < 3:
            s.seq_reset(slot)
    other = nm.tokens(60, cfg, 70)  # beside the last one, whose pages stay
    _close(_feed(s, 2, other, [33, 2]), logits(other), path)
    from llama_rust_b200 import NativeCudaError
    with pytest.raises(NativeCudaError) as e:
        s.forward([(1, nm.tokens(60, cfg, 71))], [[]])
    assert e.value.code == 7
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_truncated_prompts_are_read_on(ex, stock, path):
    cfg, _, folder, logits = stock("mix", path)
    a = nm.tokens(70, cfg, 80)
    b = a[:33] + nm.tokens(30, cfg, 81)
    s = _open(ex, folder, path, block_tokens=8)
    s.forward([(0, a)], [[]])
    _close(s.prompt(b)[None], logits(b)[-1:], path)
    assert s.position == len(b)
    s.free()


# ---- generation ----------------------------------------------------------------------------------------------------------
def _greedy(logits, prompt, n):
    """The plain continuation, and how far each token's logit lies above the next."""
    toks, margin = list(prompt), []
    for _ in range(n):
        row = logits(toks)[-1]
        top = np.sort(row)[-2:]
        margin.append(float(top[1] - top[0]))
        toks.append(int(row.argmax()))
    return toks[len(prompt):], margin


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_greedy_decode_of_one_sequence(ex, stock, name):
    """session.decode: its steps replay one captured graph."""
    cfg, _, folder, logits = stock(name)
    prompt = nm.tokens(21, cfg, 90)
    want, margin = _greedy(logits, prompt, 40)
    s = _open(ex, folder, nm.F32)
    s.prefill(prompt)
    ids, m = s.decode(40)
    sure = next((i for i, v in enumerate(margin) if v < 1e-3), 40)
    assert sure >= 20 and ids[:sure].tolist() == want[:sure]
    assert np.allclose(m[:sure], margin[:sure], atol=1e-3)
    s.free()


@pytest.mark.parametrize("kv_blocks,chunk", [(0, 0), (12, 9)])
def test_greedy_generation_through_the_engine(ex, stock, kv_blocks, chunk):
    """Four prompts over two slots, generated by the scheduler; with 12 blocks of four positions it has to preempt."""
    from llama_rust_b200 import Engine, EngineCfg
    cfg, _, folder, logits = stock("mix")
    prompts = [nm.tokens(n, cfg, 100 + n) for n in (5, 19, 2, 26)]
    s = _open(ex, folder, nm.F32, n_seq=2, kv_blocks=kv_blocks, block_tokens=4)
    eng = Engine(s, EngineCfg(max_seqs=2, prefill_chunk=chunk))
    ids = [eng.add(p, 15) for p in prompts]
    eng.run()
    assert kv_blocks == 0 or eng.stats.preempts > 0
    for p, i in zip(prompts, ids):
        want, margin = _greedy(logits, p, 15)
        sure = next((k for k, v in enumerate(margin) if v < 1e-3), 15)
        assert eng.take(i).generated[:sure] == want[:sure]
    s.free()


def test_engine_prompts_longer_than_a_batch(ex, stock):
    from llama_rust_b200 import Engine, EngineCfg
    cfg, _, folder, logits = stock("odd")
    prompts = [nm.tokens(n, cfg, 200 + n) for n in (530, 40)]
    s = _open(ex, folder, nm.F32, n_seq=2)
    eng = Engine(s, EngineCfg(max_seqs=2))
    ids = [eng.add(p, 3) for p in prompts]
    eng.run()
    for p, i in zip(prompts, ids):
        want, margin = _greedy(logits, p, 3)
        sure = next((k for k, v in enumerate(margin) if v < 1e-3), 3)
        assert eng.take(i).generated[:sure] == want[:sure]
    s.free()


# ---- command lines ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,path", [("float32", nm.F32), ("bfloat16", nm.AUTO)])
def test_trace_run(stock, tmp_path, dtype, path):
    cfg, _, folder, logits = stock("groups", path)
    a, b = nm.tokens(95, cfg, 7), nm.tokens(30, cfg, 8)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:60], want=[0, 59, 17])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[]), dict(id="a", tokens=a[60:62], want=[1])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[62:], want=[32])], end=["a"]),
             dict(step=3, entries=[dict(id="a", tokens=b, want=[29, 28])], end=["a", "b"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "130"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    la, lb = logits(a), logits(b)
    for n, rows in ((0, la[[0, 59, 17]]), (1, la[[61]]), (2, la[[94]]), (3, lb[[29, 28]])):
        got = np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert got.shape == rows.shape
        d = got - rows
        d = d - d.mean(-1, keepdims=True)
        assert np.sqrt((d * d).mean(-1)).max() <= nm.TOLERANCE[path] * la.std()


def test_generate_command(stock):
    cfg, _, folder, logits = stock("mix")
    prompts = [nm.tokens(6, cfg, 1), nm.tokens(11, cfg, 2)]
    r = subprocess.run([sys.executable, "-m", "llama_rust_b200.generate", "--model", folder, "--dtype", "float32", "--n", "8"] +
                       [x for p in prompts for x in ("--tokens", ",".join(map(str, p)))], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    lines = [json.loads(ln) for ln in r.stdout.strip().split("\n")]
    for p, ln in zip(prompts, lines):
        want, margin = _greedy(logits, p, 8)
        sure = next((k for k, v in enumerate(margin) if v < 1e-3), 8)
        assert ln["prompt"] == p and ln["generated"][:sure] == want[:sure]


# ---- refusals --------------------------------------------------------------------------------------------------------------
def test_a_model_the_kernels_cannot_run_is_refused(ex, stock, tmp_path):
    from llama_rust_b200 import NativeCudaError
    cfg, w, folder, _ = stock("mix")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][2]["mixer"]["kv_from"] = 3
    with pytest.raises(NativeCudaError, match="kv_from"):
        _open(ex, nm.write(tmp_path / "late", bad, w))
    s = _open(ex, folder)
    with pytest.raises(NativeCudaError, match="token id"):
        s.forward([(0, [cfg["vocab"]])], [[]])
    with pytest.raises(NativeCudaError, match="context"):
        s.forward([(0, [1] * 400), ], [[]]), s.forward([(0, [1] * 400)], [[]])
    with pytest.raises(NativeCudaError, match="wanted row"):
        s.batch_rows([(0, [1, 2])], [2])
    s.free()


def test_a_session_outlives_its_executor_as_a_dead_handle(stock):
    from llama_rust_b200 import Executor, models
    _, _, folder, _ = stock("odd")
    e = Executor(0)
    s = models.load(e, folder)
    s.forward([(0, [1, 2, 3])], [[2]])
    h = s._h
    e.close()
    from llama_rust_b200.executor import lib
    assert lib().llr_session_reset(h) != 0
    s.free()
