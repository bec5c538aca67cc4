"""Mukunex on the GPU (recurrent mixers, rotated attention with a sink, mixers beside each other, norms on inputs) against the
plain float64 statement of the design: each mechanism alone, prompts whole and in portions, token by token, in batches, over
freed pages and slots, long decoding, greedy generation through the engine, and the command lines.  Two kernel paths: f32
arithmetic throughout, and the path that serves (bfloat16 products, binary16 attention operands for prompt chunks)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import mukunex_models as mm
import mukunex_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PATHS = [mm.F32, mm.AUTO]


@pytest.fixture(scope="module")
def ex():
    from llama_rust_b200 import Executor
    with Executor(0) as e:
        yield e


@pytest.fixture(scope="module")
def stock(tmp_path_factory):
    """name -> (config, weights, folder, plain logits of a token list)"""
    made, known = {}, {}

    def get(name):
        if name not in made:
            cfg = mm.MODELS[name]
            w = mm.weights(cfg, 11)
            made[name] = (cfg, w, mm.write(tmp_path_factory.mktemp("m"), cfg, w))
        cfg, w, folder = made[name]

        def logits(toks):
            key = (name, tuple(toks))
            if key not in known:
                known[key] = plain.forward(cfg, w, toks)
            return known[key]
        return cfg, w, folder, logits
    return get


def _open(ex, folder, path=mm.F32, n_ctx=700, **kw):
    from llama_rust_b200 import models
    ex.set_path(path)
    return models.load(ex, folder, n_ctx=n_ctx, **kw)


def _feed(s, seq, toks, cuts):
    """All logits of toks, fed in portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(s.forward([(seq, toks[at:at + n])], [list(range(n))]))
        at, i = at + n, i + 1
    return np.concatenate(out)


def _close(got, want, path, what=""):
    e = mm.error(got, want)
    assert e.max() <= mm.TOLERANCE[path], f"{what}: position {int(e.argmax())} of {len(e)} off by {e.max():.2e}"


# ---- each mechanism alone ------------------------------------------------------------------------------------------
R8, R32 = mm.rot(8, 1e4), mm.rot(32, 1e4, (4.0, 1.0, 4.0, 64))
ALONE = {
    "attention beside retention": ([mm.parallel((4, 2, 32, 40, R32, 0.2), (2, 16, 24, R8, [0.9, 0.999]))], 0),
    "one head each": ([mm.parallel((1, 1, 64, 16, R8, 0.125), (1, 8, 8, R8, [0.99]))], 0),
    "many query heads per key": ([mm.parallel((20, 2, 16, 24, R8, 0.25), (5, 16, 8, R8, [0.5, 0.9, 0.99, 0.999, 1.0]))], 0),
    "attention only": ([mm.parallel((4, 2, 32, 40, R32, 0.2), (2, 16, 24, R8, [0.9, 0.999]), (1.0, 0.0))], 0),
    "retention only": ([mm.parallel((4, 2, 32, 40, R32, 0.2), (2, 16, 24, R8, [0.9, 0.999]), (0.0, 1.0))], 0),
    "rows of odd lengths": ([mm.parallel((3, 1, 12, 7, mm.rot(2, 100.0), 0.3), (3, 7, 11, mm.rot(6, 1e4), [0.9, 0.99, 0.999]))], 0),
    "gated recurrence": ([mm.rglru(96, 4, 4)], 0),
    "gated recurrence, one block": ([mm.rglru(40, 1, 4)], 0),
    "gated recurrence, no memory in the convolution": ([mm.rglru(64, 2, 1)], 0),
    "gated recurrence, many taps": ([mm.rglru(48, 6, 9)], 0),
    "delta rule": ([mm.delta(4, 4, 32, 32, 4)], 0),
    "delta rule, shared keys": ([mm.delta(6, 2, 16, 40, 4)], 0),
    "delta rule, one head": ([mm.delta(1, 1, 64, 8, 2)], 0),
    "delta rule, no memory in the convolution": ([mm.delta(2, 1, 24, 16, 1)], 0),
    "delta rule, many taps, odd ranks": ([mm.delta(2, 2, 12, 20, 7, (5, 3))], 0),
    "delta rule and feed-forward": ([mm.delta(2, 1, 16, 16, 3)], 200),
}


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(ALONE))
def test_one_mechanism(ex, tmp_path, name, path):
    layers, ff = ALONE[name]
    cfg = mm.config(80, 120, layers, ff)
    w = mm.weights(cfg, 5)
    toks, stream = mm.tokens(90, cfg, 4), []
    want = plain.forward(cfg, w, toks, stream)
    s = _open(ex, mm.write(tmp_path / "m", cfg, w), path)
    got = s.forward([(0, toks)], [list(range(len(toks)))])
    x = s.residual(len(toks))
    assert np.abs(x - stream[-1]).max() <= mm.TOLERANCE[path] * np.abs(stream[-1]).max()
    _close(got, want, path, name)
    for cuts in ([20, 1], [2], [1]):
        s.reset()
        _close(_feed(s, 0, toks, cuts), want, path, f"{name}, {cuts}")
    s.free()


def test_residual_stream_layer_by_layer(ex, stock, tmp_path):
    """The first k layers of a model as models of their own: the residual stream after each layer."""
    cfg, w, _, _ = stock("mix")
    toks, stream = mm.tokens(50, cfg, 8), []
    plain.forward(cfg, w, toks, stream)
    for k in range(1, len(cfg["layers"]) + 1):
        sub = dict(cfg, layers=cfg["layers"][:k])
        sw = {n: a for n, a in w.items() if not n.startswith("l") or int(n[1:n.index(".")]) < k}
        s = _open(ex, mm.write(tmp_path / str(k), sub, sw), mm.F32)
        s.forward([(0, toks)], [[]])
        assert np.abs(s.residual(len(toks)) - stream[k - 1]).max() <= 2e-5 * np.abs(stream[k - 1]).max(), k
        s.free()


# ---- prompts, portions, decoding ---------------------------------------------------------------------------------------
CUTS = {"whole": [10 ** 6], "one by one": [1], "twos": [2], "sevens": [7], "sixteens": [16], "37": [37], "changing": [5, 64, 1, 1, 2, 90, 3, 17, 1, 40],
        "most, then one by one": [140, 1]}


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(mm.MODELS))
def test_portions(ex, stock, name, path):
    """Every way of cutting a prompt gives the plain logits at every position: page borders (blocks of five positions), the
    convolutions' reach and the scans' stages fall inside, before and behind the cuts."""
    cfg, _, folder, logits = stock(name)
    toks = mm.tokens(190, cfg, 6)
    want = logits(toks)
    s = _open(ex, folder, path, n_seq=2, block_tokens=5)
    for cut, sizes in CUTS.items():
        s.seq_reset(1)
        _close(_feed(s, 1, toks, sizes), want, path, f"{name}, {cut}")
    s.free()


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_f32_results_do_not_depend_on_the_cut(ex, stock, name):
    """With f32 arithmetic a position's logits are the same however its prompt was cut: the recurrences run token by token."""
    cfg, _, folder, _ = stock(name)
    toks = mm.tokens(80, cfg, 9)
    s = _open(ex, folder, mm.F32)
    ref = _feed(s, 0, toks, [10 ** 6])
    for sizes in ([1], [2], [9], [33, 1]):
        s.reset()
        assert mm.error(_feed(s, 0, toks, sizes), ref.astype(np.float64)).max() < 2e-6, sizes
    s.free()


@pytest.mark.parametrize("n", [1, 2, 3, 17])
def test_the_first_tokens(ex, stock, n):
    for name in mm.MODELS:
        for path in PATHS:
            cfg, _, folder, logits = stock(name)
            toks = mm.tokens(n, cfg, 30 + n)
            s = _open(ex, folder, path)
            _close(_feed(s, 0, toks, [n]), logits(toks), path, name)
            s.free()


@pytest.mark.parametrize("path", PATHS)
def test_long_decoding(ex, stock, path):
    cfg, _, folder, logits = stock("groups")
    toks = mm.tokens(400, cfg, 12)
    s = _open(ex, folder, path, block_tokens=16)
    _close(_feed(s, 0, toks, [3, 1]), logits(toks), path)
    s.free()


def test_states_that_hardly_fade(ex, tmp_path):
    """Decays next to 1 over a thousand positions: the recurrences' rounding must not add up."""
    cfg = mm.config(64, 60, [mm.rglru(96, 3, 4), mm.parallel((2, 1, 16, 16, R8, 0.25), (2, 16, 16, R8, [0.9999, 1.0])), mm.delta(2, 1, 16, 16, 4)], 0)
    w = mm.weights(cfg, 31)
    w["l0.mix.lam"] = mm.rounded(w["l0.mix.lam"] - 5.0)
    w["l2.mix.dt_bias"] = mm.rounded(w["l2.mix.dt_bias"] - 4.0)
    toks = mm.tokens(1100, cfg, 14)
    want = plain.forward(cfg, w, toks)
    s = _open(ex, mm.write(tmp_path / "m", cfg, w), mm.F32, n_ctx=1100)
    for sizes in ([1100], [1000, 1]):
        s.reset()
        e = mm.error(_feed(s, 0, toks, sizes), want)
        assert e.max() <= 2e-5, e.max()
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_prompt_longer_than_a_batch(ex, stock, path):
    cfg, _, folder, logits = stock("tiles")
    toks = mm.tokens(600, cfg, 13)
    s = _open(ex, folder, path)
    assert s.max_batch == 512
    _close(_feed(s, 0, toks, [10 ** 6]), logits(toks), path)
    s.free()


# ---- far tokens --------------------------------------------------------------------------------------------------------
def _one_key_model(left, key_at, n):
    """A one-layer model in which the token id 1 at any position draws all attention it can get: a marker direction of the
    embedding reaches the last pair of every key head -- which turns so slowly that the key is the same anywhere -- and all
    other tokens answer to it with their queries.  The retention beside it hardly speaks."""
    cfg = mm.config(64, 40, [mm.parallel(left, (1, 8, 8, R8, [0.9]), (1.0, 0.05))], 0)
    w = mm.weights(cfg, 3)
    e = w["embed"] * 0.3
    e[:, 0], e[:, 1] = 0.0, 3.0    # every token asks
    e[1, 0], e[1, 1] = 6.0, 0.0    # the marker answers
    w["embed"] = e
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    d, still = left[2], left[4]["dims"] // 2 - 1
    k, q = w["l0.mix.left.k"] * 0.05, w["l0.mix.left.q"] * 0.05
    k[still::d, 0] = 4.0
    q[still::d, 1] = 4.0 / left[5] / 8
    w["l0.mix.left.k"], w["l0.mix.left.q"] = k, q
    toks = (2 + np.random.default_rng(0).integers(0, 38, n)).tolist()
    toks[key_at] = 1
    return cfg, {name: mm.rounded(a) for name, a in w.items()}, toks


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("key_at", [0, 15, 16, 40, 63, 64, 100])
def test_one_key_among_hundreds(ex, tmp_path, key_at, path):
    """One key outweighs all others and the sink: every later position sees it, hundreds of tokens on, in prompts and in
    decoding, at page borders (blocks of sixteen), at the borders of the attention kernels' tiles and slices, and inside."""
    n = 420
    cfg, w, toks = _one_key_model((4, 2, 16, 24, mm.rot(16, 1e7), 0.25), key_at, n)
    want = plain.forward(cfg, w, toks)
    without = list(toks)
    without[key_at] = 2
    gap = mm.error(plain.forward(cfg, w, without), want)
    assert gap[key_at:].min() > 4 * mm.TOLERANCE[mm.AUTO] and (key_at == 0 or gap[:key_at].max() < 1e-9)
    s = _open(ex, mm.write(tmp_path / "m", cfg, w), path, block_tokens=16)
    for sizes in ([n], [key_at + 1, 1], [key_at or 1, 2], [17], [300, 20, 1]):
        s.reset()
        _close(_feed(s, 0, toks, sizes), want, path, str(sizes))
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_a_sink_that_outweighs_the_keys(ex, tmp_path, path):
    """Heads whose sink is far above every score give next to nothing, heads whose sink is far below are plain softmax heads; a
    large sink must not overflow."""
    cfg = mm.config(64, 50, [mm.parallel((4, 1, 32, 16, R8, 0.2), (1, 8, 8, R8, [0.9]), (2.0, 0.1))], 0)
    w = mm.weights(cfg, 21)
    w["l0.mix.left.sink"] = np.array([90.0, -90.0, 5.0, 0.0])
    toks = mm.tokens(150, cfg, 3)
    want = plain.forward(cfg, w, toks)
    s = _open(ex, mm.write(tmp_path / "m", cfg, w), path)
    for sizes in ([150], [70, 1]):
        s.reset()
        _close(_feed(s, 0, toks, sizes), want, path, str(sizes))
    s.free()


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("kind", ["retention", "gated recurrence", "delta rule"])
def test_states_remember(ex, tmp_path, kind, path):
    """A token at position 3 still shows 250 positions on: in the plain statement its replacement changes the logits by far more
    than the tolerance everywhere, and the session agrees however the tokens between were cut."""
    layer = {"retention": mm.parallel((1, 1, 8, 8, R8, 0.3), (2, 16, 16, mm.rot(2, 1e6), [1.0, 0.9999]), (0.01, 2.0)),
             "gated recurrence": mm.rglru(64, 2, 3), "delta rule": mm.delta(2, 2, 32, 16, 3)}[kind]
    cfg = mm.config(64, 40, [layer], 0)
    w = mm.weights(cfg, 8)
    p = "l0.mix."
    if kind == "retention":  # only the marker's value is large: the others hardly add to the state
        w["embed"][:, 0] = 0.0
        w["embed"][1] = 0.0
        w["embed"][1, 0] = 4.0
        w[p + "right.v"] = w[p + "right.v"] * 0.02
        w[p + "right.v"][:, 0] = 1.5
        w["embed"][2:, 1] = 3.0  # and every other token asks for the marker's key: no result is a small difference
        w[p + "right.q"][:, 1] = 1.0
        w[p + "right.k"][:, 0] = 1.0
    elif kind == "gated recurrence":  # states fade by 0.001 per token, and only the marker passes the input gate
        w[p + "lam"] = np.full_like(w[p + "lam"], -9.0)
        w["embed"][:, 0] = 0.0
        w["embed"][1] = 0.0
        w["embed"][1, 0] = 4.0
        w[p + "x"] = w[p + "x"] * 0.02
        w[p + "x"][:, 0] = 3.0
        w[p + "x.b"], w[p + "conv.b"] = w[p + "x.b"] * 0, w[p + "conv.b"] * 0
        w[p + "conv"][:, -1] = 1.0
    else:  # no fading, and only the marker writes
        w[p + "dt_bias"] = np.full_like(w[p + "dt_bias"], -12.0)
        w[p + "a2"] = w[p + "a2"] * 0.01
        w["embed"][:, 0] = -3.0
        w["embed"][1, 0] = 3.0
        w[p + "b"][:, 0] = 4.0
    w = {n: mm.rounded(a) for n, a in w.items()}
    toks = (2 + np.random.default_rng(1).integers(0, 38, 260)).tolist()
    toks[3] = 1
    want = plain.forward(cfg, w, toks)
    without = list(toks)
    without[3] = 2
    assert np.median(mm.error(plain.forward(cfg, w, without), want)[200:]) > 3 * mm.TOLERANCE[mm.AUTO]
    s = _open(ex, mm.write(tmp_path / "m", cfg, w), path)
    for sizes in ([260], [4, 1], [3, 2], [130, 129, 1]):
        s.reset()
        _close(_feed(s, 0, toks, sizes), want, path, f"{kind}, {sizes}")
    s.free()


# ---- batches, slots, pages ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["mix", "tiles", "odd"])
def test_batches_of_unequal_requests(ex, stock, name, path):
    """Requests of different lengths interleaved in ragged batches -- long prompts beside single tokens -- against the plain
    logits of each alone."""
    cfg, _, folder, logits = stock(name)
    reqs = [mm.tokens(n, cfg, 40 + n) for n in (150, 3, 77, 41)]
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
    a, b = mm.tokens(40, cfg, 50), mm.tokens(23, cfg, 51)
    s = _open(ex, folder, mm.F32, n_seq=2)
    alone = [_feed(s, q, t, [10 ** 6]) for q, t in ((0, a), (1, b))]
    s.reset()
    both = s.forward([(1, b), (0, a)], [list(range(23)), list(range(40))])
    assert mm.error(both[:23], alone[1].astype(np.float64)).max() < 2e-6 and mm.error(both[23:], alone[0].astype(np.float64)).max() < 2e-6
    s.free()


def test_a_long_prompt_beside_many_sequences(ex, stock):
    """More groups than the scans take by blocks: 70 sequences, one of them with a long portion."""
    cfg, _, folder, logits = stock("mix")
    reqs = [mm.tokens(40 if q == 33 else 3, cfg, 300 + q) for q in range(70)]
    s = _open(ex, folder, mm.F32, n_ctx=64, n_seq=70)
    for lo, hi in ((0, 2), (2, 40)):
        live = [q for q in range(70) if len(reqs[q]) > lo]
        out = s.forward([(q, reqs[q][lo:hi]) for q in live], [[len(reqs[q][lo:hi]) - 1] for q in live])
        for k, q in enumerate(live):
            _close(out[k:k + 1], logits(reqs[q][:hi])[-1:], mm.F32, f"sequence {q}")
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_pages_and_slots_that_are_used_again(ex, stock, path):
    """A pool that holds one long request: what earlier requests left in pages, slots and states must not be seen."""
    cfg, _, folder, logits = stock("mix")
    s = _open(ex, folder, path, n_seq=3, kv_blocks=30, block_tokens=4)  # 120 positions
    for rnd, (slot, n) in enumerate([(0, 110), (2, 97), (1, 120), (0, 30), (0, 1), (0, 40)]):
        toks = mm.tokens(n, cfg, 60 + rnd)
        _close(_feed(s, slot, toks, [50, 1, 1, 30]), logits(toks), path, f"use {rnd}")
        if rnd < 5:
            s.seq_reset(slot)
    other = mm.tokens(60, cfg, 70)  # beside the last one, whose pages stay
    _close(_feed(s, 2, other, [33, 2]), logits(other), path)
    from llama_rust_b200 import NativeCudaError
    with pytest.raises(NativeCudaError) as e:
        s.forward([(1, mm.tokens(60, cfg, 71))], [[]])
    assert e.value.code == 7
    # a batch that was refused has touched no state
    more = mm.tokens(5, cfg, 72)
    _close(_feed(s, 2, more, [5]), logits(other + more)[-5:], path)
    s.free()


@pytest.mark.parametrize("path", PATHS)
def test_prompts_that_share_a_beginning(ex, stock, path):
    """A recurrent state cannot be rewound: the session says so, and prompt reuse reads the prompt again or reads on."""
    from llama_rust_b200 import NativeCudaError
    cfg, _, folder, logits = stock("mix")
    a = mm.tokens(70, cfg, 80)
    b = a[:33] + mm.tokens(30, cfg, 81)
    s = _open(ex, folder, path, block_tokens=8)
    s.forward([(0, a)], [[]])
    with pytest.raises(NativeCudaError, match="rewound"):
        s.seq_truncate(0, 33)
    _close(s.prompt(b)[None], logits(b)[-1:], path)
    assert s.position == len(b)
    c = b + mm.tokens(7, cfg, 82)
    assert len(s.prompt_suffix(c)) == 7
    _close(s.prefill(c[len(b):], want_logits=True)[None], logits(c)[-1:], path)
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


def _same(got, want, margin):
    sure = next((k for k, v in enumerate(margin) if v < 1e-3), len(want))
    assert sure >= 2 and list(got[:sure]) == want[:sure]
    return sure


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_greedy_decode_of_one_sequence(ex, stock, name):
    """session.decode: its steps replay one captured graph; a second call goes on from the state the first one left."""
    cfg, _, folder, logits = stock(name)
    prompt = mm.tokens(21, cfg, 90)
    want, margin = _greedy(logits, prompt, 36)
    s = _open(ex, folder, mm.F32)
    s.prefill(prompt)
    first, m = s.decode(20)
    sure = _same(first.tolist() + s.decode(16)[0].tolist(), want, margin)
    assert np.allclose(m[:min(sure, 20)], margin[:min(sure, 20)], atol=1e-3)
    s.free()


@pytest.mark.parametrize("kv_blocks,chunk", [(0, 0), (12, 9)])
def test_greedy_generation_through_the_engine(ex, stock, kv_blocks, chunk):
    """Four prompts over two slots, generated by the scheduler; with 12 blocks of four positions it has to preempt."""
    from llama_rust_b200 import Engine, EngineCfg
    cfg, _, folder, logits = stock("mix")
    prompts = [mm.tokens(n, cfg, 100 + n) for n in (5, 19, 2, 26)]
    s = _open(ex, folder, mm.F32, n_ctx=64, n_seq=2, kv_blocks=kv_blocks, block_tokens=4)
    eng = Engine(s, EngineCfg(max_seqs=2, prefill_chunk=chunk))
    ids = [eng.add(p, 15) for p in prompts]
    eng.run()
    assert kv_blocks == 0 or eng.stats.preempts > 0
    for p, i in zip(prompts, ids):
        _same(eng.take(i).generated, *_greedy(logits, p, 15))
    s.free()


# ---- command lines ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,path", [("float32", mm.F32), ("bfloat16", mm.AUTO)])
def test_trace_run(stock, tmp_path, dtype, path):
    cfg, _, folder, logits = stock("groups")
    a, b = mm.tokens(95, cfg, 7), mm.tokens(30, cfg, 8)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:60], want=[0, 59, 17])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[]), dict(id="a", tokens=a[60:62], want=[1])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[62:], want=[32])], end=["a"]),
             dict(step=3, entries=[dict(id="a", tokens=b, want=[29, 28])], end=["a", "b"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "125"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    la, lb = logits(a), logits(b)
    for n, rows in ((0, la[[0, 59, 17]]), (1, la[[61]]), (2, la[[94]]), (3, lb[[29, 28]])):
        got = np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert got.shape == rows.shape
        d = got - rows
        d = d - d.mean(-1, keepdims=True)
        assert np.sqrt((d * d).mean(-1)).max() <= mm.TOLERANCE[path] * la.std()


def test_generate_command(stock):
    cfg, _, folder, logits = stock("odd")
    prompts = [mm.tokens(6, cfg, 1), mm.tokens(11, cfg, 2)]
    r = subprocess.run([sys.executable, "-m", "llama_rust_b200.generate", "--model", folder, "--dtype", "float32", "--n", "8"] +
                       [x for p in prompts for x in ("--tokens", ",".join(map(str, p)))], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    for p, ln in zip(prompts, map(json.loads, r.stdout.strip().split("\n"))):
        assert ln["prompt"] == p
        _same(ln["generated"], *_greedy(logits, p, 8))


# ---- refusals --------------------------------------------------------------------------------------------------------------
def test_a_model_the_kernels_cannot_run_is_refused(ex, tmp_path):
    from llama_rust_b200 import NativeCudaError
    cfg = mm.config(80, 40, [mm.delta(1, 1, 1100, 8, 2)], 0)
    with pytest.raises(NativeCudaError, match="head sizes"):
        _open(ex, mm.write(tmp_path / "long", cfg, mm.weights(cfg, 1)))
    cfg = mm.config(80, 40, [mm.parallel((2, 1, 16, 16, R8, 0.2), (2, 16, 16, R8, [0.9]))], 0)
    with pytest.raises(ValueError, match="1 decays for 2 heads"):
        _open(ex, mm.write(tmp_path / "decays", cfg, mm.weights(cfg, 1)))
