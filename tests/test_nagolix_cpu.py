"""What of the Nagolix design needs no GPU: the plain statement is sensitive to every mechanism's mistakes at the tests'
tolerances, the safetensors reader, the registry, and the bookkeeping of batches, slots and the trace runner."""
import copy
import json
import struct

import numpy as np
import pytest

import nagolix_models as nm
import nagolix_plain as plain


def _logits(cfg, w, toks):
    return plain.forward(cfg, w, toks)


@pytest.fixture(scope="module", params=list(nm.SHARP.values()))
def model(request):
    cfg, buckets = nm.MODELS["mix"]
    w = nm.weights(cfg, 1, buckets, request.param)
    toks = nm.tokens(60, cfg, 2)
    return cfg, w, toks, _logits(cfg, w, toks)


@pytest.mark.parametrize("layer,where,change,first_seen", [
    (0, ("mask", "size"), 1, 9), (0, ("mask", "size"), -1, 8), (1, ("mask", "size"), 1, 14), (1, ("mask", "size"), -1, 13),
    (1, ("mask", "keep_first"), 1, 14), (1, ("mask", "keep_first"), -1, 13), (2, ("mask", "size"), -1, 20), (1, ("bias_max",), 8, 10),
])
def test_a_wrong_constant_shows(model, layer, where, change, first_seen):
    """One token more or less in a window, one kept token more or less, another last bucket: the logits differ by more than
    the serving tolerance somewhere, and not at all before the first position that can tell."""
    cfg, w, toks, right = model
    bad = copy.deepcopy(cfg)
    d = bad["layers"][layer]["mixer"]
    for k in where[:-1]:
        d = d[k]
    d[where[-1]] += change
    e = nm.error(_logits(bad, w, toks), right)
    assert e.max() > 2 * nm.TOLERANCE[nm.AUTO]
    assert e[:first_seen].max() == 0 and e[first_seen] > 50 * nm.TOLERANCE[nm.F32], e[first_seen - 1:first_seen + 2]


@pytest.mark.parametrize("zero", ["l1.mix.rel", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l0.mix.g", "l1.mix.g", "pos", "l0.norm1", "l0.norm2", "final.norm"])
def test_a_mechanism_that_is_left_out_shows(model, zero):
    cfg, w, toks, right = model
    bad = dict(w)
    bad[zero] = np.zeros_like(w[zero])
    assert nm.error(_logits(cfg, bad, toks), right).max() > nm.TOLERANCE[nm.AUTO]


def test_a_layer_that_makes_its_own_latents_instead_of_reading_them_shows(model):
    cfg, w, toks, right = model
    bad = copy.deepcopy(cfg)
    del bad["layers"][2]["mixer"]["kv_from"]
    w2 = dict(w, **{"l2.mix.dkv": w["l0.mix.dkv"], "l2.mix.dkv.norm": w["l0.mix.dkv.norm"]})
    assert nm.error(_logits(bad, w2, toks), right).max() > 2 * nm.TOLERANCE[nm.AUTO]


@pytest.mark.parametrize("name", list(nm.MODELS))
def test_rounding_products_to_bfloat16_stays_within_the_serving_tolerance(name):
    cfg, buckets = nm.MODELS[name]
    w = nm.weights(cfg, 11, buckets, nm.SHARP[nm.AUTO])
    toks = nm.tokens(190, cfg, 6)
    e = nm.error(plain.forward(cfg, w, toks, cast=plain.bf16_round), plain.forward(cfg, w, toks))
    assert 1e-3 < np.median(e) and e.max() < nm.TOLERANCE[nm.AUTO]


def test_distance_buckets():
    got = [plain.distance_bucket(n, 8, 64) for n in range(70)]
    assert got[:4] == [0, 1, 2, 3]
    # h = 4, ratio 16, four buckets: powers of two are the borders
    assert [got.index(b) for b in range(4, 8)] == [4, 8, 16, 32] and got[-1] == 7
    assert all(b >= a for a, b in zip(got, got[1:]))
    assert [plain.distance_bucket(n, 5, 9) for n in (1, 5, 8, 9, 10)] == [1, 3, 4, 4, 4]


def test_clamped_unit():
    y = plain.clamped_glu(np.array([-9.0, 0.0, 9.0]), np.array([9.0, -9.0, 9.0]), 2.0)
    s = plain.sigmoid
    assert np.allclose(y, [-9 * s(-9 * 1.702) * 3, 0.0, 2 * s(3.404) * 3])


def test_safetensors_reader(tmp_path):
    from llama_rust_b200.safetensors import SafetensorsError, SafetensorsFile
    a, b = np.arange(6, dtype=np.float32), np.array([1.5, -2.0], np.float32)
    head = {"__metadata__": {"k": "v"}, "a": dict(dtype="F32", shape=[2, 3], data_offsets=[0, 24]), "b": dict(dtype="BF16", shape=[2], data_offsets=[24, 28])}

    def put(head, data):
        h = json.dumps(head).encode()
        p = tmp_path / "m.safetensors"
        p.write_bytes(struct.pack("<Q", len(h)) + h + data)
        return p
    data = a.tobytes() + plain.f32_to_bf16(b).tobytes()
    f = SafetensorsFile(put(head, data))
    assert sorted(f.names()) == ["a", "b"] and f.shape("a") == (2, 3) and f.dtype("b") == "BF16" and "c" not in f
    assert np.array_equal(f.f32("a"), a.reshape(2, 3)) and np.array_equal(f.f32("b"), b)
    with pytest.raises(SafetensorsError):
        f.raw("c")
    for bad in (dict(head, a=dict(dtype="F32", shape=[2, 3], data_offsets=[0, 20])), dict(head, b=dict(dtype="BF16", shape=[2], data_offsets=[26, 30])),
                dict(head, a=dict(dtype="X9", shape=[2, 3], data_offsets=[0, 24])), [1]):
        with pytest.raises(SafetensorsError):
            SafetensorsFile(put(bad, data))
    p = tmp_path / "short"
    p.write_bytes(struct.pack("<Q", 1000) + b"{}")
    with pytest.raises(SafetensorsError):
        SafetensorsFile(p)


def test_registry_names_what_it_knows(tmp_path):
    from llama_rust_b200 import models
    assert {"Nagolix", "llama"} <= set(models.architectures())
    (tmp_path / "config.json").write_text('{"architecture": "Unheard"}')
    with pytest.raises(ValueError, match="Unheard"):
        models.load(None, tmp_path)


class _Recorder:
    """Stands for the executor: remembers the stacked matrices the loader uploads."""

    def __init__(self):
        self.mats = []

    def upload(self, dtype, rows, cols, packed):
        self.mats.append((dtype, rows, cols, np.array(packed)))
        return self.mats[-1]


@pytest.mark.parametrize("name", list(nm.MODELS))
def test_loader_stacks_and_checks(tmp_path, monkeypatch, name):
    from llama_rust_b200 import models
    from llama_rust_b200.models import nagolix
    from llama_rust_b200.safetensors import SafetensorsError
    cfg, buckets = nm.MODELS[name]
    w = nm.weights(cfg, 3, buckets)
    folder = nm.write(tmp_path / "m", cfg, w)
    seen = {}
    monkeypatch.setattr(nagolix, "DecoderSession", lambda ex, c, embd, layers, norm, **kw: seen.update(c=c, layers=layers, norm=norm, kw=kw) or "session")
    assert models.load(_Recorder(), folder, n_seq=3) == "session"
    assert seen["c"]["n_ctx"] == cfg["max_positions"] and seen["kw"]["n_seq"] == 3
    for i, (L, D) in enumerate(zip(cfg["layers"], seen["layers"])):
        m, d = L["mixer"], D["mixer"]
        parts = ["q", "k", "v", "g"] if L["type"] == "attention" else ["q"] + ([] if "kv_from" in m else ["dkv"]) + ["g"]
        want = np.concatenate([plain.f32_to_bf16(w[f"l{i}.mix.{p}"]).reshape(-1) for p in parts])
        assert np.array_equal(d["in"][3].view(np.uint16), want)
        assert (d["n_head"], d["dim"], d["vdim"], d["window"]) == (m["heads"], m["dim"], m["vdim"], m["mask"]["size"])
        assert d.get("keep_first", 0) == m["mask"].get("keep_first", 0) and d.get("kv_from", -1) == m.get("kv_from", -1)
        assert (D["mlp"] is None) == (L["mlp"] is None)
        assert np.allclose(D["mixer_norm"], 1 + w[f"l{i}.norm1"])
    bad = dict(w)
    bad["l0.mix.o"] = bad["l0.mix.o"][:-1]
    with pytest.raises(SafetensorsError, match="l0.mix.o"):
        models.load(_Recorder(), nm.write(tmp_path / "bad", cfg, bad))
    bad = dict(w)
    del bad["final.norm"]
    with pytest.raises(SafetensorsError, match="final.norm"):
        models.load(_Recorder(), nm.write(tmp_path / "bad2", cfg, bad))
    for key, value, text in (("type", "unheard", "unheard"), ("mlp", dict(kind="sparse", ff=8, limit=1.0), "sparse")):
        c = copy.deepcopy(cfg)
        c["layers"][0][key] = value
        with pytest.raises(ValueError, match=text):
            models.load(_Recorder(), nm.write(tmp_path / "bad3", c, w))


def _fake_session(n_seq, cap):
    """A Session whose batches are answered on the host: the logits of a row are (sequence, position, token)."""
    from llama_rust_b200.executor import Session

    class Fake(Session):
        max_batch = cap

        def __init__(self):
            self.n_seq, self.n_vocab, self._h = n_seq, 3, None
            self.pos, self.sizes = [0] * n_seq, []

        def batch_rows(self, groups, want):
            rows = []
            for q, t in groups:
                rows += [(q, self.pos[q] + i, v) for i, v in enumerate(t)]
                self.pos[q] += len(t)
            assert len(rows) <= self.max_batch and len({q for q, _ in groups}) == len(groups)
            self.sizes.append(len(rows))
            return np.array([rows[i] for i in want], np.float32).reshape(len(want), 3)

        def seq_reset(self, q):
            self.pos[q] = 0
    return Fake()


def test_forward_cuts_long_groups_and_keeps_the_order_of_the_wanted_rows():
    s = _fake_session(3, 10)
    groups = [(2, list(range(100, 117))), (0, [5]), (1, list(range(200, 212)))]
    want = [[16, 0, 9, 10], [0], [11, 3]]
    got = s.forward(groups, want)
    expect = [(2, 16, 116), (2, 0, 100), (2, 9, 109), (2, 10, 110), (0, 0, 5), (1, 11, 211), (1, 3, 203)]
    assert got.tolist() == [list(map(float, e)) for e in expect]
    assert max(s.sizes) == 10 and sum(s.sizes) == 30
    assert s.forward([(0, [7])], [[]]).shape == (0, 3) and s.pos == [2, 12, 17]


def test_trace_runner_gives_slots_back(tmp_path):
    from llama_rust_b200.trace import TraceRunner
    s = _fake_session(2, 8)
    r = TraceRunner(s, str(tmp_path))
    r.step(dict(step=0, entries=[dict(id="a", tokens=[1, 2, 3], want=[2, 0])], end=[]))
    r.step(dict(step=1, entries=[dict(id="b", tokens=[4], want=[]), dict(id="a", tokens=[5], want=[0])], end=["a"]))
    r.step(dict(step=2, entries=[dict(id="c", tokens=[6, 7], want=[1])], end=["b", "c", "never seen"]))
    r.step(dict(step=3, entries=[dict(id="d", tokens=[8], want=[]), dict(id="e", tokens=[9], want=[])], end=[]))
    out = {n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 3) for n in (0, 1, 2)}
    assert not (tmp_path / "3.f32").exists()
    qa = out[0][0, 0]
    assert out[0].tolist() == [[qa, 2, 3], [qa, 0, 1]] and out[1].tolist() == [[qa, 3, 5]]
    assert out[2].tolist() == [[qa, 1, 7]]  # the freed sequence, from position 0
    with pytest.raises(RuntimeError):
        r.step(dict(step=4, entries=[dict(id="f", tokens=[1], want=[])], end=[]))
