"""What of the Mukunex design needs no GPU: the plain statement against independent forms of its recurrences, its sensitivity to
every mechanism's mistakes at the tests' tolerances, the loader, and the bookkeeping of sessions that cannot rewind."""
import copy

import numpy as np
import pytest

import mukunex_models as mm
import mukunex_plain as plain


@pytest.fixture(scope="module")
def model():
    cfg = mm.MODELS["mix"]
    w = mm.weights(cfg, 1)
    toks = mm.tokens(90, cfg, 2)
    return cfg, w, toks, plain.forward(cfg, w, toks)


def test_retention_is_a_sum_over_the_past():
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((30, 2, n)) for n in (5, 5, 7))
    decay = np.array([0.5, 0.97])
    got = plain.retention_scan(q, k, v, decay)
    i, j = np.arange(30)[:, None], np.arange(30)[None, :]
    fade = np.where(j <= i, decay[:, None, None] ** np.maximum(i - j, 0), 0.0)
    assert np.allclose(got, np.einsum("hij,ihd,jhd,jhv->ihv", fade, q, k, v), atol=1e-10)


def test_delta_rule_replaces_what_a_key_held():
    """beta 1 and no fading: reading a unit key gives the value written last for it, whatever was there."""
    rng = np.random.default_rng(1)
    k = plain.unit(rng.standard_normal((1, 1, 6))) * np.ones((4, 1, 1))
    v = rng.standard_normal((4, 1, 3))
    one = np.ones((4, 1, 6))
    assert np.allclose(plain.delta_scan(k, k, v, one, np.ones((4, 1))), v, atol=1e-5)
    half = plain.delta_scan(k, k, v, one, np.full((4, 1), 0.5))
    assert np.allclose(half[1], 0.5 * v[1] + 0.25 * v[0], atol=1e-5)
    faded = plain.delta_scan(k, k, v, 0.5 * one, np.zeros((4, 1)))
    assert np.allclose(faded, 0.0)


def test_gated_scan_and_convolution():
    a, b = np.array([[0.5], [0.25], [1.0]]), np.array([[1.0], [2.0], [3.0]])
    assert plain.gated_scan(a, b).ravel().tolist() == [1.0, 2.25, 5.25]
    x = np.arange(1.0, 6.0)[:, None]
    assert plain.causal_conv(x, np.array([[100.0, 10.0, 1.0]])).ravel().tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]


def test_frequencies():
    r = mm.rot(16, 1e4, (4.0, 1.0, 4.0, 64))
    f, base = plain.frequencies(r), plain.frequencies(mm.rot(16, 1e4))
    wave = 2 * np.pi / base
    assert np.allclose(f[wave < 16], base[wave < 16]) and np.allclose(f[wave > 64], base[wave > 64] / 4)
    between = (wave >= 16) & (wave <= 64)
    assert (wave < 16).any() and between.any() and (wave > 64).any()
    assert ((f < base) & (f > base / 4))[between].all()
    from llama_rust_b200.models.mukunex import rotation
    for r in (r, mm.rot(6, 1e3), mm.rot(32, 5e5, (8.0, 0.5, 3.0, 100))):
        assert np.allclose(rotation(r), plain.frequencies(r), rtol=1e-14)


@pytest.mark.parametrize("layer,path,value", [
    (0, ("mixer", "kv_heads"), None), (1, ("mixer", "left", "scale"), 0.4), (1, ("mixer", "left", "rot", "scaling"), None), (1, ("mixer", "left", "rot", "dims"), 8),
    (1, ("mixer", "right", "rot", "base"), 1e3), (1, ("mixer", "right", "decay"), [0.9, 0.99, 0.99]), (1, ("mixer", "left_scale"), 1.0),
    (1, ("mixer", "right_scale"), 1.0), (4, ("mixer", "left", "rot", "dims"), 24), (4, ("mixer", "right", "decay"), [0.998, 0.75])])
def test_a_wrong_constant_shows(model, layer, path, value):
    cfg, w, toks, right = model
    if value is None and path[-1] == "kv_heads":
        bad = dict(w)  # the other way of sharing query / key heads: heads h, h + kv_heads, ... share one
        order = [0, 2, 1, 3]
        for t, n in (("v", 40), ("v.conv", 40)):
            bad["l0.mix." + t] = w["l0.mix." + t].reshape(4, n, -1)[order].reshape(w["l0.mix." + t].shape)
        assert mm.error(plain.forward(cfg, bad, toks), right).max() > 2 * mm.TOLERANCE[mm.AUTO]
        return
    bad = copy.deepcopy(cfg)
    d = bad["layers"][layer]
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    assert mm.error(plain.forward(bad, w, toks), right).max() > 2 * mm.TOLERANCE[mm.AUTO]


@pytest.mark.parametrize("name,value", [
    ("l1.mix.left.sink", -60.0), ("l4.mix.left.sink", -60.0), ("l1.mix.left.g", 0.0), ("l1.mix.right.g", 0.0), ("l2.mix.y.b", 0.0), ("l2.mix.x.b", 0.0),
    ("l2.mix.conv.b", 0.0), ("l2.mix.ra.b", 0.0), ("l2.mix.ri.b", 0.0), ("l2.mix.lam", 0.0), ("l0.mix.dt_bias", 0.0), ("l0.mix.A_log", 0.0), ("l0.mix.norm", 1.0),
    ("l0.mix.b", 0.0), ("l0.mix.g2", 0.0), ("l0.mix.a2", 0.0), ("l0.norm1", 1.0), ("l0.norm2", 1.0), ("final.norm", 1.0)])
def test_a_mechanism_that_is_left_out_shows(model, name, value):
    cfg, w, toks, right = model
    bad = dict(w, **{name: np.full_like(w[name], value)})
    assert mm.error(plain.forward(cfg, bad, toks), right).max() > mm.TOLERANCE[mm.AUTO]


@pytest.mark.parametrize("name", ["l0.mix.q.conv", "l0.mix.k.conv", "l0.mix.v.conv", "l2.mix.conv", "l3.mix.v.conv"])
def test_a_convolution_the_wrong_way_round_shows(model, name):
    cfg, w, toks, right = model
    bad = dict(w, **{name: w[name][:, ::-1]})
    assert mm.error(plain.forward(cfg, bad, toks), right).max() > 2 * mm.TOLERANCE[mm.AUTO]


@pytest.mark.parametrize("planted", ["delta read before write", "delta without fading", "retention state lost", "gated state lost"])
def test_a_wrong_recurrence_shows(model, monkeypatch, planted):
    """Mistakes in the scans: an order of steps, a state that does not survive position 40."""
    cfg, w, toks, right = model
    if planted.startswith("delta"):
        def scan(q, k, v, g, beta):
            S, out = np.zeros((q.shape[1], q.shape[2], v.shape[2])), []
            for t in range(len(q)):
                S = S * (1.0 if "fading" in planted else g[t][:, :, None])
                if "read" in planted:
                    out.append(np.einsum("hdv,hd->hv", S, q[t]))
                u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None, :]
                if "read" not in planted:
                    out.append(np.einsum("hdv,hd->hv", S, q[t]))
            return np.array(out)
        monkeypatch.setattr(plain, "delta_scan", scan)
    elif planted.startswith("retention"):
        f = plain.retention_scan
        monkeypatch.setattr(plain, "retention_scan", lambda q, k, v, d: np.concatenate([f(q[:40], k[:40], v[:40], d), f(q[40:], k[40:], v[40:], d)]))
    else:
        f = plain.gated_scan
        monkeypatch.setattr(plain, "gated_scan", lambda a, b: np.concatenate([f(a[:40], b[:40]), f(a[40:], b[40:])]))
    e = mm.error(plain.forward(cfg, w, toks), right)
    assert e.max() > 2 * mm.TOLERANCE[mm.AUTO]
    if "lost" in planted:
        assert e[:40].max() == 0 and e[40:44].max() > mm.TOLERANCE[mm.AUTO]


@pytest.mark.parametrize("name", list(mm.MODELS))
def test_rounding_products_to_bfloat16_stays_within_the_serving_tolerance(name):
    cfg = mm.MODELS[name]
    w = mm.weights(cfg, 11)
    toks = mm.tokens(120, cfg, 6)
    e = mm.error(plain.forward(cfg, w, toks, cast=plain.bf16_round), plain.forward(cfg, w, toks))
    assert 1e-3 < np.median(e) and e.max() < mm.TOLERANCE[mm.AUTO]


class _Recorder:
    """Stands for the executor: remembers the stacked matrices the loader uploads."""

    def upload(self, dtype, rows, cols, packed):
        raw = np.frombuffer(np.ascontiguousarray(packed).tobytes(), np.uint16)
        assert raw.size == rows * cols
        return plain.bf16_to_f64(raw.tobytes()).reshape(rows, cols)


@pytest.mark.parametrize("name", list(mm.MODELS))
def test_loader_stacks_and_checks(tmp_path, monkeypatch, name):
    from llama_rust_b200 import executor as ex
    from llama_rust_b200 import models
    from llama_rust_b200.models import mukunex
    from llama_rust_b200.safetensors import SafetensorsError
    cfg = mm.MODELS[name]
    w = mm.weights(cfg, 3)
    seen = {}
    monkeypatch.setattr(mukunex, "DecoderSession", lambda ex, c, embd, layers, norm, **kw: seen.update(c=c, embd=embd, layers=layers, norm=norm, kw=kw) or "session")
    assert models.load(_Recorder(), mm.write(tmp_path / "m", cfg, w), n_seq=3, n_ctx=77) == "session"
    assert seen["c"]["n_ctx"] == 77 and seen["kw"]["n_seq"] == 3 and seen["c"]["norm_place"] == ex.NORM_INPUT
    assert np.array_equal(seen["kw"]["output"], w["head"]) and np.array_equal(seen["embd"], w["embed"])
    for i, (L, D) in enumerate(zip(cfg["layers"], seen["layers"])):
        m, d, p = L["mixer"], D["mixer"], f"l{i}.mix."
        W_in, at = d["in"], 0

        def rows(*names):
            nonlocal at
            for n in names:
                assert np.array_equal(W_in[at:at + len(w[p + n])], w[p + n]), n
                at += len(w[p + n])
        if L["type"] == "parallel":
            rows("left.q", "left.k", "left.v", "left.g")
            at = -(-at // 8) * 8
            rows("right.q", "right.k", "right.v", "right.g")
            assert np.array_equal(d["out"], np.concatenate([w[p + "left.o"], w[p + "right.o"]], 1))
            assert np.allclose(d["rot_freq"], plain.frequencies(m["left"]["rot"])) and np.allclose(D["beside"]["rot_freq"], plain.frequencies(m["right"]["rot"]))
            assert (D["mixer_scale"], D["beside_scale"]) == (m["left_scale"], m["right_scale"]) and np.array_equal(d["sink"], w[p + "left.sink"])
        elif L["type"] == "rglru":
            rows("y", "x")
            bs = m["width"] // m["blocks"]
            for b in range(m["blocks"]):
                assert np.array_equal(d["gates"][2 * b * bs:(2 * b + 1) * bs], w[p + "ra"][b]) and np.array_equal(d["gates"][(2 * b + 1) * bs:(2 * b + 2) * bs], w[p + "ri"][b])
        else:
            rows("q", "k", "v", "a1", "g1", "b")
            assert (d["decay_rank"], d["gate_rank"]) == cfg["ranks"][i]
            assert np.array_equal(d["conv"], np.concatenate([w[p + t + ".conv"] for t in "qkv"]))
        assert (D["mlp"] is None) == (L["mlp"] is None)
    for key in ("l0.norm1", "head"):
        bad = dict(w)
        bad[key] = bad[key][:-1]
        with pytest.raises(SafetensorsError, match=key):
            models.load(_Recorder(), mm.write(tmp_path / "bad", cfg, bad))
    for key, value, text in (("type", "unheard", "unheard"), ("mlp", dict(kind="sparse", ff=8), "sparse")):
        c = copy.deepcopy(cfg)
        c["layers"][0][key] = value
        with pytest.raises(ValueError, match=text):
            models.load(_Recorder(), mm.write(tmp_path / "bad2", c, w))


def test_prompts_of_a_session_that_cannot_rewind_are_read_again():
    from llama_rust_b200.executor import Session

    class Fake(Session):
        def __init__(self, rewinds):
            self.rewinds, self._h, self.n_seq = rewinds, None, 1
            self._ids, self.cut = [[5, 6, 7, 8]], []

        def seq_truncate(self, seq, n_keep):
            self.cut.append(n_keep)
            del self._ids[seq][n_keep:]
    for prompt, rest, cut in (([5, 6, 7, 8, 9], [9], 4), ([5, 6, 9], [5, 6, 9], 0), ([5, 6, 7, 8], [5, 6, 7, 8], 0), ([1], [1], 0)):
        s = Fake(False)
        assert s.prompt_suffix(prompt) == rest and s.cut == [cut]
    s = Fake(True)
    assert s.prompt_suffix([5, 6, 9]) == [9] and s.cut == [2]
