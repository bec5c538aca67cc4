"""Small Mukunex models with random weights, written as a folder (config.json, model.safetensors), and the comparisons the
tests make.  Queries and keys are large enough that a softmax rests on few keys and decays slow enough that states remember:
a key, a sink or a state that is missing changes the logits by far more than the tolerances."""
import json
import os
import struct

import numpy as np

import mukunex_plain as plain


def rot(dims, base, scaling=None):
    r = dict(base=float(base), dims=dims)
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def parallel(left, right, scales=(0.7, 1.3)):
    """left: heads, kv_heads, dim, vdim, rot, scale; right: heads, dim, vdim, rot, decays"""
    return dict(type="parallel", mixer=dict(left=dict(zip(("heads", "kv_heads", "dim", "vdim", "rot", "scale"), left)),
                                            right=dict(zip(("heads", "dim", "vdim", "rot", "decay"), right)), left_scale=scales[0], right_scale=scales[1]))


def rglru(width, blocks, conv):
    return dict(type="rglru", mixer=dict(width=width, blocks=blocks, conv=conv))


def delta(heads, kv_heads, dim, vdim, conv, ranks=(8, 16)):
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), ranks=ranks)


def config(width, vocab, layers, ff, eps=1e-5):
    """ff: one size for all layers, or a list with 0 for a layer without a feed-forward."""
    ff = ff if isinstance(ff, list) else [ff] * len(layers)
    return dict(architecture="Mukunex", width=width, vocab=vocab, norm=dict(eps=eps),
                layers=[dict(type=L["type"], mixer=L["mixer"], mlp=dict(kind="dense", ff=f) if f else None) for L, f in zip(layers, ff)],
                ranks=[L.get("ranks") for L in layers])


def rounded(a):
    return plain.bf16_to_f64(plain.f32_to_bf16(np.asarray(a, np.float32)).tobytes()).reshape(np.shape(a))


def weights(cfg, seed, sharp=1.0):
    """name -> float array, already rounded to bfloat16.  The ranks of the low-rank pairs come from cfg["ranks"]."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, shape, std=None, mean=0.0):
        std = std if std is not None else 1.0 / np.sqrt(shape[-1])
        w[name] = rounded(mean + rng.standard_normal(shape) * std)
    W = cfg["width"]
    put("embed", (cfg["vocab"], W), 1.0)
    put("head", (cfg["vocab"], W))
    put("final.norm", (W,), 0.2, 1.0)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        put(f"l{i}.norm1", (W,), 0.2, 1.0)
        if L["type"] == "parallel":
            a, r = m["left"], m["right"]
            for t, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"])):
                put(p + "left." + t, (n, W), np.sqrt(1.5 * sharp) * (a["scale"] ** 2 * a["dim"]) ** -0.25 / np.sqrt(W))
            put(p + "left.v", (a["kv_heads"] * a["vdim"], W))
            put(p + "left.sink", (a["heads"],), 1.0, 4.0)
            put(p + "left.g", (a["heads"], W))
            put(p + "left.o", (W, a["heads"] * a["vdim"]))
            for t, n in (("q", r["heads"] * r["dim"]), ("k", r["heads"] * r["dim"]), ("v", r["heads"] * r["vdim"]), ("g", r["heads"] * r["vdim"])):
                put(p + "right." + t, (n, W))
            put(p + "right.o", (W, r["heads"] * r["vdim"]))
        elif L["type"] == "rglru":
            n, B, T = m["width"], m["blocks"], m["conv"]
            for t in "yx":
                put(p + t, (n, W))
                put(p + t + ".b", (n,), 0.3)
            put(p + "conv", (n, T), 0.5)
            put(p + "conv.b", (n,), 0.2)
            for t in ("ra", "ri"):
                put(p + t, (B, n // B, n // B))
                put(p + t + ".b", (B, n // B), 0.5)
            put(p + "lam", (n,), 1.5, -4.0)
            put(p + "o", (W, n))
        else:
            H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            ra, rg = cfg["ranks"][i]
            for t, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                put(p + t, (n, W))
                put(p + t + ".conv", (n, T), 0.6)
            put(p + "b", (H, W))
            put(p + "A_log", (H,), 0.5, -1.0)
            put(p + "norm", (dv,), 0.2, 1.0)
            put(p + "a1", (ra, W))
            put(p + "a2", (H * d, ra))
            put(p + "dt_bias", (H * d,), 1.0, -3.0)
            put(p + "g1", (rg, W))
            put(p + "g2", (H * dv, rg))
            put(p + "o", (W, H * dv))
        if L["mlp"]:
            put(f"l{i}.norm2", (W,), 0.2, 1.0)
            for t, s in (("gate", (L["mlp"]["ff"], W)), ("up", (L["mlp"]["ff"], W)), ("down", (W, L["mlp"]["ff"]))):
                put(f"l{i}.mlp.{t}", s)
    return w


def write(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump({k: v for k, v in cfg.items() if k != "ranks"}, f)
    head, data = {}, b""
    for name, a in w.items():
        raw = plain.f32_to_bf16(a).tobytes()
        head[name] = dict(dtype="BF16", shape=list(a.shape), data_offsets=[len(data), len(data) + len(raw)])
        data += raw
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + data)
    return str(folder)


# Sizes, ratios, taps, rotations and the order of layers differ between these, and include values that other models make
# equal or 1; "odd" has no size that is a multiple of eight, "tiles" sizes at the tensor-core kernels' and the scans' full
# widths, "long heads" heads longer than the eight-lane scans take
MODELS = {
    "mix": config(96, 211, [delta(4, 2, 24, 40, 4), parallel((6, 2, 24, 40, rot(16, 1e4, (4.0, 1.0, 4.0, 64)), 0.3), (3, 16, 24, rot(8, 5e4), [0.9, 0.99, 0.9995])),
                            rglru(80, 5, 4), delta(3, 3, 16, 8, 2, (24, 8)), parallel((4, 1, 32, 16, rot(32, 1e5), 0.15), (2, 40, 48, rot(40, 1e4), [0.75, 0.998]), (1.2, 0.4))],
                  [72, 0, 56, 88, 40]),
    "groups": config(128, 150, [rglru(128, 1, 3), parallel((12, 1, 16, 48, rot(16, 2e4, (8.0, 1.0, 2.0, 48)), 0.25), (1, 64, 72, rot(64, 1e6), [0.9999])),
                                delta(8, 2, 32, 16, 3, (40, 8)), rglru(64, 8, 1)], 104, eps=1e-3),
    "odd": config(44, 101, [parallel((3, 1, 10, 6, rot(4, 1e3, (2.0, 0.5, 1.5, 20)), 0.5), (3, 6, 5, rot(2, 1e4), [0.5, 0.96875, 0.999])), rglru(30, 6, 2),
                            delta(3, 1, 7, 9, 5, (3, 5))], 30),
    "tiles": config(192, 130, [delta(2, 1, 128, 128, 4, (32, 32)), parallel((8, 2, 128, 128, rot(64, 5e5, (4.0, 1.0, 4.0, 128)), 0.08), (2, 128, 256, rot(128, 1e4), [0.98, 0.9998])),
                               rglru(256, 2, 4), delta(2, 2, 64, 256, 4, (8, 8))], 256),
    "long heads": config(64, 90, [delta(1, 1, 300, 20, 2, (8, 8)), parallel((2, 1, 264, 136, rot(264, 1e4), 0.06), (1, 288, 24, rot(100, 1e4), [0.995])),
                                  delta(2, 1, 200, 72, 3, (16, 8)), rglru(512, 2, 4)], 64),
}


def tokens(n, cfg, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def error(got, want):
    """Per position: root mean square of the difference with its mean taken off, over the logits' own."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    ref = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((ref * ref).mean())


F32, AUTO = 3, 0  # kernel paths: f32 arithmetic throughout, the kernels that serve
TOLERANCE = {F32: 4e-5, AUTO: 3e-2}
