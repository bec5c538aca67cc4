"""Small Nagolix models with random weights, written as a folder (config.json, model.safetensors), and the comparisons the
tests make.  Query/key norm weights are large enough that a softmax rests on few keys: a key that should not be seen, or
one that is missing, changes the logits by far more than the tolerances."""
import json
import os
import struct

import numpy as np

import nagolix_plain as plain


def attention(heads, kv_heads, dim, vdim, window, keep, bias_max, scale=None):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, bias_max=bias_max,
                                             mask=dict(size=window, keep_first=keep)))


def latent(heads, dim, vdim, rank, window, kv_from=None, scale=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, scale=scale or dim ** -0.5, mask=dict(size=window))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m)


def config(width, vocab, layers, ff, limit=1.5, eps=1e-5, scale=2.5, positions=640):
    """ff: one size for all layers, or a list with 0 for a layer without a feed-forward."""
    ff = ff if isinstance(ff, list) else [ff] * len(layers)
    return dict(architecture="Nagolix", width=width, vocab=vocab, max_positions=positions, norm=dict(eps=eps), embedding=dict(scale=scale),
                layers=[dict(L, mlp=dict(kind="dense", ff=f, limit=limit) if f else None) for L, f in zip(layers, ff)])


def weights(cfg, seed, buckets=12, sharp=3.0):
    """name -> float array, already rounded to bfloat16."""
    rng = np.random.default_rng(seed)
    w = {}

    def put(name, shape, std=None, mean=0.0):
        std = std if std is not None else 1.0 / np.sqrt(shape[-1])
        a = (mean + rng.standard_normal(shape) * std).astype(np.float32)
        w[name] = plain.bf16_to_f64(plain.f32_to_bf16(a).tobytes()).reshape(shape)
    W = cfg["width"]
    put("embed", (cfg["vocab"], W), 0.4)
    put("pos", (cfg["max_positions"], W), 0.5)
    put("final.norm", (W,), 0.2)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        put(f"l{i}.norm1", (W,), 0.3)
        put(p + "q", (H * d, W))
        put(p + "o", (W, H * dv))
        if L["type"] == "attention":
            G = m["kv_heads"]
            for t, n in (("k", G * d), ("v", G * dv)):
                put(p + t, (n, W))
            for t, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                put(p + t + ".b", (n,), 0.5)
            put(p + "q.norm", (H * d,), 0.2, sharp)
            put(p + "k.norm", (G * d,), 0.2, 1.0)
            put(p + "rel", (buckets, H), 1.5)
            put(p + "g", (H * dv, W))
        else:
            R = m["kv_rank"]
            w[p + "q"] *= 2 * sharp / np.sqrt(cfg["embedding"]["scale"])
            w[p + "q"] = plain.bf16_to_f64(plain.f32_to_bf16(w[p + "q"]).tobytes()).reshape(H * d, W)
            if "kv_from" not in m:
                put(p + "dkv", (R, W))
                put(p + "dkv.norm", (R,), 0.3, 1.0)
            put(p + "uk", (H * d, R))
            put(p + "uv", (H * dv, R))
            put(p + "g", (H, W))
        if L["mlp"]:
            put(f"l{i}.norm2", (W,), 0.3)
            for t, s in (("gate", (L["mlp"]["ff"], W)), ("up", (L["mlp"]["ff"], W)), ("down", (W, L["mlp"]["ff"]))):
                put(f"l{i}.mlp.{t}", s)
    return w


def write(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, data = {}, b""
    for name, a in w.items():
        raw = plain.f32_to_bf16(a).tobytes()
        head[name] = dict(dtype="BF16", shape=list(a.shape), data_offsets=[len(data), len(data) + len(raw)])
        data += raw
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + data)
    return str(folder)


# heads, head sizes, ranks, windows, order of layers and buckets differ between these, and include values that other models
# make equal or 1; "odd" has no size that is a multiple of eight, "tiles" sizes at the tensor-core kernels' full width
MODELS = {
    "mix": (config(96, 211, [latent(5, 16, 24, 48, 9), attention(6, 2, 24, 40, 11, 3, 24), latent(7, 8, 16, 48, 21, kv_from=0),
                             attention(4, 4, 32, 16, 17, 5, 40)], [72, 0, 56, 88]), 8),
    "groups": (config(128, 150, [attention(12, 1, 16, 48, 33, 1, 16), latent(12, 24, 8, 80, 37), latent(1, 40, 72, 80, 5, kv_from=1),
                                 attention(3, 3, 72, 24, 1, 2, 10)], 104, limit=0.6, eps=1e-3, scale=1.0), 6),
    "odd": (config(44, 101, [attention(3, 1, 10, 6, 13, 2, 12), latent(3, 9, 7, 18, 15), attention(2, 2, 5, 3, 4, 0, 30)], 30), 7),
    "tiles": (config(192, 130, [latent(16, 64, 64, 512, 100), attention(8, 2, 128, 128, 70, 4, 90), latent(4, 64, 128, 256, 130),
                                attention(4, 2, 64, 256, 150, 9, 64)], 256), 32),
    "wide window": (config(64, 90, [attention(2, 1, 32, 64, 1000, 7, 200), latent(2, 32, 32, 136, 2000)], 64), 20),
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
TOLERANCE = {F32: 2e-5, AUTO: 6e-2}
SHARP = {F32: 3.0, AUTO: 1.5}  # sharper models amplify the rounding of bfloat16 products beyond the serving tolerance
