"""A plain, slow statement of the Nagolix decoder in float64 numpy: one function per mechanism, a whole sequence at a
time, no cache.  Test infrastructure: what the device-resident session is compared with; it shares no code with it."""
import json
import os
import struct

import numpy as np


def bf16_to_f64(raw):
    return (np.frombuffer(raw, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def f32_to_bf16(a):
    """Nearest bfloat16 (ties to even) as uint16."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def read_model(folder):
    cfg = json.load(open(os.path.join(folder, "config.json")))
    data = open(os.path.join(folder, "model.safetensors"), "rb").read()
    n, = struct.unpack("<Q", data[:8])
    head = json.loads(data[8:8 + n])
    w = {}
    for name, t in head.items():
        if name != "__metadata__":
            a, b = t["data_offsets"]
            assert t["dtype"] == "BF16"
            w[name] = bf16_to_f64(data[8 + n + a:8 + n + b]).reshape(t["shape"])
    return cfg, w


def bf16_round(a):
    """Nearest bfloat16 values (what the serving path feeds its products with)."""
    return bf16_to_f64(f32_to_bf16(a).tobytes()).reshape(np.shape(a))


def exact(a):
    return a


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, np.float64)))


def softmax(z):
    e = np.exp(z - z.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def embed(tokens, table, pos, scale):
    return table[tokens] * scale + pos[:len(tokens)]


def visible(n, window, keep_first):
    """[i, j]: does position i see position j?"""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    if window:
        seen &= (i - j < window) | (j < keep_first)
    return seen


def distance_bucket(n, buckets, bias_max):
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + int(np.floor(np.log(n / half) / np.log(bias_max / half) * (buckets - half) + 1e-9)))


def clamped_glu(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(x, w, p, limit, cast=exact):
    x = cast(x)
    return cast(clamped_glu(x @ w[p + "gate"].T, x @ w[p + "up"].T, limit)) @ w[p + "down"].T


def latent_of(h, w, p, eps, cast=exact):
    return rms(cast(h) @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]


def latent_attention(h, c, w, p, m, cast=exact):
    n, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    h, c = cast(h), cast(c)
    q = (h @ w[p + "q"].T).reshape(n, H, d)
    k = (c @ w[p + "uk"].T).reshape(n, H, d)
    v = (c @ w[p + "uv"].T).reshape(n, H, dv)
    s = np.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = np.where(visible(n, m["mask"]["size"], 0)[None], s, -np.inf)
    o = np.einsum("hij,jhd->ihd", softmax(s), v) * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return cast(o.reshape(n, H * dv)) @ w[p + "o"].T


def biased_attention(h, w, p, m, eps, cast=exact):
    n, H, G, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = cast(h)
    q = rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = h @ w[p + "v"].T + w[p + "v.b"]
    q, k, v = q.reshape(n, H, d), k.reshape(n, G, d), v.reshape(n, G, dv)
    k, v = np.repeat(k, H // G, axis=1), np.repeat(v, H // G, axis=1)
    s = np.einsum("ihd,jhd->hij", q, k) * m["scale"]
    rel = w[p + "rel"]
    by_distance = rel[[distance_bucket(t, len(rel), m["bias_max"]) for t in range(n)]]  # [distance, head]
    dist = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0)
    s = s + by_distance[dist].transpose(2, 0, 1)
    s = np.where(visible(n, m["mask"]["size"], m["mask"]["keep_first"])[None], s, -np.inf)
    o = np.einsum("hij,jhd->ihd", softmax(s), v).reshape(n, H * dv)
    return cast(o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def forward(cfg, w, tokens, stream=None, cast=exact):
    """Logits [n, vocab] of one sequence; `stream` (a list) receives the residual stream after every layer.  cast: applied
    to what enters a product (bf16_round: how much that rounding alone changes)."""
    eps = cfg["norm"]["eps"]
    x = embed(np.asarray(tokens), w["embed"], w["pos"], cfg["embedding"]["scale"])
    latents = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        if L["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_of(x, w, p, eps, cast)
            y = latent_attention(x, latents[i if src is None else src], w, p, m, cast)
        else:
            y = biased_attention(x, w, p, m, eps, cast)
        x = x + rms(y, eps) * (1.0 + w[f"l{i}.norm1"])
        if L["mlp"] is not None:
            x = x + rms(dense_ff(x, w, f"l{i}.mlp.", L["mlp"]["limit"], cast), eps) * (1.0 + w[f"l{i}.norm2"])
        if stream is not None:
            stream.append(x.copy())
    return cast(rms(x, eps) * (1.0 + w["final.norm"])) @ w["embed"].T
