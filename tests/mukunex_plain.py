"""A plain, slow statement of the Mukunex decoder in float64 numpy: one function per mechanism, a whole sequence at a time,
recurrences token by token, no cache.  Test infrastructure: what the device-resident session is compared with; it shares no
code with it."""
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


def bf16_round(a):
    """Nearest bfloat16 values (what the serving path feeds its products with)."""
    return bf16_to_f64(f32_to_bf16(a).tobytes()).reshape(np.shape(a))


def exact(a):
    return a


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


# ---- elementary functions ------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, np.float64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


# ---- rotation -------------------------------------------------------------------------------------------------------
def frequencies(rot):
    f = []
    for i in range(rot["dims"] // 2):
        v = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * np.pi / v
            if wave > sc["original"] / sc["low"]:
                v = v / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                v = (1.0 - s) * v / sc["factor"] + s * v
        f.append(v)
    return np.array(f)


def rotate(x, rot):
    """x [n, heads, dim], row p at position p."""
    half = rot["dims"] // 2
    a = np.arange(len(x))[:, None, None] * frequencies(rot)[None, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * half:]], -1)


# ---- short convolution ----------------------------------------------------------------------------------------------
def causal_conv(x, taps):
    """x [n, channels], taps [channels, T]: the last column weighs the row itself."""
    T = taps.shape[1]
    padded = np.concatenate([np.zeros((T - 1, x.shape[1])), x])
    return sum(padded[j:j + len(x)] * taps[:, j] for j in range(T))


# ---- mixers ----------------------------------------------------------------------------------------------------------
def sink_softmax(s, sink):
    """s [h, i, j] with -inf where unseen; sink [h] stands in the denominator only."""
    top = np.maximum(s.max(-1), sink[:, None])
    e = np.exp(s - top[..., None])
    return e / (e.sum(-1) + np.exp(sink[:, None] - top))[..., None]


def sink_attention(h, w, p, m, cast=exact):
    n, H, G, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = cast(h)
    q = rotate((h @ w[p + "q"].T).reshape(n, H, d), m["rot"])
    k = rotate((h @ w[p + "k"].T).reshape(n, G, d), m["rot"])
    v = (h @ w[p + "v"].T).reshape(n, G, dv)
    k, v = np.repeat(cast(k), H // G, axis=1), np.repeat(cast(v), H // G, axis=1)
    s = np.einsum("ihd,jhd->hij", cast(q), k) * m["scale"]
    s = np.where(np.tril(np.ones((n, n), bool))[None], s, -np.inf)
    o = np.einsum("hij,jhd->ihd", sink_softmax(s, w[p + "sink"]), v)
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return cast(o.reshape(n, H * dv)) @ w[p + "o"].T


def retention_scan(q, k, v, decay):
    """q, k [n, H, d], v [n, H, dv]; a matrix state per head that fades by a fixed factor."""
    S, out = np.zeros((q.shape[1], q.shape[2], v.shape[2])), []
    for t in range(len(q)):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(np.einsum("hdv,hd->hv", S, q[t]))
    return np.array(out)


def retention(h, w, p, m, eps, cast=exact):
    n, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    h = cast(h)
    q = rotate((h @ w[p + "q"].T).reshape(n, H, d), m["rot"])
    k = rotate((h @ w[p + "k"].T).reshape(n, H, d), m["rot"]) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(n, H, dv)
    o = rms(retention_scan(q, k, v, np.array(m["decay"], np.float64)), eps).reshape(n, H * dv)
    return cast(o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps, cast=exact):
    return m["left_scale"] * sink_attention(h, w, p + "left.", m["left"], cast) + m["right_scale"] * retention(h, w, p + "right.", m["right"], eps, cast)


def gated_scan(a, b):
    """S_t = a_t S_(t-1) + b_t per channel."""
    S, out = np.zeros(a.shape[1]), []
    for t in range(len(a)):
        S = a[t] * S + b[t]
        out.append(S)
    return np.array(out)


def rglru(h, w, p, m, eps, cast=exact):
    n, W, B = len(h), m["width"], m["blocks"]
    h = cast(h)
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    parts = u.reshape(n, B, W // B)
    r = sigmoid(np.einsum("boc,nbc->nbo", w[p + "ra"], parts) + w[p + "ra.b"]).reshape(n, W)
    i = sigmoid(np.einsum("boc,nbc->nbo", w[p + "ri"], parts) + w[p + "ri.b"]).reshape(n, W)
    log_a = -8.0 * r * softplus(w[p + "lam"])
    a = np.exp(log_a)
    S = gated_scan(a, np.sqrt(1.0 - a * a) * i * u)
    return cast(S * y) @ w[p + "o"].T


def delta_scan(q, k, v, g, beta):
    """q, k, g [n, H, d], v [n, H, dv], beta [n, H]: fade the state's key channels, correct what it holds for k towards v,
    read it with q."""
    S, out = np.zeros((q.shape[1], q.shape[2], v.shape[2])), []
    for t in range(len(q)):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(np.einsum("hdv,hd->hv", S, q[t]))
    return np.array(out)


def channel_delta(h, w, p, m, eps, cast=exact):
    n, H, G, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = cast(h)
    q, k, v = (silu(causal_conv(h @ w[p + t].T, w[p + t + ".conv"])) for t in "qkv")
    q, k = unit(q.reshape(n, G, d)) * d ** -0.5, unit(k.reshape(n, G, d))
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus(cast(h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(n, H, d)
    g = np.exp(-np.exp(w[p + "A_log"])[:, None] * step)
    o = rms(delta_scan(q, k, v.reshape(n, H, dv), g, beta), eps) * w[p + "norm"]
    o = o.reshape(n, H * dv) * sigmoid(cast(h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return cast(o) @ w[p + "o"].T


MIXERS = {"parallel": parallel, "rglru": rglru, "channel_delta": channel_delta}


def dense_ff(x, w, p, cast=exact):
    x = cast(x)
    return cast(gelu_tanh(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, tokens, stream=None, cast=exact):
    """Logits [n, vocab] of one sequence; `stream` (a list) receives the residual stream after every layer.  cast: applied
    to what enters a product (bf16_round: how much that rounding alone changes)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    for i, L in enumerate(cfg["layers"]):
        x = x + MIXERS[L["type"]](rms(x, eps) * w[f"l{i}.norm1"], w, f"l{i}.mix.", L["mixer"], eps, cast)
        if L.get("mlp") is not None:
            x = x + dense_ff(rms(x, eps) * w[f"l{i}.norm2"], w, f"l{i}.mlp.", cast)
        if stream is not None:
            stream.append(x.copy())
    return cast(rms(x, eps) * w["final.norm"]) @ w["head"].T
