"""Mukunex: a decoder whose layers mix, each by itself, a gated delta rule with a decay per key channel, a real-gated linear
recurrence behind a short convolution, or rotated attention with a sink beside a retention that reads the same input; norms
on the sublayers' inputs, a gelu gated unit.  This file reads config.json and the tensors; the mechanisms are those of
executor.DecoderSession.

config.json: vocab, width, norm.eps and `layers`, each with `type`, `mixer` (sizes, rotations, decays, scales) and `mlp` (or
null).  Tensors: embed, head, final.norm and, per layer i, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*.  The design sets no
limit to a sequence: n_ctx is the caller's choice."""
from __future__ import annotations

import math

import numpy as np

from ..executor import (DecoderSession, GATE_HEAD, MIXER_ATTENTION, MIXER_DELTA, MIXER_GATED_LINEAR, MIXER_RETENTION, NORM_INPUT, UNIT_GELU)
from ..safetensors import SafetensorsFile
from . import register
from .weights import Weights

UNIT_EPS = 1e-6      # of the delta rule's unit vectors
DECAY_FACTOR = 8.0   # of the gated recurrence: log a = -8 r softplus(lam)
DEFAULT_CTX = 8192   # positions a session holds when the caller does not say


def rotation(rot: dict) -> np.ndarray:
    """An angle per position for each pair: base^(-2 i / dims); with `scaling`, long wavelengths are stretched by `factor`, short
    ones kept, and those between blended."""
    f = float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
    sc = rot.get("scaling")
    if sc:
        turns = sc["original"] * f / (2.0 * math.pi)  # of the pair over the original context
        blend = np.clip((turns - sc["low"]) / max(sc["high"] - sc["low"], 1e-300), 0.0, 1.0)
        f = (1.0 - blend) * f / sc["factor"] + blend * f
    return f


def _parallel(w: Weights, p: str, m: dict, width: int) -> dict:
    a, r = m["left"], m["right"]
    H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
    rh, rd, rv = r["heads"], r["dim"], r["vdim"]
    left, right = p + "left.", p + "right."
    rows = H * d + G * d + G * dv + H
    return dict(
        mixer=dict(kind=MIXER_ATTENTION, n_head=H, n_head_kv=G, dim=d, vdim=dv, scale=a["scale"], gate=GATE_HEAD, rot_freq=rotation(a["rot"]),
                   sink=w.vector(left + "sink", H), out=w.beside((left + "o", width, H * dv), (right + "o", width, rh * rv)),
                   **{"in": w.stack((left + "q", H * d, width), (left + "k", G * d, width), (left + "v", G * dv, width), (left + "g", H, width), -rows % 8,
                                    (right + "q", rh * rd, width), (right + "k", rh * rd, width), (right + "v", rh * rv, width),
                                    (right + "g", rh * rv, width), -(2 * rh * (rd + rv)) % 8)}),
        beside=dict(kind=MIXER_RETENTION, n_head=rh, dim=rd, vdim=rv, scale=rd ** -0.5, rot_freq=rotation(r["rot"]), decay=_per_head(r["decay"], rh)),
        mixer_scale=m["left_scale"], beside_scale=m["right_scale"])


def _per_head(values, heads):
    if len(values) != heads:
        raise ValueError(f"{len(values)} decays for {heads} heads")
    return values


def _rglru(w: Weights, p: str, m: dict, width: int) -> dict:
    W, B = m["width"], m["blocks"]
    return dict(mixer=dict(
        kind=MIXER_GATED_LINEAR, width=W, blocks=B, taps=m["conv"], scale=DECAY_FACTOR,
        in_bias=np.concatenate([w.vector(p + "y.b", W), w.vector(p + "x.b", W)]), conv=w.vector(p + "conv", W, m["conv"]), conv_bias=w.vector(p + "conv.b", W),
        gates=w.blocks(B, W // B, W // B, p + "ra", p + "ri"),
        gate_bias=np.stack([w.vector(p + "ra.b", B, W // B), w.vector(p + "ri.b", B, W // B)], 1),
        decay=w.vector(p + "lam", W), out=w.stack((p + "o", width, W)), **{"in": w.stack((p + "y", W, width), (p + "x", W, width))}))


def _channel_delta(w: Weights, p: str, m: dict, width: int) -> dict:
    H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    ra, rg = w.rows(p + "a1"), w.rows(p + "g1")
    rows = 2 * G * d + H * dv + ra + rg + H
    return dict(mixer=dict(
        kind=MIXER_DELTA, n_head=H, n_head_kv=G, dim=d, vdim=dv, scale=d ** -0.5, taps=T, unit_eps=UNIT_EPS, decay_rank=ra, gate_rank=rg,
        conv=np.concatenate([w.vector(p + t + ".conv", n, T) for t, n in (("q", G * d), ("k", G * d), ("v", H * dv))]),
        decay=w.vector(p + "A_log", H), step_bias=w.vector(p + "dt_bias", H * d), head_norm=w.vector(p + "norm", dv),
        decay_up=w.stack((p + "a2", H * d, ra)), gate_up=w.stack((p + "g2", H * dv, rg)), out=w.stack((p + "o", width, H * dv)),
        **{"in": w.stack((p + "q", G * d, width), (p + "k", G * d, width), (p + "v", H * dv, width), (p + "a1", ra, width), (p + "g1", rg, width),
                         (p + "b", H, width), -rows % 8)}))


MIXERS = {"parallel": _parallel, "rglru": _rglru, "channel_delta": _channel_delta}


def _dense(w: Weights, p: str, f: dict, width: int) -> dict:
    if f["kind"] != "dense":
        raise ValueError(f"unknown feed-forward {f['kind']!r}")
    return dict(n_ff=f["ff"], unit=UNIT_GELU, gate_up=w.stack((p + "gate", f["ff"], width), (p + "up", f["ff"], width)),
                down=w.stack((p + "down", width, f["ff"])))


@register("Mukunex", "folder")
def load(ex, model, n_ctx=None, **session_args):
    cfg, path = model
    w = Weights(ex, SafetensorsFile(path))
    width, vocab = cfg["width"], cfg["vocab"]
    layers = []
    for i, L in enumerate(cfg["layers"]):
        if L["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}; known: {', '.join(sorted(MIXERS))}")
        mlp = L.get("mlp")
        layers.append(dict(MIXERS[L["type"]](w, f"l{i}.mix.", L["mixer"], width), mixer_norm=w.vector(f"l{i}.norm1", width),
                           mlp=None if mlp is None else _dense(w, f"l{i}.mlp.", mlp, width),
                           mlp_norm=None if mlp is None else w.vector(f"l{i}.norm2", width)))
    return DecoderSession(ex, dict(n_embd=width, n_vocab=vocab, n_ctx=n_ctx or DEFAULT_CTX, norm_eps=cfg["norm"]["eps"], embd_scale=1.0, norm_place=NORM_INPUT),
                          w.stack(("embed", vocab, width)), layers, w.vector("final.norm", width), output=w.stack(("head", vocab, width)), **session_args)
