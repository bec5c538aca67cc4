"""Nagolix: a decoder whose layers mix sliding-window latent attention and windowed attention with kept first tokens and
a learned distance bias, norms on the sublayers' outputs only, a clamped gated unit, learned positions and a tied
output.  This file reads config.json and the tensors; the mechanisms are those of executor.DecoderSession.

config.json: vocab, width, max_positions, norm.eps, embedding.scale and `layers`, each with `type`, `mixer` (sizes, scale,
mask) and `mlp` (or null).  Tensors: embed, pos, final.norm and, per layer i, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*."""
from __future__ import annotations

import numpy as np

from ..executor import DecoderSession, GATE_ELEMENT, GATE_HEAD, MIXER_ATTENTION, MIXER_LATENT
from ..safetensors import SafetensorsFile
from . import register
from .weights import Weights

GLU_ALPHA, GLU_SHIFT = 1.702, 1.0  # fixed by the design


def _latent(w: Weights, p: str, m: dict, width: int) -> dict:
    H, d, dv, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    src = m.get("kv_from")
    own = [] if src is not None else [(p + "dkv", R, width)]
    return dict(kind=MIXER_LATENT, n_head=H, dim=d, vdim=dv, kv_rank=R, scale=m["scale"], kv_from=-1 if src is None else src,
                window=m["mask"]["size"], gate=GATE_HEAD,
                up_k=w.stack((p + "uk", H * d, R)), up_v=w.stack((p + "uv", H * dv, R)), out=w.stack((p + "o", width, H * dv)),
                kv_norm=None if src is not None else w.vector(p + "dkv.norm", R),
                **{"in": w.stack((p + "q", H * d, width), *own, (p + "g", H, width))})


def _attention(w: Weights, p: str, m: dict, width: int) -> dict:
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rel = w.file.f32(p + "rel")
    w.expect(p + "rel", rel.shape[0], H)
    return dict(kind=MIXER_ATTENTION, n_head=H, n_head_kv=G, dim=d, vdim=dv, scale=m["scale"], window=m["mask"]["size"],
                keep_first=m["mask"]["keep_first"], gate=GATE_ELEMENT, rel=rel, bias_max=m["bias_max"],
                in_bias=np.concatenate([w.vector(p + "q.b", H * d), w.vector(p + "k.b", G * d), w.vector(p + "v.b", G * dv)]),
                q_norm=w.vector(p + "q.norm", H * d), k_norm=w.vector(p + "k.norm", G * d), out=w.stack((p + "o", width, H * dv)),
                **{"in": w.stack((p + "q", H * d, width), (p + "k", G * d, width), (p + "v", G * dv, width), (p + "g", H * dv, width))})


MIXERS = {"latent_attention": _latent, "attention": _attention}


def _dense(w: Weights, p: str, f: dict, width: int) -> dict:
    if f["kind"] != "dense":
        raise ValueError(f"unknown feed-forward {f['kind']!r}")
    return dict(n_ff=f["ff"], limit=f["limit"], alpha=GLU_ALPHA, shift=GLU_SHIFT,
                gate_up=w.stack((p + "gate", f["ff"], width), (p + "up", f["ff"], width)), down=w.stack((p + "down", width, f["ff"])))


@register("Nagolix", "folder")
def load(ex, model, n_ctx=None, **session_args):
    cfg, path = model
    w = Weights(ex, SafetensorsFile(path))
    width, vocab, positions = cfg["width"], cfg["vocab"], cfg["max_positions"]
    layers = []
    for i, L in enumerate(cfg["layers"]):
        if L["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {L['type']!r}; known: {', '.join(sorted(MIXERS))}")
        mlp = L.get("mlp")
        layers.append(dict(mixer=MIXERS[L["type"]](w, f"l{i}.mix.", L["mixer"], width), mixer_norm=1.0 + w.vector(f"l{i}.norm1", width),
                           mlp=None if mlp is None else _dense(w, f"l{i}.mlp.", mlp, width),
                           mlp_norm=None if mlp is None else 1.0 + w.vector(f"l{i}.norm2", width)))
    return DecoderSession(ex, dict(n_embd=width, n_vocab=vocab, n_ctx=min(n_ctx or positions, positions), norm_eps=cfg["norm"]["eps"],
                                   embd_scale=cfg["embedding"]["scale"]),
                          w.stack(("embed", vocab, width)), layers, 1.0 + w.vector("final.norm", width), pos_embd=w.stack(("pos", positions, width)),
                          **session_args)
