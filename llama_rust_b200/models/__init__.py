"""Model registry: which architectures the framework serves, and the step from a model on disk to a session.

A model is a GGUF file (`general.architecture` names it) or a folder with config.json (`architecture`) and
model.safetensors.  `load` picks the loader by that name; every loader uploads the weights and returns a session whose
interface is that of executor.Session, so the engine, the command line and the trace runner do not care which one it is."""
from __future__ import annotations

import json
import os

_LOADERS = {}


def register(name: str, source: str):
    """Decorator: fn(executor, opened model, **session arguments) -> Session.  source: "gguf" or "folder"."""
    def add(fn):
        _LOADERS[(source, name)] = fn
        return fn
    return add


def architectures() -> list:
    return sorted(name for _, name in _LOADERS)


def read_config(folder) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load(ex, path, **session_args):
    """The session of the model at `path`.  session_args: n_ctx (default: what the model allows), n_seq, kv_blocks,
    block_tokens."""
    if os.path.isdir(path):
        cfg = read_config(path)
        name, source, model = cfg.get("architecture"), "folder", (cfg, os.path.join(path, "model.safetensors"))
    else:
        from ..gguf import GgufFile
        model = GgufFile(path)
        name, source = model.kv_string("general.architecture") or "llama", "gguf"
    if (source, name) not in _LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _LOADERS[(source, name)](ex, model, **session_args)


from . import llama, mukunex, nagolix  # noqa: E402,F401  (they register themselves)
