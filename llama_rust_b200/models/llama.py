"""The Llama family from GGUF files (dense, or with routed experts)."""
from ..gguf import load_llama
from . import register


@register("llama", "gguf")
def load(ex, gguf, n_ctx=None, **session_args):
    try:
        return load_llama(ex, gguf, n_ctx, **session_args)
    finally:
        gguf.close()
