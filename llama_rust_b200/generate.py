"""Greedy generation from the command line, through the registry and the engine:

    python -m llama_rust_b200.generate --model PATH --tokens 5,17,3 [--tokens ...] --n 32

PATH is a GGUF file or a folder with config.json and model.safetensors.  Every --tokens is one prompt (token ids); they are
served together by the batch scheduler.  Prints one JSON line per prompt."""
from __future__ import annotations

import argparse
import json


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--tokens", action="append", required=True, help="a prompt: token ids with commas between them")
    ap.add_argument("--n", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--eos", type=int, default=None)
    ap.add_argument("--ctx", type=int, default=None, help="context length (default: what the model allows)")
    ap.add_argument("--max-seqs", type=int, default=8, help="sequences served at a time")
    ap.add_argument("--prefill-chunk", type=int, default=0)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16",
                    help="float32: f32 arithmetic throughout")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.replace(" ", "").split(",")] for p in a.tokens]
    from . import build
    build.ensure()
    from . import Engine, EngineCfg, Executor, models
    from .executor import PATH_AUTO, PATH_MMA
    with Executor(0) as ex:
        ex.set_path(PATH_AUTO if a.dtype == "bfloat16" else PATH_MMA)
        n_seq = min(a.max_seqs, len(prompts))
        s = models.load(ex, a.model, n_ctx=a.ctx, n_seq=n_seq)
        eng = Engine(s, EngineCfg(max_seqs=n_seq, eos=a.eos, prefill_chunk=a.prefill_chunk))
        ids = [eng.add(p, a.n) for p in prompts]
        eng.run()
        for p, i in zip(prompts, ids):
            print(json.dumps({"prompt": p, "generated": eng.take(i).generated}))
        s.free()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
