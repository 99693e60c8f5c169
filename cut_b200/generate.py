"""Command line: greedy generation from token ids.

    python -m cut_b200.generate --model DIR|FILE.gguf --tokens 5,17,3 --n 32 [--dtype bfloat16|float32] [--portion N]

A model folder (config.json, model.safetensors) is served by the class the registry names for it; a llama-style GGUF file by
the C++ runner.  Several prompts, separated by ';', are served one after the other."""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m cut_b200.generate", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="a model folder or a .gguf file")
    ap.add_argument("--tokens", required=True, help="prompt token ids with commas between them; ';' between prompts")
    ap.add_argument("--n", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="arithmetic of a model folder")
    ap.add_argument("--portion", type=int, default=None, help="feed prompts in portions of this many tokens")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",") if t.strip()] for p in a.tokens.split(";")]
    if a.model.endswith(".gguf"):
        from .llama_decode import run_cpp_runner

        longest = max(len(p) for p in prompts) + a.n
        for p in prompts:
            out = run_cpp_runner(a.model, p, max(0, a.n - 1), max_seq=longest, batch_prompt=len(p) > 1)
            print(json.dumps({"prompt": p, "tokens": [int(t) for t in out["tokens"][len(p) - 1:]][: a.n]}), flush=True)
        return 0
    from . import _lib, build
    from .decoding import RequestQueue
    from .models import load_model

    _lib.load(build.build_layers())
    dec = load_model(a.model, a.dtype, max_seq=max(len(p) for p in prompts) + a.n)
    queue = RequestQueue(dec, a.portion)
    requests = [queue.submit(p, a.n) for p in prompts]
    queue.run()
    for r in requests:
        print(json.dumps({"prompt": r.prompt, "tokens": r.tokens}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
