"""Replays a trace of steps through a model and writes the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  Each
entry's tokens continue the request of that id (a new id opens a sequence); the logits of the places in "want" go to
OUT/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of the entries and of want); requests in "end" give their
place back.  After every step a line "done <step>" is printed."""
from __future__ import annotations

import argparse
import json
import os
import sys


def replay(decoder, lines, out_dir: str, report) -> None:
    live = {}
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        chunks = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = decoder.open()
            want = [int(w) for w in e["want"]]
            order = sorted(set(want))
            rows = decoder.forward(live[e["id"]], e["tokens"], order)
            if want:
                host = rows.float().cpu().numpy()
                chunks.append(host[[order.index(w) for w in want]].astype("<f4").tobytes())
        for i in step.get("end", []):
            if i in live:
                decoder.close(live.pop(i))
        decoder.check_status()
        if chunks:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(b"".join(chunks))
        report(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=1, help="requests that may be live at the same time")
    a = ap.parse_args(argv)
    from . import _lib, build
    from .models import load_model, read_config

    entry, _ = read_config(a.model)
    if a.dtype not in entry.dtypes:
        print(f"{a.dtype}: this model does not run in it", file=sys.stderr)
        return 3
    _lib.load(build.build_layers())
    decoder = load_model(a.model, a.dtype, max_seq=a.max_tokens, slots=a.slots)
    replay(decoder, sys.stdin, a.out, lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
