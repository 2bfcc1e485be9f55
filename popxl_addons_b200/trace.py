"""Trace replay: feeds given token ids through a model step by step and writes logits. Nothing is sampled; the steps run on
the same `SequenceGenerator` as generation does.

Standard input holds one JSON object a line, `{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}`. A new id
takes a slot, its tokens continue where its last entry ended, the ids in `end` give their slots back after the step. When
something is wanted, `<out>/<step>.f32` receives the logits at the wanted places (entry by entry) as little-endian float32;
after every step the line `done <step>` is printed. Exit code 0 at the end of input.
"""
import argparse
import json
import os
import sys

import numpy as np

__all__ = ["main", "replay"]


def replay(gen, lines, out_dir: str, echo=print) -> None:
    for line in lines:
        if not line.strip():
            continue
        msg = json.loads(line)
        step, entries = int(msg["step"]), msg["entries"]
        ids = [e["id"] for e in entries]
        if len(set(ids)) != len(ids):
            raise ValueError(f"step {step} has two entries of one request")
        for e in entries:
            if e["id"] not in gen.slots:
                gen.admit(e["id"])
        want = {e["id"]: e.get("want") or [] for e in entries}
        logits = gen.step({e["id"]: e["tokens"] for e in entries}, want)
        rows = [logits[i] for i in ids if want[i]]
        if rows:
            path = os.path.join(out_dir, f"{step}.f32")
            np.concatenate(rows).astype("<f4").tofile(path + ".part")
            os.replace(path + ".part", path)
        for i in msg.get("end") or ():
            gen.release(i)
        echo(f"done {step}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="folder that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--requests", type=int, default=1, help="most requests that are live at a time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    from .models.registry import load_model

    gen = load_model(a.model, dtype=a.dtype, batch=a.requests, max_seq=max(1, a.max_tokens), device=a.device)
    replay(gen, sys.stdin, a.out, echo=lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
