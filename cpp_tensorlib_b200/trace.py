"""Replay of a token trace: given ids are run through a model step by step and the logits at chosen
places are written out.  Nothing is sampled.

Standard input has one JSON object a line, ``{"step": n, "entries": [{"id", "tokens", "want"}],
"end": [ids]}``; a step with wanted places writes ``<out>/<n>.f32`` (little-endian f32,
[wanted, vocab]), and every step prints ``done <n>``.  A step brings the next tokens of the one live
sequence; a new id starts a new sequence once the one before it has ended.
"""
import argparse
import json
import os
import sys

import numpy as np

from .registry import DTYPES, load_model


def replay(model, lines, out_dir, emit):
    live = None
    if not model.captured:
        model.capture()
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        if len(step["entries"]) > 1:
            raise ValueError("one sequence at a time: a step has at most one entry")
        parts = []
        for e in step["entries"]:
            if live is None:
                model.set_pos(0)
                live = e["id"]
            elif live != e["id"]:
                raise ValueError("a sequence starts while another one is live")
            if e["tokens"]:
                places = sorted(set(e["want"]))
                got = model.extend(e["tokens"], places)
                parts += [got[places.index(w)] for w in e["want"]]
        if parts:
            np.stack(parts).astype("<f4").tofile(os.path.join(out_dir, "%d.f32" % step["step"]))
        if live in step.get("end", ()):
            live = None
        emit("done %d" % step["step"])


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=DTYPES, default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="capacity of the sequence state, in tokens")
    a = ap.parse_args(argv)
    model = load_model(a.model, a.dtype, a.max_tokens)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()
    replay(model, iter(sys.stdin.readline, ""), a.out, emit)
    model.close()
    return 0
