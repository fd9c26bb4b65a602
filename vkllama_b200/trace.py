"""Replays a trace of token ids through a model and writes the logits it is asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one step per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Each step feeds the next tokens of one sequence ("id"); "want" lists the places among them whose logits
go to OUT/<step>.f32 (little-endian fp32, [wanted, vocab]; no file when nothing is wanted). "end" names the
sequences that are finished. After every step a line "done <step>" is printed. The model holds one sequence
at a time: a new one starts at position 0 of the same caches once the one before has ended.
"""
import argparse
import json
import os
import sys

import numpy as np

from . import build as _build


def replay(model, lines, out_dir, say):
    """Runs the steps in `lines` (JSON texts) on `model`."""
    live, pos = None, 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        wanted = []
        for e in step["entries"]:
            if live is None:
                live, pos = e["id"], 0
            elif e["id"] != live:
                raise ValueError("sequence %r has not ended: one sequence is live at a time" % (live,))
            toks, want = e["tokens"], e.get("want", [])
            if not toks:
                continue
            y = model.forward_rows(toks, pos, want)
            pos += len(toks)
            if len(want):
                wanted.append(y)
        if wanted:
            path = os.path.join(out_dir, "%d.f32" % step["step"])
            np.concatenate(wanted).astype("<f4").tofile(path)
        if live is not None and live in step.get("end", []):
            live = None
        say("done %d" % step["step"])


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through a model")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold")
    a = ap.parse_args(argv)
    _build.build()  # nothing to do when the library is newer than its sources
    import vkllama_b200 as vk
    dev = vk.Device(0)
    model = vk.load_model(dev, a.model, a.max_tokens, vk.FP32 if a.dtype == "float32" else vk.BF16)

    def say(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(model, sys.stdin, a.out, say)
    model.close()
    dev.close()
    return 0
