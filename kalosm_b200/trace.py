"""Replays a trace of token ids through a model, step by step, and writes logits (bin/trace_run).

Steps come on standard input, one JSON object a line:
  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": []}
A step runs its tokens from the state that earlier steps left; the logits at the wanted places go to
<out>/<step>.f32 (little-endian f32, [wanted, vocab]), then the line "done <step>" is printed. Requests come
one after the other: the model's session is reset when a request ends.
"""
import argparse
import json
import os
import sys

import numpy as np


class Session:
    """One request at a time over a Decoder."""

    def __init__(self, model):
        self.model, self.live = model, None

    def run(self, entry):
        """Feeds an entry's tokens; returns the logits at its wanted places."""
        if self.live is None:
            self.model.reset()
            self.live = entry["id"]
        elif self.live != entry["id"]:
            raise RuntimeError(f"request {entry['id']} starts before {self.live} has ended: one request at a time")
        tokens, want = entry["tokens"], entry.get("want") or []
        if not tokens:
            return np.empty((0, self.model.vocab), np.float32)
        self.model.forward(tokens, want_logits=False)
        return self.model.logits_at(want)

    def end(self, name):
        if self.live == name:
            self.live = None
            self.model.reset()


def replay(model, lines, out_dir, emit):
    session = Session(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = [session.run(e) for e in step["entries"]]
        if any(e.get("want") for e in step["entries"]):
            path = os.path.join(out_dir, f"{step['step']}.f32")
            np.concatenate(rows).astype("<f4").tofile(path)
        for name in step.get("end") or []:
            session.end(name)
        emit(f"done {step['step']}")


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a GGUF file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens a live request holds")
    args = ap.parse_args(argv)
    import kalosm_b200
    from . import Device, build, models
    if "FB200_LIB_PATH" not in os.environ:  # compile what this model needs, if it is not there
        kalosm_b200.LIB_PATH = build.build(part="dense" if models.architecture(args.model) in models.DENSE else "all")
    model = models.load_model(Device(0), args.model, max_seq_len=max(args.max_tokens, 16), dtype=args.dtype)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()
    replay(model, iter(sys.stdin.readline, ""), args.out, emit)
    return 0
