"""Trace replay: given tokens of several requests, step by step, through a decoder session, writing the logits that are
asked for.  Steps come as JSON lines on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Each request holds one of the session's sequences from its first entry until a step's "end" names it; its tokens
continue where its last entry ended.  A step that wants logits writes <out>/<step>.f32 (rows in the order asked for,
little-endian f32); every step answers "done <step>" on standard output."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

import emel_cpp_b200 as eb
from emel_cpp_b200 import models


class Slots:
    """Requests -> the session's sequences; a finished request's sequence is taken by the next one."""

    def __init__(self, session, count: int):
        self.session = session
        self.free = list(range(count))
        self.at = {}        # id -> [sequence, tokens so far]

    def feed(self, rid, tokens, want):
        if rid not in self.at:
            if not self.free:
                raise RuntimeError("more live requests than sequences")
            self.at[rid] = [self.free.pop(0), 0]
        slot = self.at[rid]
        if not self.session.select_sequence(slot[0]):
            raise eb.BackendError(f"select_sequence failed with error mask {self.session.last_error}")
        order = sorted(set(want))
        rows = self.session.prefill_logits(tokens, slot[1], order)
        slot[1] += len(tokens)
        return rows[[order.index(w) for w in want]] if want else None

    def end(self, rid):
        if rid in self.at:
            self.free.append(self.at.pop(rid)[0])


def replay(session, lines, out_dir: str, slots: int, emit) -> None:
    live = Slots(session, slots)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if not e["tokens"]:
                continue
            r = live.feed(e["id"], e["tokens"], e.get("want") or [])
            if r is not None:
                rows.append(r)
        if rows:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end") or []:
            live.end(rid)
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="replay a token trace through a model")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=2, help="most requests alive at any time")
    a = ap.parse_args(argv)
    backend = eb.Backend(0)
    session = models.load(backend, a.model, n_ctx=max(a.max_tokens, 1), float32=a.dtype == "float32")
    if not session.set_sequences(a.slots):
        raise eb.BackendError(f"set_sequences failed with error mask {session.last_error}")

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()
    replay(session, sys.stdin, a.out, a.slots, emit)
    session.close()
    backend.close()
    return 0
