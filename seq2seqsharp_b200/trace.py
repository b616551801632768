"""Replays a trace of given token ids through a model and writes logits.

Steps come as JSON lines: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}.  Every entry appends
its tokens to the request's cache; "want" names the places among them whose logits are written to OUT/<step>.f32 (little-endian
float32, [wanted, vocab], in the order of the entries).  "end" lists requests that are finished after the step; their slots are
given back.  After every step a line "done <step>" is printed.

It drives the same engine as generation: a portion of a prompt runs like a prompt on top of a slot's cache, a single token of the
only live request like a step of the token loop (the captured decode step with its id given from the host).
"""
import argparse
import json
import os
import sys

import numpy as np

MAX_LIVE = 4


class TraceReplay:
    """Requests by id on the slots of an engine."""

    def __init__(self, gpt):
        from .gpt import DecodingOptions
        self.gpt, self.opts = gpt, DecodingOptions()
        self.slot_of = {}
        self.length = {}
        gpt.Reset()

    def run_entry(self, rid, tokens, want) -> np.ndarray:
        if rid not in self.slot_of:
            used = set(self.slot_of.values())
            slot = next(i for i in range(self.gpt.max_batch + 1) if i not in used)
            if slot >= self.gpt.max_batch:
                raise ValueError("more than %d live requests" % self.gpt.max_batch)
            self.gpt.SlotReset(slot)
            self.slot_of[rid], self.length[rid] = slot, 0
        slot = self.slot_of[rid]
        if len(tokens) == 1 and self.length[rid] > 0 and self.gpt.Batch() == 1:
            self.gpt.StepHost(np.asarray(tokens, dtype=np.int32), self.opts)
            out = self.gpt.Logits(want_probs=False)[0][[0] * len(want)]
        else:
            out = self.gpt.SlotLogits(slot, tokens, want)
        self.length[rid] += len(tokens)
        return out

    def end(self, rid):
        slot = self.slot_of.pop(rid)
        self.length.pop(rid)
        if self.slot_of:
            self.gpt.SlotReset(slot)
        else:
            self.gpt.Reset()

    def step(self, entries, end) -> np.ndarray:
        rows = [self.run_entry(e["id"], e["tokens"], e.get("want", [])) for e in entries if e["tokens"]]
        for rid in end:
            self.end(rid)
        return np.concatenate(rows) if rows else np.zeros((0, self.gpt.cfg.V), dtype=np.float32)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given token ids through a model step by step and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    from . import build
    build.build()
    from .registry import load_model
    gpt = load_model(a.model, dtype=a.dtype, max_batch=MAX_LIVE, max_tokens=a.max_tokens + 2)
    replay = TraceReplay(gpt)
    for line in sys.stdin:
        if not line.strip():
            continue
        j = json.loads(line)
        logits = replay.step(j.get("entries", []), j.get("end", []))
        if len(logits):
            np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(a.out, "%d.f32" % j["step"]))
        print("done %d" % j["step"], flush=True)
    gpt.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
