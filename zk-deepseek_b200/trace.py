"""Replays a trace: steps of given token ids, read as JSON lines, through the step function that generation uses.

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings the next tokens of a request and names the places among them whose logits are wanted; "end" lists
requests that are finished, whose cache slot is given back.  A step with wanted places writes <out>/<step>.f32
(float32, [wanted, vocab]); every step answers "done <step>" on standard output.
"""
import argparse
import json
import os
import sys

import torch

try:
    from . import registry
except ImportError:  # pragma: no cover - this directory first on sys.path
    import registry

SLOTS = 4            # requests that may be open at the same time


class Replayer:
    def __init__(self, model):
        self.model, self.open = model, {}          # request id -> [slots of begin_batch, tokens so far]

    def entry(self, rid, tokens, want):
        """float32 logits [len(want), vocab] on the host"""
        if not tokens or not all(0 <= t < self.model.args.vocab_size for t in tokens):
            raise ValueError("request %s: no tokens, or ids outside the vocabulary" % rid)
        if rid not in self.open:
            self.open[rid] = [self.model.begin_batch(1), 0]
        req = self.open[rid]
        toks = torch.tensor([tokens], dtype=torch.int64)
        logits, _ = self.model.step(toks, req[1], req[0], want=want)
        req[1] += len(tokens)
        return logits.reshape(-1, logits.shape[-1]).float().cpu()

    def end(self, rid):
        slots, _ = self.open.pop(rid)
        self.model.end_batch(slots)


def run(model, lines, out_dir, reply):
    rp = Replayer(model)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = [rp.entry(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        for rid in step.get("end", []):
            rp.end(rid)
        if any(len(p) for p in parts):
            data = torch.cat(parts).contiguous().numpy().astype("<f4")
            path = os.path.join(out_dir, "%d.f32" % step["step"])
            with open(path + ".part", "wb") as f:
                f.write(data.tobytes())
            os.replace(path + ".part", path)
        reply("done %d" % step["step"])


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="directory with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits of every step")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that open requests hold at any time")
    args = ap.parse_args(argv)
    model = registry.load(args.model, dtype=args.dtype, max_seq_len=args.max_tokens, max_batch_size=SLOTS)

    def reply(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    run(model, sys.stdin, args.out, reply)
    return 0
