"""Replays a trace of token ids through a model, step by step, and writes logits.

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

An entry brings the next tokens of a request; ``want`` names the places among them whose logits
are asked for; ``end`` lists the requests that are finished after the step.  The logits of a step
go to OUT/<step>.f32 (little-endian float32, [wanted, vocab]); after every step the line
``done <step>`` is printed.  Nothing is sampled.  A request holds a slot of the decoder from its
first tokens to its end; a single further token goes through the decoder's batched step, more
tokens through its prompt path.
"""

from __future__ import annotations

import argparse
import json
import os
import sys


class Replay:
    """Requests over a decoder's slots."""

    def __init__(self, decoder):
        self.decoder = decoder
        self.free = list(range(decoder.cfg.max_batch))[::-1]
        self.slot, self.length = {}, {}

    def feed(self, name, tokens, want):
        """The request's next tokens; returns the wanted logits [len(want), vocab] (numpy)."""
        import numpy as np
        dec = self.decoder
        for tok in tokens:
            if not 0 <= int(tok) < dec.cfg.vocab:
                raise ValueError(f"token id {tok} out of range (vocab {dec.cfg.vocab})")
        if name not in self.slot:
            if not self.free:
                raise ValueError(f"request {name!r}: all {dec.cfg.max_batch} slots are in use")
            self.slot[name], self.length[name] = self.free.pop(), 0
        slot, at = self.slot[name], self.length[name]
        if not tokens:
            return np.zeros((0, dec.cfg.vocab), np.float32)
        if len(tokens) == 1 and at > 0:
            ids, positions = [0] * dec.cfg.max_batch, [None] * dec.cfg.max_batch
            ids[slot], positions[slot] = int(tokens[0]), at
            dec.start(ids, positions)
            dec.step()
            dec.ctx.synchronize()
            logits = dec.logits[slot:slot + 1][[0] * len(want)]
        else:
            logits = dec.prefill(tokens, seq=slot, first_position=at, want=want)
        self.length[name] = at + len(tokens)
        return logits.cpu().numpy().astype("<f4", copy=False)

    def end(self, name):
        if name in self.slot:
            self.free.append(self.slot.pop(name))
            del self.length[name]


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at a time")
    ap.add_argument("--slots", type=int, default=1, help="requests that may be live at a time")
    a = ap.parse_args(argv)
    import numpy as np

    from .gpu import GpuContext
    from .registry import load_decoder
    decoder = load_decoder(GpuContext.init(), a.model, serving=a.dtype, max_batch=a.slots,
                           max_seq=max(a.max_tokens, 16))
    replay = Replay(decoder)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        out = [replay.feed(e["id"], e["tokens"], e.get("want") or []) for e in step["entries"]]
        out = [o for o in out if len(o)]
        if out:
            np.concatenate(out).tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for name in step.get("end") or []:
            replay.end(name)
        print(f"done {step['step']}", flush=True)
    return 0
