"""What the tests of layered decoders share: row errors and their limits, logits of prompts,
portions and decoded tokens, greedy continuations of a restatement."""

import numpy as np

from vogizen_models import bf16


def row_errors(got, want):
    """Root-mean-square difference of each row, relative to the spread of the expected rows."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return np.sqrt(((got - want) ** 2).mean(axis=-1)) / want.std()


class Limit:
    """What a model's rows may differ by: in float32 a constant, in bfloat16 twice what rounding
    the linears' inputs alone does to the worst row of the restatement ``ref``."""

    def __init__(self, ref, cfg, w, toks, want, serving):
        self.value = 2e-5
        if serving == "bfloat16":
            with ref.rounded_operands(bf16):
                self.value = 2 * row_errors(ref.forward(cfg, w, toks), want).max()
            assert self.value < 0.12, "too sensitive a model to tell a fault from rounding"


def assert_rows(got, want, limit, what=""):
    err = row_errors(got, want)
    assert np.isfinite(err).all() and err.max() <= limit.value, (what, int(err.argmax()), float(err.max()), limit.value)


def prompt_logits(dec, toks, slot=0, portions=None):
    """Logits of every position, the tokens fed in the given portions."""
    out, at = [], 0
    for n in portions or [len(toks)]:
        out.append(dec.prefill(toks[at:at + n], slot, at, want=range(n)).cpu().numpy())
        at += n
    assert at == len(toks)
    return np.concatenate(out)


def decode_logits(dec, toks, at, slot=0):
    """Logits of tokens at positions ``at`` .., one batched step each."""
    out = []
    B = dec.cfg.max_batch
    for i, t in enumerate(toks):
        dec.start([t if s == slot else 0 for s in range(B)], [at + i if s == slot else None for s in range(B)])
        dec.step()
        dec.ctx.synchronize()
        out.append(dec.logits[slot].cpu().numpy())
    return np.stack(out)


def greedy_oracle(ref, cfg, w, prompt, n):
    """Continuation and, per token, how far the choice was ahead of the second best."""
    toks, out = list(prompt), []
    for _ in range(n):
        row = ref.forward(cfg, w, toks)[-1]
        best = int(row.argmax())
        out.append((best, float(row[best] - np.partition(row, -2)[-2]) / row.std()))
        toks.append(best)
    return out


def agree(got, want, serving):
    for g, (best, lead) in zip(got, want):
        if g != best:
            assert lead < (1e-4 if serving == "float32" else 0.1), (got, want)
            return
    assert len(got) == len(want)
