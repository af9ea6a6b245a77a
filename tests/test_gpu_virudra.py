"""Virudra on the device against the NumPy restatement: every mechanism, prompts, decoding,
portions, batches, slots used again, far keys, bias and temperature edges, generation, the trace
runner."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import virudra_np as ref

import layered_checks as checks
import virudra_models as vm
from layered_checks import agree, assert_rows, decode_logits, greedy_oracle, prompt_logits

pytestmark = pytest.mark.gpu
both = pytest.mark.parametrize("serving", ["float32", "bfloat16"])
kernels = pytest.mark.parametrize("dim", [16, 64])   # (head sizes of both kernels of a portion)


def Limit(cfg, w, toks, want, serving):
    return checks.Limit(ref, cfg, w, toks, want, serving)


def decoder(ctx, cfg, w, serving, **settings):
    from quantibbler_b200 import virudra
    from quantibbler_b200.layered import LayeredDecoder
    settings = dict(dict(max_seq=512, prefill_chunk=64), **settings)
    t = vm.tensors(w)
    virudra.check_tensors(cfg, t)
    return LayeredDecoder(ctx, virudra.parse(cfg, serving=serving, **settings), t)


@both
@pytest.mark.parametrize("name", sorted(vm.MODELS))
def test_each_mechanism(gpu_ctx, name, serving):
    """The residual stream after every layer run and the logits: one prompt in one portion, then
    in short ones, then token by token."""
    cfg, rows = vm.MODELS[name]
    w = vm.weights(cfg, 11, rows)
    toks = vm.prompt(cfg, 75)
    per = []
    want = ref.forward(cfg, w, toks, per_layer=per)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=128)
    got = []
    dec.after_layer = lambda x: got.append(x.cpu().numpy())
    logits = prompt_logits(dec, toks)
    dec.after_layer = None
    assert len(got) == len(per)
    for i, (a, b) in enumerate(zip(got, per)):
        assert_rows(a, b, lim, f"after layer run {i}")
    assert_rows(logits, want, lim, "whole prompt")
    assert_rows(prompt_logits(dec, toks, portions=[2, 3, 1, 17, 2, 4, 30, 16]), want, lim, "portions")
    assert_rows(np.concatenate([prompt_logits(dec, toks[:1]), decode_logits(dec, toks[1:], 1)]), want, lim, "tokens")


@both
def test_portions_of_every_size(gpu_ctx, serving):
    """Portions down to two tokens and longer than the decoder's own pieces; nothing depends on
    where a prompt is cut."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 2, vm.MIXED_ROWS)
    toks = vm.prompt(cfg, 150)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=48)
    whole = prompt_logits(dec, toks)
    assert_rows(whole, want, lim, "whole")
    for size in (2, 3, 5, 16, 17, 31, 48, 64, 65, 130):
        cuts = [size] * (150 // size) + ([150 % size] if 150 % size else [])
        got = prompt_logits(dec, toks, portions=cuts)
        assert_rows(got, want, lim, f"portions of {size}")
        assert_rows(got, whole, lim, f"portions of {size} against one")


@both
def test_long_decoding(gpu_ctx, serving):
    """Several hundred decoded tokens: the splits of the keys and the bias table's end move along."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 4, vm.MIXED_ROWS)
    toks = vm.prompt(cfg, 340)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, max_seq=340)
    got = np.concatenate([prompt_logits(dec, toks[:20]), decode_logits(dec, toks[20:], 20)])
    assert_rows(got, want, lim)
    # decoding, a portion in between, decoding again
    got = np.concatenate([prompt_logits(dec, toks[:1]), decode_logits(dec, toks[1:30], 1),
                          dec.prefill(toks[30:65], 0, 30, want=range(35)).cpu().numpy(), decode_logits(dec, toks[65:80], 65)])
    rows = want.copy()
    rows[:80] = got
    assert_rows(rows, want, lim, "mixed")


@both
@pytest.mark.parametrize("batch", [3, 7, 20])
def test_batches_of_unequal_requests_and_slots_used_again(gpu_ctx, serving, batch):
    """Slots at different positions step together, some idle; a slot that a request has left is
    taken by another, also by one of a single token.  Every request as if it were alone.  What the
    caches hold before a request and behind its last position is never read."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 6, vm.MIXED_ROWS)
    dec = decoder(gpu_ctx, cfg, w, serving, max_batch=batch)
    for _, _, state in dec.runs:
        state.k.fill_(float("nan"))
        state.v.fill_(float("nan"))
    lengths = ([31, 5, 1, 64, 12, 2, 40] * 3)[:batch]
    known = {}
    for generation in range(2):
        seqs = [vm.prompt(cfg, n + 8, seed=100 * generation + s) for s, n in enumerate(lengths)]
        for s, t in enumerate(seqs):
            want = ref.forward(cfg, w, t)
            known[s] = want, Limit(cfg, w, t, want, serving)
        for s, n in enumerate(lengths):
            rows = known[s][0].copy()
            rows[:n] = prompt_logits(dec, seqs[s][:n], slot=s)
            assert_rows(rows, *known[s], f"prompt {s}")
        done = [0] * batch
        for step in range(12):
            live = [s for s in range(batch) if done[s] < 8 and (step + s) % 3 != 0]
            dec.start([seqs[s][lengths[s] + done[s]] if s in live else 0 for s in range(batch)],
                      [lengths[s] + done[s] if s in live else None for s in range(batch)])
            dec.step()
            dec.ctx.synchronize()
            out = dec.logits.cpu().numpy()
            for s in live:
                rows = known[s][0].copy()      # (errors relative to the spread of the whole sequence's rows)
                rows[lengths[s] + done[s]] = out[s]
                assert_rows(rows, *known[s], (generation, step, s))
                done[s] += 1
        assert min(done) == 8
        lengths = lengths[::-1]


def needle_model(bias_rows=12, strength=1.0, dim=16, **kw):
    """One attention layer in which every query looks for one token's key: channel 6 is the same
    for every token and makes the query, channel 5 marks the needle and makes its key; the needle's
    value stands out too."""
    cfg = vm.config([vm.bare(vm.attention(heads=4, kv_heads=2, dim=dim, vdim=dim, scale=1.0, **kw))], width=48, vocab=40)
    w = vm.weights(cfg, 9, bias_rows)
    needle = 7
    w["embed"][:, 5] = 0.0
    w["embed"][:, 6] = 6.0
    w["embed"][needle, 5] = 6.0
    w["l0.norm1"][:] = 0.0
    w["l0.mix.q"][:] *= 0.1
    w["l0.mix.q"][::dim] = 0.0
    w["l0.mix.q"][::dim, 6] = 2.0 * strength
    w["l0.mix.k"][:] *= 0.1
    w["l0.mix.k"][::dim] = 0.0
    w["l0.mix.k"][::dim, 5] = 1.0 * strength
    w["l0.mix.v"][:, 5] = 1.5
    w["l0.mix.rel"][:] = 0.0
    return cfg, {n: vm.bf16(a) for n, a in w.items()}, needle


@both
@kernels
def test_far_keys(gpu_ctx, serving, dim):
    """One key among hundreds, at every distance from the rows behind it: the attention finds it as
    a prompt, in portions and decoded (it would drop out of the row if any split, tile or page edge
    lost it; checked on the restatement)."""
    cfg, w, needle = needle_model(dim=dim, coef=0.0)
    base = [t if t != needle else 8 for t in vm.prompt(cfg, 400)]
    for at in (0, 1, 15, 16, 63, 64, 129):
        toks = list(base)
        toks[at] = needle
        want = ref.forward(cfg, w, toks)
        lim = Limit(cfg, w, toks, want, serving)
        blind = dict(w, **{"l0.mix.k": w["l0.mix.k"] * (np.arange(48) != 5)})
        moved = checks.row_errors(ref.forward(cfg, blind, toks), want)
        assert moved[at + 1:].min() > 2 * lim.value, "the test would not see a lost key"
        dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=256)
        assert_rows(prompt_logits(dec, toks), want, lim, f"prompt, {at}")
        assert_rows(prompt_logits(dec, toks, portions=[at + 1, 2, 199, 198 - at]), want, lim, f"portions, {at}")
        rows = want.copy()
        rows[:at + 1] = prompt_logits(dec, toks[:at + 1])
        rows[at + 1:at + 80] = decode_logits(dec, toks[at + 1:at + 80], at + 1)
        dec.prefill(toks[:380], 0, 0)
        rows[380:] = decode_logits(dec, toks[380:], 380)
        assert_rows(rows, want, lim, f"decoded, {at}")


def bucket_ranges(rows, bias_max):
    """{bucket: (first, last distance)}; the last one ends nowhere."""
    out = {}
    for n in range(4 * bias_max if bias_max < 100 else bias_max + 5):
        b = ref.bucket(n, rows, bias_max)
        out[b] = (out.get(b, (n, n))[0], n)
    return out


@both
@kernels
@pytest.mark.parametrize("rows,bias_max", [(12, 40), (7, 30), (32, 33), (2, 5), (9, 200)])
def test_bias_bucket_edges(gpu_ctx, serving, rows, bias_max, dim, monkeypatch):
    """One bucket at a time draws all the attention.  A bucket that began or ended a token off
    would move the rows whose distance to the needle lies at its edges (checked on the
    restatement); rows far behind it see only the last bucket."""
    cfg, w, needle = needle_model(rows, 0.0, dim=dim, bias_max=bias_max)
    toks = [t if t != needle else 8 for t in vm.prompt(cfg, 40 + 3 * min(bias_max, 100))]
    at = 30
    toks[at] = needle
    ranges = bucket_ranges(rows, bias_max)
    for b in sorted(ranges)[::1 if len(ranges) < 9 else 3] + [rows - 1]:
        first, last = ranges[b]
        w["l0.mix.rel"][:] = 0.0
        w["l0.mix.rel"][b] = 9.0
        want = ref.forward(cfg, w, toks)
        lim = Limit(cfg, w, toks, want, serving)
        bucket = ref.bucket
        for off, distance in ((1, first - 1), (-1, first)):
            if distance < 0:
                continue
            monkeypatch.setattr(ref, "bucket", lambda n, r, m, off=off: bucket(max(n + off, 0), r, m))
            moved = checks.row_errors(ref.forward(cfg, w, toks), want)
            monkeypatch.setattr(ref, "bucket", bucket)
            assert moved[at + distance] > 1.5 * lim.value, "the test would not see the edge"
        dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=256)
        assert_rows(prompt_logits(dec, toks), want, lim, f"prompt, bucket {b}")
        n = len(toks)
        assert_rows(prompt_logits(dec, toks, portions=[29, 2, 18, 5, n - 54]), want, lim, f"portions, bucket {b}")
        cut = max(1, min(at + first - 1, n - 5))
        got = want.copy()
        got[cut:cut + 5] = decode_after(dec, toks, cut, 5)
        assert_rows(got, want, lim, f"decoded, bucket {b}")


def decode_after(dec, toks, cut, n):
    """Logits of ``n`` tokens decoded behind a prompt of ``cut``."""
    dec.prefill(toks[:cut], 0, 0)
    return decode_logits(dec, toks[cut:cut + n], cut)


@both
@kernels
@pytest.mark.parametrize("every,coef", [(1, 0.7), (16, 3.0), (50, 3.0), (7.5, 2.0)])
def test_temperature_steps(gpu_ctx, serving, every, coef, dim, monkeypatch):
    """The factor on the queries steps at positions every k - 1: a step one position off would move
    those rows (checked on the restatement)."""
    cfg, w, needle = needle_model(strength=0.2, dim=dim, every=every, coef=coef)
    toks = vm.prompt(cfg, 130)
    toks[3] = needle
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    true = ref.query_temperature
    monkeypatch.setattr(ref, "query_temperature", lambda p, c, e: true(p - 1, c, e))
    moved = checks.row_errors(ref.forward(cfg, w, toks), want)
    monkeypatch.setattr(ref, "query_temperature", true)
    if every > 1:
        step = int(np.ceil(every)) - 1
        assert moved[step] > 2 * lim.value, "the test would not see the step"
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=256)
    assert_rows(prompt_logits(dec, toks), want, lim, "prompt")
    assert_rows(np.concatenate([prompt_logits(dec, toks[:5]), decode_logits(dec, toks[5:], 5)]), want, lim, "decoded")


@both
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5])
def test_first_tokens(gpu_ctx, serving, n):
    cfg = vm.mixed()
    w = vm.weights(cfg, 17, vm.MIXED_ROWS)
    toks = vm.prompt(cfg, 40, seed=n)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving)
    rows = want.copy()
    rows[:n + 3] = np.concatenate([prompt_logits(dec, toks[:n]), decode_logits(dec, toks[n:n + 3], n)])
    assert_rows(rows, want, lim)


@both
def test_longer_sequences_at_wider_sizes(gpu_ctx, serving):
    """Several tiles of every matrix form, experts with more than one tile of rows and experts with
    none (the tables name only some)."""
    layers = [vm.dense(vm.attention(heads=8, kv_heads=2, dim=64, vdim=48, bias_max=150, every=60), 352),
              vm.moe(vm.attention(heads=6, kv_heads=3, dim=128, vdim=128, bias_max=90, every=100), 160, 9, 2)]
    cfg = vm.config(layers, width=320, vocab=700, loop=(0, 2, 2))
    w = vm.weights(cfg, 8, 32)
    rng = np.random.default_rng(1)   # most tokens share expert 0, nobody has expert 7
    w["l1.mlp.table"][:] = [[0, rng.choice([1, 2, 8])] if t % 4 else rng.permutation([3, 4, 5, 6])[:2] for t in range(700)]
    toks = vm.prompt(cfg, 330)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=512)
    assert_rows(prompt_logits(dec, toks), want, lim, "whole")
    assert_rows(prompt_logits(dec, toks, portions=[129, 66, 135]), want, lim, "portions")
    got = np.concatenate([prompt_logits(dec, toks[:300]), decode_logits(dec, toks[300:], 300)])
    assert_rows(got, want, lim, "decoded")


@both
def test_greedy_generation(gpu_ctx, serving):
    cfg = vm.mixed()
    w = vm.weights(cfg, 13, vm.MIXED_ROWS)
    for n in (1, 23):
        prompt = vm.prompt(cfg, n, seed=n)
        want = greedy_oracle(ref, cfg, w, prompt, 12)
        dec = decoder(gpu_ctx, cfg, w, serving)
        out = dec.generate(prompt, 12)
        assert out["finish"] == "length" and out["prompt_tokens"] == n
        agree(out["completion_tokens"], want, serving)
        # the same through a captured graph: the capture moves no sequence on
        dec.prefill(prompt, 0, 0)
        first = int(dec.best_idx[0].item())
        dec.advance()
        dec._host_positions = [n]
        dec.capture()
        rest = dec.decode(11)[:, 0]
        assert [first] + [int(t) for t in rest] == out["completion_tokens"]
        eos = out["completion_tokens"][3]
        stopped = dec.generate(prompt, 12, eos_token_id=eos)
        assert stopped["finish"] == "stop" and eos not in stopped["completion_tokens"]


@both
def test_batched_greedy_decode_through_a_graph(gpu_ctx, serving):
    """Six prompts of different lengths, decoded together by the replayed step: the choices are
    sorted by expert inside the graph."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 14, vm.MIXED_ROWS)
    dec = decoder(gpu_ctx, cfg, w, serving, max_batch=6)
    prompts = [vm.prompt(cfg, n, seed=n) for n in (3, 30, 9, 64, 17, 1)]
    for s, p in enumerate(prompts):
        dec.prefill(p, s, 0)
    first = dec.best_idx.cpu().numpy().copy()
    dec.advance()
    dec._host_positions = [len(p) for p in prompts]
    dec.capture()
    rest = dec.decode(8)
    for s, p in enumerate(prompts):
        agree([int(first[s])] + [int(t) for t in rest[:, s]], greedy_oracle(ref, cfg, w, p, 9), serving)


def test_refusals(gpu_ctx):
    cfg, rows = vm.MODELS["mixed"]
    dec = decoder(gpu_ctx, cfg, vm.weights(cfg, 0, rows), "float32", max_seq=32)
    with pytest.raises(ValueError, match="does not fit"):
        dec.prefill(list(range(33)), 0, 0)
    with pytest.raises(ValueError, match="does not fit"):
        dec.start([1], [32])
    with pytest.raises(ValueError, match="sequence slot 1"):
        dec.prefill([1], 1, 0)


@both
def test_trace_runner(gpu_ctx, tmp_path, serving):
    """The runner as a program: requests one after the other and two at a time."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 21, vm.MIXED_ROWS)
    vm.write_model(tmp_path / "model", cfg, w)
    a, b = vm.prompt(cfg, 40, 1), vm.prompt(cfg, 25, 2)
    want = {"a": ref.forward(cfg, w, a), "b": ref.forward(cfg, w, b)}
    toks, at = {"a": a, "b": b}, {"a": 0, "b": 0}
    lims = {name: Limit(cfg, w, toks[name], want[name], serving) for name in toks}
    plan = [[("a", 20)], [("b", 7), ("a", 2)], [("a", 1), ("b", 1)], [("b", 17)], [("a", 17)]]
    lines, rows = [], []
    for n, entries in enumerate(plan):
        es, r = [], []
        for name, k in entries:
            want_at = [i for i in range(k) if (at[name] + i) % 3 != 1]
            es.append({"id": name, "tokens": toks[name][at[name]:at[name] + k], "want": want_at})
            r += [(name, at[name] + i) for i in want_at]
            at[name] += k
        lines.append(json.dumps({"step": n, "entries": es, "end": [x for x, _ in entries if at[x] == len(toks[x])]}))
        rows.append(r)
    # the slot of a request that has ended serves another one
    lines.append(json.dumps({"step": 5, "entries": [{"id": "c", "tokens": b, "want": [24]}], "end": ["c"]}))
    rows.append([("b", 24)])
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"),
                        "--dtype", serving, "--out", str(out), "--max-tokens", "80", "--slots", "2"],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert p.stdout.split("\n")[:6] == [f"done {n}" for n in range(6)]
    for n, r in enumerate(rows):
        path = out / f"{n}.f32"
        if not r:
            assert not path.exists()
            continue
        got = np.fromfile(path, "<f4").reshape(len(r), cfg["vocab"])
        for (name, i), row in zip(r, got):
            rows_of = want[name].copy()
            rows_of[i] = row
            assert_rows(rows_of, want[name], lims[name], f"step {n}")


def test_command_line_generates(gpu_ctx, tmp_path):
    cfg = vm.mixed()
    w = vm.weights(cfg, 22, vm.MIXED_ROWS)
    vm.write_model(tmp_path, cfg, w)
    prompt = vm.prompt(cfg, 19)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([sys.executable, "-m", "quantibbler_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                        "--prompt", ",".join(map(str, prompt)), "--max-tokens", "6"], cwd=root, capture_output=True,
                       text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    out = json.loads(p.stdout)
    assert out["prompt_tokens"] == 19 and out["finish"] == "length"
    agree(out["completion_tokens"], greedy_oracle(ref, cfg, w, prompt, 6), "float32")
