"""Vogizen on the device against the NumPy restatement: every mechanism, prompts, decoding,
portions, batches, slots used again, window edges, generation, the trace runner."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import vogizen_np as ref

import layered_checks as checks
import vogizen_models as vm
from layered_checks import agree, assert_rows, decode_logits, greedy_oracle, prompt_logits

pytestmark = pytest.mark.gpu


def Limit(cfg, w, toks, want, serving):
    return checks.Limit(ref, cfg, w, toks, want, serving)


def decoder(ctx, cfg, w, serving, **settings):
    from quantibbler_b200 import vogizen
    from quantibbler_b200.layered import LayeredDecoder
    settings = dict(dict(max_seq=512, prefill_chunk=64), **settings)
    return LayeredDecoder(ctx, vogizen.parse(cfg, serving=serving, **settings), vm.tensors(w))


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(vm.MODELS))
def test_each_mechanism(gpu_ctx, name, serving):
    """The residual stream after every layer run and the logits: one prompt in one portion, then
    in short ones, then token by token."""
    cfg = vm.MODELS[name]
    w = vm.weights(cfg, 11)
    toks = vm.prompt(cfg, 45)
    per = []
    want = ref.forward(cfg, w, toks, per_layer=per)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving)
    got = []
    dec.after_layer = lambda x: got.append(x.cpu().numpy())
    logits = prompt_logits(dec, toks)
    dec.after_layer = None
    assert len(got) == len(per)
    for i, (a, b) in enumerate(zip(got, per)):
        assert_rows(a, b, lim, f"after layer run {i}")
    assert_rows(logits, want, lim, "whole prompt")
    assert_rows(prompt_logits(dec, toks, portions=[2, 3, 1, 17, 2, 4, 16]), want, lim, "portions")
    assert_rows(np.concatenate([prompt_logits(dec, toks[:1]), decode_logits(dec, toks[1:], 1)]), want, lim, "tokens")


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
def test_portions_of_every_size(gpu_ctx, serving):
    """Portions down to two tokens, longer than the window and longer than the decoder's own
    pieces; nothing depends on where a prompt is cut."""
    cfg = vm.mixed(size=21)
    w = vm.weights(cfg, 2)
    toks = vm.prompt(cfg, 150)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=48)
    whole = prompt_logits(dec, toks)
    assert_rows(whole, want, lim, "whole")
    for size in (2, 3, 5, 16, 17, 21, 64, 65, 130):
        cuts = [size] * (150 // size) + ([150 % size] if 150 % size else [])
        got = prompt_logits(dec, toks, portions=cuts)
        assert_rows(got, want, lim, f"portions of {size}")
        assert_rows(got, whole, lim, f"portions of {size} against one")


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
def test_long_decoding_wraps_the_ring(gpu_ctx, serving):
    """A ring of 9 - 1 + 8 rows, 120 decoded tokens: every row is overwritten many times."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 4)
    toks = vm.prompt(cfg, 140)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=8)
    got = np.concatenate([prompt_logits(dec, toks[:20]), decode_logits(dec, toks[20:], 20)])
    assert_rows(got, want, lim)
    # decoding, a portion in between, decoding again
    got = np.concatenate([prompt_logits(dec, toks[:1]), decode_logits(dec, toks[1:30], 1),
                          dec.prefill(toks[30:65], 0, 30, want=range(35)).cpu().numpy(), decode_logits(dec, toks[65:80], 65)])
    assert_rows(got, want[:80], lim, "mixed")


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [3, 7])
def test_batches_of_unequal_requests_and_slots_used_again(gpu_ctx, serving, batch):
    """Slots at different positions step together, some idle; a slot that a request has left is
    taken by another, also by one of a single token.  Every request as if it were alone."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 6)
    dec = decoder(gpu_ctx, cfg, w, serving, max_batch=batch)
    lengths = [31, 5, 1, 64, 12, 2, 40][:batch]
    for generation in range(2):
        seqs = [vm.prompt(cfg, n + 12, seed=100 * generation + s) for s, n in enumerate(lengths)]
        want = [ref.forward(cfg, w, t) for t in seqs]
        lims = [Limit(cfg, w, t, x, serving) for t, x in zip(seqs, want)]
        for s, n in enumerate(lengths):
            assert_rows(prompt_logits(dec, seqs[s][:n], slot=s), want[s][:n], lims[s], f"prompt {s}")
        done = [0] * batch
        for step in range(18):
            live = [s for s in range(batch) if done[s] < 12 and (step + s) % 3 != 0]
            dec.start([seqs[s][lengths[s] + done[s]] if s in live else 0 for s in range(batch)],
                      [lengths[s] + done[s] if s in live else None for s in range(batch)])
            dec.step()
            dec.ctx.synchronize()
            out = dec.logits.cpu().numpy()
            for s in live:
                rows = want[s].copy()      # (errors relative to the spread of the whole sequence's rows)
                rows[lengths[s] + done[s]] = out[s]
                assert_rows(rows, want[s], lims[s], (generation, step, s))
                done[s] += 1
        assert min(done) == 12
        lengths = lengths[::-1]


def needle_model(size):
    """One attention layer in which every query looks for one token's key: channel 6 is the same
    for every token and makes the query, channel 5 marks the needle and makes its key."""
    cfg = vm.config([vm.mlp(vm.attention(heads=2, dim=16, vdim=16, kv_rank=16, q_rank=16, size=size, scale=1.0))],
                    side=None, width=48, vocab=40, scale=1.0)
    w = vm.weights(cfg, 9)
    needle = 7
    e = np.zeros(48, np.float32)
    e[5] = 12.0
    w["embed"][:, 5] = 0.0
    w["embed"][:, 6] = 8.0
    w["embed"][needle] = w["embed"][needle] + e
    w["l0.norm1"][:] = 1.0
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, 5] = 8.0        # latent 0: the needle
    w["l0.mix.dkv"][1:] *= 0.5
    w["l0.mix.dkv.norm"][:] = 1.0
    w["l0.mix.uk"][:] *= 0.05
    w["l0.mix.uk"][::16, 0] = 2.0      # the first key entry of each head
    w["l0.mix.dq"][0] = 0.0
    w["l0.mix.dq"][0, 6] = 8.0
    w["l0.mix.dq.norm"][:] = 1.0
    w["l0.mix.uq"][:] *= 0.05
    w["l0.mix.uq"][::16, 0] = 2.0
    return cfg, {n: vm.bf16(a) for n, a in w.items()}, needle


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [1, 2, 33, 70, 128])
def test_window_edges(gpu_ctx, size, serving):
    """The needle just inside and just outside the window, in prompts, portions and decoding: a
    window one token off would move the row by much more than the limit (checked on the oracle)."""
    cfg, w, needle = needle_model(size)
    toks = [t if t != needle else 8 for t in vm.prompt(cfg, 200)]
    toks[20] = needle
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    inside, outside = 20 + size - 1, 20 + size
    wrong = json.loads(json.dumps(cfg))
    for off, row in ((1, outside), (-1, inside)):
        if size + off < 1:
            continue
        wrong["layers"][0]["mixer"]["mask"]["size"] = size + off
        moved = ref.forward(wrong, w, toks)[row] - want[row]
        assert np.sqrt((moved ** 2).mean()) > 1.2 * lim.value * want.std(), "the test would not see the edge"
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=256)
    assert_rows(prompt_logits(dec, toks), want, lim, "prompt")
    assert_rows(prompt_logits(dec, toks, portions=[19, 2, size, 179 - size]), want, lim, "portions")
    cut = inside - 1
    got = np.concatenate([prompt_logits(dec, toks[:cut]), decode_logits(dec, toks[cut:cut + 4], cut)])
    assert_rows(got, want[:cut + 4], lim, "decoded")


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
def test_longer_sequences_at_wider_sizes(gpu_ctx, serving):
    """Several tiles of every matrix form: more than 64 and more than 128 rows, several key tiles."""
    layers = [vm.mlp(vm.attention(heads=4, dim=64, vdim=48, kv_rank=192, q_rank=160, size=100), 352),
              vm.mlp(vm.delta(heads=8, kv_heads=4, dim=64, vdim=40, conv=4))]
    cfg = vm.config(layers, width=320, vocab=700, loop=(0, 2, 2), side=40)
    w = vm.weights(cfg, 8)
    toks = vm.prompt(cfg, 330)
    want = ref.forward(cfg, w, toks)
    lim = Limit(cfg, w, toks, want, serving)
    dec = decoder(gpu_ctx, cfg, w, serving, prefill_chunk=512)
    assert_rows(prompt_logits(dec, toks), want, lim, "whole")
    assert_rows(prompt_logits(dec, toks, portions=[129, 66, 135]), want, lim, "portions")
    got = np.concatenate([prompt_logits(dec, toks[:300]), decode_logits(dec, toks[300:], 300)])
    assert_rows(got, want, lim, "decoded")


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
def test_greedy_generation(gpu_ctx, serving):
    cfg = vm.mixed()
    w = vm.weights(cfg, 13)
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


def test_batched_greedy_decode_through_a_graph(gpu_ctx):
    """Five prompts of different lengths, decoded together by the replayed step."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 14)
    dec = decoder(gpu_ctx, cfg, w, "float32", max_batch=5)
    prompts = [vm.prompt(cfg, n, seed=n) for n in (3, 30, 9, 64, 17)]
    for s, p in enumerate(prompts):
        dec.prefill(p, s, 0)
    first = dec.best_idx.cpu().numpy().copy()
    dec.advance()
    dec._host_positions = [len(p) for p in prompts]
    dec.capture()
    rest = dec.decode(8)
    for s, p in enumerate(prompts):
        agree([int(first[s])] + [int(t) for t in rest[:, s]], greedy_oracle(ref, cfg, w, p, 9), "float32")


def test_refusals(gpu_ctx):
    cfg = vm.MODELS["mixed"]
    dec = decoder(gpu_ctx, cfg, vm.weights(cfg), "float32", max_seq=32)
    with pytest.raises(ValueError, match="does not fit"):
        dec.prefill(list(range(33)), 0, 0)
    with pytest.raises(ValueError, match="wanted places"):
        dec.prefill([1, 2, 3], 0, 0, want=[3])
    with pytest.raises(ValueError, match="sequence slot 1"):
        dec.prefill([1], 1, 0)
    from quantibbler_b200.trace import Replay
    replay = Replay(dec)
    replay.feed("a", [1, 2], [])
    with pytest.raises(ValueError, match="all 1 slots are in use"):
        replay.feed("b", [1], [])
    with pytest.raises(ValueError, match="out of range"):
        replay.feed("a", [cfg["vocab"]], [])


@pytest.mark.parametrize("serving", ["float32", "bfloat16"])
def test_trace_runner(gpu_ctx, tmp_path, serving):
    """The runner as a program: requests one after the other and two at a time."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 21)
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
            want[name][i], expected = row, want[name].copy()
            assert_rows(want[name], expected, lims[name], f"step {n}")
            want[name] = expected


def test_command_line_generates(gpu_ctx, tmp_path):
    cfg = vm.mixed()
    w = vm.weights(cfg, 22)
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
