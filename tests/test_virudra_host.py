"""Virudra without a GPU: the restatement's mechanisms against independent formulas, the distance
buckets, config and tensor checks, and that the restatement reacts to the faults the device tests
look for."""

import json

import numpy as np
import pytest

from oracle import virudra_np as ref
from quantibbler_b200 import safetensors, virudra
from quantibbler_b200.layers import distance_buckets

import virudra_models as vm


def copy(cfg):
    return json.loads(json.dumps(cfg))


@pytest.mark.parametrize("rows,bias_max", [(2, 2), (2, 9), (7, 9), (13, 40), (32, 33), (32, 500), (80, 44), (16, 128), (9, 1000)])
def test_distance_buckets(rows, bias_max):
    """The product's table up to where it ends, against the formula and its edges solved for n."""
    got = distance_buckets(rows, bias_max)
    assert got[-1] == rows - 1 and (len(got) == 1 or got[-2] < rows - 1)
    for n in range(3 * bias_max + 100):
        assert got[min(n, len(got) - 1)] == ref.bucket(n, rows, bias_max), n
    half = rows // 2
    assert got[:half] == tuple(range(half))
    for n, b in enumerate(got[half:], half):
        k = b - half    # n >= half * (bias_max / half) ** (k / (rows - half))
        assert n >= half * (bias_max / half) ** (k / (rows - half)) * (1 - 1e-9)
        if b < rows - 1:
            assert n < half * (bias_max / half) ** ((k + 1) / (rows - half)) * (1 + 1e-9)
    assert len(got) <= bias_max + 1


@pytest.mark.parametrize("rows,bias_max", [(1, 10), (0, 10), (16, 8), (16, 3)])
def test_distance_buckets_refusals(rows, bias_max):
    with pytest.raises(ValueError, match="distance bias"):
        distance_buckets(rows, bias_max)


def test_attention_row_by_row():
    """One head and row at a time, the temperature on the scores, the bias beside them."""
    m = vm.attention(heads=4, kv_heads=2, dim=3, vdim=5, bias_max=9, coef=0.5, every=4)["mixer"]
    rng = np.random.default_rng(0)
    w = {"q": rng.standard_normal((12, 7)), "k": rng.standard_normal((6, 7)), "v": rng.standard_normal((10, 7)),
         "rel": rng.standard_normal((6, 4)), "o": rng.standard_normal((7, 20))}
    h = rng.standard_normal((15, 7))
    got, p = ref.attention(h, m, w, return_weights=True)
    for i in (0, 1, 3, 4, 14):
        heads = []
        for a in range(4):
            g = a // 2
            factor = 1 + 0.5 * np.log((i + 1) // 4 + 1)
            s = [factor * m["scale"] * (w["q"][3 * a:3 * a + 3] @ h[i]) @ (w["k"][3 * g:3 * g + 3] @ h[j])
                 + w["rel"][[0, 1, 2, 3, 3, 4, 4, 5, 5, 5][min(i - j, 9)], a] for j in range(i + 1)]
            e = np.exp(s)
            np.testing.assert_allclose(p[a, i, :i + 1], e / e.sum())
            assert not p[a, i, i + 1:].any()
            heads.append(sum(x * (w["v"][5 * g:5 * g + 5] @ h[j]) for j, x in enumerate(e / e.sum())))
        np.testing.assert_allclose(got[i], w["o"] @ np.concatenate(heads))


def test_temperature_norm_cap_activations():
    assert ref.query_temperature(0, 0.7, 50) == 1.0 and ref.query_temperature(48, 0.7, 50) == 1.0
    assert ref.query_temperature(49, 0.7, 50) == 1 + 0.7 * np.log(2)
    assert ref.query_temperature(99, 0.7, 50) == 1 + 0.7 * np.log(3)
    assert ref.query_temperature(0, 2.0, 1) == 1 + 2 * np.log(2)
    x = np.array([[1.0, 2.0, 6.0]])
    np.testing.assert_allclose(ref.rms_norm(x, 0.25, 0.5), 1.25 * x / np.sqrt(41 / 3 + 0.5))
    np.testing.assert_allclose(ref.softcap(np.array([0.0, 3.0, -1e9]), 3.0), [0, 3 * np.tanh(1), -3])
    np.testing.assert_allclose(ref.silu(np.array([0.0, 2.0])), [0, 2 / (1 + np.exp(-2))])
    np.testing.assert_allclose(ref.gelu_tanh(np.array([1.0])), 0.8411919906082768)


def test_table_mixture_weighs_its_experts_the_same():
    cfg, rows = vm.MODELS["moe"]
    w = {n[len("l0.mlp."):]: a for n, a in vm.weights(cfg, 0, rows).items() if n.startswith("l0.mlp.")}
    h = np.random.default_rng(0).standard_normal((4, cfg["width"]))
    got = ref.table_mixture(h, [5, 90, 5, 0], cfg["layers"][0]["mlp"]["router"], w)
    for t, token in enumerate([5, 90, 5, 0]):
        a, b = w["table"][token]
        want = sum(w[f"e{e}.down"] @ (ref.silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])) for e in (a, b)) / 2
        np.testing.assert_allclose(got[t], want)


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (1, 3, 2), (2, 4, 3), (3, 4, 2)])
def test_run_order(loop):
    cfg = vm.mixed(loop=loop)
    assert [i for i, _ in virudra.parse(cfg).run_order()] == ref.run_order(cfg)


@pytest.mark.parametrize("name", sorted(vm.MODELS))
def test_shapes_match_the_models(name):
    cfg, rows = vm.MODELS[name]
    w = vm.weights(cfg, 0, rows)
    shapes = virudra.shapes(cfg)
    assert set(shapes) == set(w)
    virudra.check_tensors(cfg, vm.tensors(w))


def test_config_is_read():
    c = virudra.parse(vm.mixed(), serving="float32", max_batch=3)
    assert (c.vocab, c.width, c.norm_eps, c.logit_softcap, c.loop, c.max_batch) == (97, 72, 1e-5, 9.0, (1, 3, 2), 3)
    assert c.post_norms and c.norm_offset == 1.0
    assert c.layers[1].sizes["temperature"] == (0.4, 3.0) and c.layers[1].sizes["bias_max"] == 30
    assert [x.experts for x in c.layers] == [None, 5, None, 7]
    assert [x.activation for x in c.layers] == ["gelu_tanh", "silu", None, "silu"]
    assert virudra.parse({k: v for k, v in vm.mixed().items() if k not in ("loop", "logit_softcap")}).loop is None


def test_config_refusals():
    with pytest.raises(virudra.ConfigError, match="missing key 'vocab'"):
        virudra.parse({k: v for k, v in vm.mixed().items() if k != "vocab"})
    for change, text in ((lambda c: c["layers"][0].update(type="delta"), "unknown mixer type 'delta'"),
                         (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward kind"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads over 4"),
                         (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "6 of 5 experts"),
                         (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "query temperature"),
                         (lambda c: c["loop"].update(stop=9), "loop over layers 1..9")):
        bad = copy(vm.mixed())
        change(bad)
        with pytest.raises(virudra.ConfigError, match=text):
            virudra.parse(bad)


def test_tensor_refusals():
    cfg = vm.mixed()

    def check(change, text):
        t = vm.tensors(vm.weights(cfg, 0, vm.MIXED_ROWS))
        change(t)
        with pytest.raises(virudra.ConfigError, match=text):
            virudra.check_tensors(cfg, t)

    check(lambda t: t.pop("l1.mlp.e3.up"), "missing tensor 'l1.mlp.e3.up'")
    check(lambda t: t.update({"l0.mix.o": t["l0.mix.o"][:-1]}), "l0.mix.o")
    check(lambda t: t.update({"l0.mix.rel": t["l0.mix.rel"][:, :-1]}), "l0.mix.rel")
    check(lambda t: t.update({"l0.mix.rel": t["l0.mix.rel"][:1]}), "distance bias")
    check(lambda t: t["l1.mlp.table"].fill_(5), "outside 0..4")
    check(lambda t: t["l1.mlp.table"].fill_(-1), "outside 0..4")
    check(lambda t: t["l1.mlp.table"].fill_(1), "twice")
    check(lambda t: t.update({"l1.mlp.table": t["l1.mlp.table"].float()}), "integers")


def test_integer_tensors_round_trip(tmp_path):
    cfg = vm.mixed()
    w = vm.weights(cfg, 5, vm.MIXED_ROWS)
    vm.write_model(tmp_path, cfg, w)
    got = safetensors.load(tmp_path / "model.safetensors")
    assert set(got) == set(w)
    for n, a in w.items():
        np.testing.assert_array_equal(got[n].numpy() if a.dtype.kind == "i" else got[n].float().numpy(), a)


def test_the_oracle_sees_the_faults_the_device_tests_look_for(monkeypatch):
    """A bias bucket or a temperature step off by one, a missing pass, cap or norm offset, another
    token's experts: each moves the restatement's logits by far more than the device tests allow."""
    cfg = vm.mixed()
    w = vm.weights(cfg, 3, vm.MIXED_ROWS)
    toks = vm.prompt(cfg, 40)
    base = ref.forward(cfg, w, toks)

    def moved(other=cfg, weights=w):
        d = ref.forward(other, weights, toks)[20:] - base[20:]
        return np.sqrt((d ** 2).mean(axis=1)).max() / base.std()

    for change in (lambda c: c["loop"].update(times=1), lambda c: c.update(logit_softcap=1e9),
                   lambda c: c["layers"][0]["mixer"].update(bias_max=20),
                   lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=2),
                   lambda c: c["layers"][2]["mixer"]["q_temp"].update(coef=0.0)):
        other = copy(cfg)
        change(other)
        assert moved(other) > 0.02
    assert moved(weights=dict(w, **{"l3.mlp.table": np.roll(w["l3.mlp.table"], 1, axis=0)})) > 0.02
    assert moved(weights=dict(w, **{"l2.norm1b": w["l2.norm1b"] - 1})) > 0.02
    bucket = ref.bucket
    monkeypatch.setattr(ref, "bucket", lambda n, r, m: bucket(n + 1, r, m))
    assert moved() > 0.02
