"""Vogizen without a GPU: the restatement's mechanisms against independent formulas, config and
tensor checks, the safetensors reader, the order of looped layers."""

import json

import numpy as np
import pytest

from oracle import vogizen_np as ref
from quantibbler_b200 import registry, safetensors, vogizen

import vogizen_models as vm


def test_delta_rule_is_the_recurrence_written_as_one_matrix():
    """S_t = g (I - beta k k^T) S_{t-1} + beta k v^T, read out after the write."""
    rng = np.random.default_rng(3)
    T, dim, vdim = 11, 5, 7
    q, k = rng.standard_normal((2, T, dim))
    v = rng.standard_normal((T, vdim))
    beta, decay = rng.uniform(0, 1, (2, T))
    out, state = ref.delta_rule(q, k, v, beta, decay)
    S = np.zeros((dim, vdim))
    for t in range(T):
        S = decay[t] * (np.eye(dim) - beta[t] * np.outer(k[t], k[t])) @ S + beta[t] * np.outer(k[t], v[t])
        np.testing.assert_allclose(out[t], q[t] @ S, atol=1e-12)
    np.testing.assert_allclose(state, S, atol=1e-12)
    again, _ = ref.delta_rule(q[6:], k[6:], v[6:], beta[6:], decay[6:],
                              ref.delta_rule(q[:6], k[:6], v[:6], beta[:6], decay[:6])[1])
    np.testing.assert_allclose(again, out[6:], atol=1e-12)


def test_causal_conv_and_window():
    x = np.arange(10.0)[:, None] ** 2
    taps = np.array([[3.0, 5.0, 7.0]])
    want = [7 * x[t, 0] + 5 * (x[t - 1, 0] if t else 0) + 3 * (x[t - 2, 0] if t > 1 else 0) for t in range(10)]
    np.testing.assert_allclose(ref.causal_conv(x, taps)[:, 0], want)
    cfg = vm.MODELS["attention"]
    w = {n[len("l0.mix."):]: a for n, a in vm.weights(cfg).items() if n.startswith("l0.mix.")}
    h = np.random.default_rng(0).standard_normal((30, cfg["width"]))
    _, p = ref.latent_attention(h, cfg["layers"][0]["mixer"], w, 1e-5, return_weights=True)
    size = cfg["layers"][0]["mixer"]["mask"]["size"]
    for i in range(30):
        seen = np.nonzero(p[0, i] > 0)[0]
        assert list(seen) == list(range(max(0, i - size + 1), i + 1))


def test_sinusoid_and_norms():
    s = ref.sinusoid([0, 3], 7)
    np.testing.assert_allclose(s[0], [0, 1, 0, 1, 0, 1, 0])
    np.testing.assert_allclose(s[1, 2], np.sin(3 * 10000 ** (-2 / 7)))
    np.testing.assert_allclose(s[1, 3], np.cos(3 * 10000 ** (-2 / 7)))
    x = np.array([[1.0, 2.0, 6.0]])
    np.testing.assert_allclose(ref.layer_norm(x, 2.0, 0.5), 2 * (x - 3) / np.sqrt(14 / 3 + 0.5))
    np.testing.assert_allclose(ref.rms_norm(x, 2.0, 0.5), 2 * x / np.sqrt(41 / 3 + 0.5))


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (1, 3, 2), (2, 4, 3), (3, 4, 2)])
def test_run_order(loop):
    cfg = vm.mixed(loop=loop)
    want = ref.run_order(cfg)
    assert vogizen.parse(cfg).run_order() == want
    if loop:
        assert len(want) == 4 + (loop[1] - loop[0]) * (loop[2] - 1)
        assert sum(first for _, first in want) == loop[2]


@pytest.mark.parametrize("name", sorted(vm.MODELS))
def test_shapes_match_the_models(name):
    cfg = vm.MODELS[name]
    assert {n: a.shape for n, a in vm.weights(cfg).items()} == vogizen.shapes(cfg)


def test_config_refusals():
    with pytest.raises(vogizen.ConfigError, match="missing key 'vocab'"):
        vogizen.parse({k: v for k, v in vm.mixed().items() if k != "vocab"})
    bad = json.loads(json.dumps(vm.mixed()))
    bad["layers"][0]["type"] = "mamba"
    with pytest.raises(vogizen.ConfigError, match="unknown mixer type 'mamba'"):
        vogizen.parse(bad)
    bad = json.loads(json.dumps(vm.mixed()))
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(vogizen.ConfigError, match="unknown feed-forward kind"):
        vogizen.parse(bad)
    with pytest.raises(vogizen.ConfigError, match="loop over layers 3..9"):
        vogizen.parse(vm.mixed(loop=(3, 9, 2)))
    cfg = vm.mixed()
    w = vm.weights(cfg)
    del w["l1.mix.uk"]
    with pytest.raises(vogizen.ConfigError, match="missing tensor 'l1.mix.uk'"):
        vogizen.check_tensors(cfg, w)
    w = vm.weights(cfg)
    w["l0.mix.A_log"] = w["l0.mix.A_log"][:-1]
    with pytest.raises(vogizen.ConfigError, match="l0.mix.A_log"):
        vogizen.check_tensors(cfg, w)


def test_safetensors_round_trip_and_refusals(tmp_path):
    import torch
    cfg = vm.MODELS["side"]
    w = vm.weights(cfg, 5)
    vm.write_model(tmp_path, cfg, w)
    got = safetensors.load(tmp_path / "model.safetensors")
    assert set(got) == set(w)
    for n, a in w.items():
        assert got[n].dtype == torch.bfloat16
        np.testing.assert_array_equal(got[n].float().numpy(), a)
    data = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "short").write_bytes(data[:-2])
    with pytest.raises(safetensors.SafetensorsError, match="has bytes"):
        safetensors.load(tmp_path / "short")
    (tmp_path / "none").write_bytes(b"\xff" * 16)
    with pytest.raises(safetensors.SafetensorsError, match="header of"):
        safetensors.load(tmp_path / "none")


def test_unknown_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(registry.UnknownArchitecture, match="'Nobody' is not served; known: .*Vogizen"):
        registry.load_decoder(None, tmp_path)


def test_the_oracle_sees_the_faults_the_device_tests_look_for():
    """A window one token off, a state dropped between passes, a missing readout of the current
    token: each moves the restatement's logits by far more than the device tests allow."""
    cfg = vm.mixed()
    w = vm.weights(cfg)
    toks = vm.prompt(cfg, 40)
    base = ref.forward(cfg, w, toks)
    for change in (lambda c: c["layers"][1]["mixer"]["mask"].update(size=10),
                   lambda c: c["layers"][1]["mixer"]["mask"].update(size=8),
                   lambda c: c["loop"].update(times=1),
                   lambda c: c["embedding"].update(scale=2.9)):
        other = json.loads(json.dumps(cfg))
        change(other)
        moved = ref.forward(other, w, toks)[-1] - base[-1]
        assert np.sqrt((moved ** 2).mean()) > 0.02 * base[-1].std()
