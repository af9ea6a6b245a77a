"""The Vogizen design: config.json and tensors -> ``LayeredConfig``.

A decoder-only model of layers with windowed latent attention (no positions inside) or a gated
delta rule, relu-gated feed-forwards on some layers, layer scales, a per-layer token input, a
sinusoidal position vector on the embedding, and a block of layers that runs several times, each
pass opening with a linear over the stream and the embedding output.  Sizes and constants come
from config.json; what the design fixes is written here.
"""

from __future__ import annotations

from .layered import LayeredConfig, LayerSpec

SINUSOID_BASE = 10000.0
UNIT_EPS = 1e-6            # under the root of the delta rule's unit vectors
MLP_ACTIVATION = "relu"


class ConfigError(ValueError):
    """A config.json or a set of tensors that does not describe a model of this design."""


def _mixer(kind: str, m: dict) -> dict:
    if kind == "latent_attention":
        mask = m.get("mask") or {}
        return dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"],
                    scale=m["scale"], window=mask.get("size"))
    if kind == "delta":
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"delta mixer: {m['heads']} heads over {m['kv_heads']} key heads")
        return dict(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], taps=m["conv"],
                    unit_eps=UNIT_EPS)
    raise ConfigError(f"unknown mixer type {kind!r}; known: latent_attention, delta")


def parse(config: dict, **settings) -> LayeredConfig:
    """``settings`` are ``LayeredConfig``'s serving settings (serving, max_seq, max_batch, ...)."""
    try:
        layers = []
        for layer in config["layers"]:
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ConfigError(f"unknown feed-forward kind {mlp['kind']!r}; known: dense")
            layers.append(LayerSpec(layer["type"], _mixer(layer["type"], layer["mixer"]),
                                    None if mlp is None else MLP_ACTIVATION))
        loop = config.get("loop")
        if loop is not None:
            loop = (loop["start"], loop["stop"], loop["times"])
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"loop over layers {loop[0]}..{loop[1]}, {loop[2]} times, of {len(layers)} layers")
        side = config.get("token_side")
        return LayeredConfig(vocab=config["vocab"], width=config["width"], layers=layers, norm="layer",
                             norm_eps=float(config["norm"]["eps"]),
                             embedding_scale=float(config["embedding"]["scale"]), sinusoid_base=SINUSOID_BASE,
                             loop=loop, side_dim=None if side is None else side["dim"], **settings)
    except KeyError as e:
        raise ConfigError(f"config.json: missing key {e.args[0]!r}") from None


def shapes(config: dict) -> dict:
    """{tensor name: shape} that a model of this config must have."""
    d, v = config["width"], config["vocab"]
    out = {"embed": (v, d), "final.norm": (d,)}
    if config.get("loop") is not None:
        out["loop.in"] = (d, 2 * d)
    side = config.get("token_side")
    if side is not None:
        out["side.embed"] = (v, len(config["layers"]) * side["dim"])
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        mix = p + "mix."
        out[p + "norm1"] = out[p + "ls1"] = (d,)
        if layer["type"] == "latent_attention":
            qk, vv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({mix + "dq": (m["q_rank"], d), mix + "dq.norm": (m["q_rank"],), mix + "uq": (qk, m["q_rank"]),
                        mix + "dkv": (m["kv_rank"], d), mix + "dkv.norm": (m["kv_rank"],),
                        mix + "uk": (qk, m["kv_rank"]), mix + "uv": (vv, m["kv_rank"]), mix + "o": (d, vv)})
        else:
            qk, vv, taps = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["conv"]
            out.update({mix + "q": (qk, d), mix + "k": (qk, d), mix + "v": (vv, d), mix + "q.conv": (qk, taps),
                        mix + "k.conv": (qk, taps), mix + "v.conv": (vv, taps), mix + "b": (m["heads"], d),
                        mix + "a": (m["heads"], d), mix + "A_log": (m["heads"],), mix + "dt_bias": (m["heads"],),
                        mix + "norm": (m["vdim"],), mix + "g": (vv, d), mix + "o": (d, vv)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (d,), p + "ls2": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d),
                        p + "mlp.down": (d, ff)})
        if side is not None:
            out.update({p + "side.gate": (side["dim"], d), p + "side.proj": (d, side["dim"]), p + "side.norm": (d,)})
    return out


def check_tensors(config: dict, tensors: dict) -> None:
    for name, shape in shapes(config).items():
        if name not in tensors:
            raise ConfigError(f"missing tensor {name!r}")
        if tuple(tensors[name].shape) != shape:
            raise ConfigError(f"tensor {name!r} has shape {list(tensors[name].shape)}; the config wants {list(shape)}")
