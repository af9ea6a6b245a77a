"""The Virudra design: config.json and tensors -> ``LayeredConfig``.

A decoder-only model of layers with grouped attention over the whole sequence (no rotation: a query
temperature and a learned distance bias carry the positions), feed-forwards that are dense or a
mixture of experts chosen by a table of token ids, RMS norms before and behind every sublayer whose
weights are offsets from one, optionally a block of layers that runs several times, and a soft cap on
the logits.  Sizes and constants come from config.json; what the design fixes is written here.
"""

from __future__ import annotations

from .layered import LayeredConfig, LayerSpec
from .layers import distance_buckets

NORM_OFFSET = 1.0
DENSE_ACTIVATION = "gelu_tanh"
EXPERT_ACTIVATION = "silu"
DEFAULT_MAX_SEQ = 8192     # positions per slot unless the caller says otherwise: the cache holds them all


class ConfigError(ValueError):
    """A config.json or a set of tensors that does not describe a model of this design."""


def _mixer(kind: str, m: dict) -> dict:
    if kind != "attention":
        raise ConfigError(f"unknown mixer type {kind!r}; known: attention")
    if m["kv_heads"] < 1 or m["heads"] % m["kv_heads"]:
        raise ConfigError(f"attention: {m['heads']} heads over {m['kv_heads']} key/value heads")
    temp = m.get("q_temp")
    if temp is not None and temp["every"] <= 0:
        raise ConfigError(f"attention: a query temperature every {temp['every']} positions")
    return dict(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
                temperature=None if temp is None else (float(temp["coef"]), float(temp["every"])), bias_max=m["bias_max"])


def _feed_forward(mlp: dict | None) -> dict:
    if mlp is None:
        return {}
    if mlp["kind"] == "dense":
        return dict(activation=DENSE_ACTIVATION)
    if mlp["kind"] == "moe":
        router = mlp["router"]
        if not 1 <= router["top"] <= router["experts"]:
            raise ConfigError(f"mixture: {router['top']} of {router['experts']} experts")
        return dict(activation=EXPERT_ACTIVATION, experts=router["experts"])
    raise ConfigError(f"unknown feed-forward kind {mlp['kind']!r}; known: dense, moe")


def parse(config: dict, **settings) -> LayeredConfig:
    """``settings`` are ``LayeredConfig``'s serving settings (serving, max_seq, max_batch, ...)."""
    try:
        layers = [LayerSpec("grouped_attention", _mixer(layer["type"], layer["mixer"]), **_feed_forward(layer.get("mlp")))
                  for layer in config["layers"]]
        loop = config.get("loop")
        if loop is not None:
            loop = (loop["start"], loop["stop"], loop["times"])
            if not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ConfigError(f"loop over layers {loop[0]}..{loop[1]}, {loop[2]} times, of {len(layers)} layers")
        cap = config.get("logit_softcap")
        return LayeredConfig(vocab=config["vocab"], width=config["width"], layers=layers, norm="rms",
                             norm_eps=float(config["norm"]["eps"]), norm_offset=NORM_OFFSET, post_norms=True, loop=loop,
                             logit_softcap=None if cap is None else float(cap),
                             **{"max_seq": DEFAULT_MAX_SEQ, **settings})
    except KeyError as e:
        raise ConfigError(f"config.json: missing key {e.args[0]!r}") from None


def shapes(config: dict) -> dict:
    """{tensor name: shape} that a model of this config must have; None stands for a size that only
    the tensor tells."""
    d, v = config["width"], config["vocab"]
    out = {"embed": (v, d), "final.norm": (d,), "head": (v, d)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        mix, qk, kk, vv = p + "mix.", m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        out.update({p + "norm1": (d,), p + "norm1b": (d,), mix + "q": (qk, d), mix + "k": (kk, d), mix + "v": (vv, d),
                    mix + "rel": (None, m["heads"]), mix + "o": (d, m["heads"] * m["vdim"])})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        out.update({p + "norm2": (d,), p + "norm2b": (d,)})
        parts = [(p + "mlp.", mlp)]
        if mlp["kind"] == "moe":
            parts = [(f"{p}mlp.e{e}.", mlp["expert"]) for e in range(mlp["router"]["experts"])]
            out[p + "mlp.table"] = (v, mlp["router"]["top"])
        for name, sizes in parts:
            out.update({name + "gate": (sizes["ff"], d), name + "up": (sizes["ff"], d), name + "down": (d, sizes["ff"])})
    return out


def check_tensors(config: dict, tensors: dict) -> None:
    """Names, shapes, the range of the expert tables (they index weights) and the distance biases."""
    try:
        wanted = shapes(config)
    except KeyError as e:
        raise ConfigError(f"config.json: missing key {e.args[0]!r}") from None
    for name, shape in wanted.items():
        if name not in tensors:
            raise ConfigError(f"missing tensor {name!r}")
        have = tuple(tensors[name].shape)
        if len(have) != len(shape) or any(w not in (None, h) for h, w in zip(have, shape)):
            raise ConfigError(f"tensor {name!r} has shape {list(have)}; the config wants {list(shape)}")
    for i, layer in enumerate(config["layers"]):
        rel = tensors[f"l{i}.mix.rel"]
        try:
            distance_buckets(rel.shape[0], layer["mixer"]["bias_max"])
        except ValueError as e:
            raise ConfigError(f"layer {i}: {e}") from None
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] == "moe":
            table = tensors[f"l{i}.mlp.table"]
            if table.is_floating_point():
                raise ConfigError(f"tensor 'l{i}.mlp.table' must hold integers")
            if int(table.min()) < 0 or int(table.max()) >= mlp["router"]["experts"]:
                raise ConfigError(f"tensor 'l{i}.mlp.table' names experts outside 0..{mlp['router']['experts'] - 1}")
            rows = table.sort(dim=1).values
            if bool((rows[:, 1:] == rows[:, :-1]).any()):
                raise ConfigError(f"tensor 'l{i}.mlp.table' names an expert twice in a row")
