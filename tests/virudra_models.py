"""Small Virudra models for the tests: configurations and random weights (bfloat16-valued, so that
both serving dtypes hold exactly the oracle's numbers)."""

import numpy as np

from vogizen_models import bf16, prompt, tensors, write_model  # noqa: F401


def attention(heads=6, kv_heads=2, dim=20, vdim=28, bias_max=40, coef=0.4, every=5, scale=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max,
                      "q_temp": {"coef": coef, "every": every}, "scale": dim ** -0.5 if scale is None else scale}}


def dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def moe(layer, ff, experts, top):
    return dict(layer, mlp={"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}})


def bare(layer):
    return dict(layer, mlp=None)


def config(layers, width=72, vocab=97, loop=None, cap=9.0, eps=1e-5):
    return {"architecture": "Virudra", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "logit_softcap": cap}


def weights(cfg, seed=0, bias_rows=13):
    """``bias_rows``: of every layer's distance bias, or a list with one entry per layer."""
    rng = np.random.default_rng(seed)
    d, v, out = cfg["width"], cfg["vocab"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=0.0, spread=0.3):
        out[name] = bf16(mean + spread * rng.standard_normal(n))

    out["embed"] = bf16(rng.standard_normal((v, d)))
    vec("final.norm", d)
    mat("head", v, d, 4.0)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        vec(p + "norm1", d)
        vec(p + "norm1b", d, -0.5)
        mat(p + "mix.q", H * dim, d, 1.2)
        mat(p + "mix.k", G * dim, d, 1.2)
        mat(p + "mix.v", G * vdim, d)
        rows = bias_rows[i] if isinstance(bias_rows, (list, tuple)) else bias_rows
        out[p + "mix.rel"] = bf16(rng.standard_normal((rows, H)) * 1.2)
        mat(p + "mix.o", d, H * vdim)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        vec(p + "norm2", d)
        vec(p + "norm2b", d, -0.5)
        parts = [(p + "mlp.", mlp)]
        if mlp["kind"] == "moe":
            experts, top = mlp["router"]["experts"], mlp["router"]["top"]
            parts = [(f"{p}mlp.e{e}.", mlp["expert"]) for e in range(experts)]
            out[p + "mlp.table"] = np.stack([rng.permutation(experts)[:top] for _ in range(v)]).astype(np.int32)
        for name, sizes in parts:
            mat(name + "gate", sizes["ff"], d)
            mat(name + "up", sizes["ff"], d)
            mat(name + "down", d, sizes["ff"])
    return out


def mixed(loop=(1, 3, 2), **kw):
    """The mechanisms together, in sizes that share no factor: dense, mixture and no feed-forward,
    layers that differ in heads, sizes, bias and temperature, a looped block in the middle."""
    return config([dense(attention(), 56), moe(attention(heads=4, kv_heads=4, dim=33, vdim=18, bias_max=30, every=3), 40, 5, 2),
                   bare(attention(heads=9, kv_heads=1, dim=16, vdim=40, bias_max=100, coef=0.9, every=17)),
                   moe(attention(heads=2, kv_heads=1, dim=24, vdim=24, bias_max=25, coef=-0.2, every=1), 24, 7, 3)],
                  loop=loop, **kw)


MIXED_ROWS = [13, 8, 32, 5]

# name: (configuration, rows of the distance biases)
MODELS = {
    "attention": (config([bare(attention())]), 13),
    "attention-one-head": (config([bare(attention(heads=1, kv_heads=1, dim=16, vdim=16))], width=50), 6),
    "attention-no-groups": (config([bare(attention(heads=3, kv_heads=3, dim=48, vdim=17))]), 32),
    "attention-large-group": (config([bare(attention(heads=22, kv_heads=2, dim=12, vdim=10))]), 9),
    "attention-wide": (config([bare(attention(heads=4, kv_heads=2, dim=144, vdim=200))], width=130), 13),
    "attention-wide-keys": (config([bare(attention(heads=2, kv_heads=1, dim=128, vdim=40))]), 13),
    "attention-tensor-memory": (config([bare(attention(heads=6, kv_heads=2, dim=72, vdim=100))]), 13),
    "attention-tensor-memory-odd-group": (config([dense(attention(heads=3, kv_heads=1, dim=64, vdim=64), 40)], loop=(0, 1, 2)), 13),
    "attention-too-wide-for-tiles": (config([bare(attention(heads=2, kv_heads=1, dim=264, vdim=300))]), 7),
    "two-buckets": (config([bare(attention(bias_max=2))]), 2),
    "bias-to-the-end": (config([bare(attention(bias_max=44))]), 80),
    "odd-buckets": (config([bare(attention(bias_max=9))]), 7),
    "no-temperature": (config([bare(attention(coef=0.0))]), 13),
    "dense": (config([dense(attention(), 100)], width=65), 13),
    "moe": (config([moe(attention(), 40, 6, 2)]), 13),
    "moe-one": (config([moe(attention(), 33, 4, 1)], width=65), 13),
    "moe-single-expert": (config([moe(attention(), 64, 1, 1)]), 13),
    "moe-all": (config([moe(attention(), 20, 3, 3)]), 13),
    "moe-many": (config([moe(attention(), 16, 70, 5)]), 13),
    "loop-whole": (config([dense(attention(), 40), moe(attention(), 30, 4, 2)], loop=(0, 2, 2)), 13),
    "loop-thrice": (config([moe(attention(heads=2), 30, 4, 2)], loop=(0, 1, 3)), 13),
    "loop-once": (config([dense(attention(), 40), bare(attention())], loop=(1, 2, 1)), 13),
    "low-cap": (config([bare(attention())], cap=1.5), 13),
    "large-eps": (config([moe(attention(), 40, 6, 4)], eps=0.5), 13),
    "mixed": (mixed(), MIXED_ROWS),
}
