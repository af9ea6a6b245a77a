"""Small Vogizen models for the tests: configurations, random weights (bfloat16-valued, so that
both serving dtypes hold exactly the oracle's numbers) and a safetensors writer."""

import json
import os

import numpy as np


def attention(heads=3, dim=20, vdim=28, kv_rank=40, q_rank=24, size=9, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": size}, "scale": dim ** -0.5 if scale is None else scale}}


def delta(heads=6, kv_heads=2, dim=12, vdim=20, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def mlp(layer, ff=None):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def config(layers, width=72, vocab=97, loop=None, side=10, scale=3.0, eps=1e-5):
    return {"architecture": "Vogizen", "width": width, "vocab": vocab, "layers": layers,
            "embedding": {"scale": scale}, "norm": {"eps": eps},
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "token_side": None if side is None else {"dim": side}}


def bf16(a):
    u = np.asarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return ((((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32)).view(np.float32)


def weights(cfg, seed=0):
    rng = np.random.default_rng(seed)
    d, v, out = cfg["width"], cfg["vocab"], {}

    def mat(name, rows, cols, gain=1.0):
        out[name] = bf16(rng.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(name, n, mean=1.0, spread=0.2):
        out[name] = bf16(mean + spread * rng.standard_normal(n))

    out["embed"] = bf16(rng.standard_normal((v, d)) * 0.3)
    vec("final.norm", d)
    if cfg["loop"] is not None:
        mat("loop.in", d, 2 * d, 1.4)
    side = cfg["token_side"]
    if side is not None:
        out["side.embed"] = bf16(rng.standard_normal((v, side["dim"] * len(cfg["layers"]))))
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        vec(p + "norm1", d)
        vec(p + "ls1", d, 0.7)
        if layer["type"] == "latent_attention":
            H, dq = m["heads"], m["dim"]
            mat(p + "mix.dq", m["q_rank"], d)
            vec(p + "mix.dq.norm", m["q_rank"])
            mat(p + "mix.uq", H * dq, m["q_rank"], 2.0)
            mat(p + "mix.dkv", m["kv_rank"], d)
            vec(p + "mix.dkv.norm", m["kv_rank"])
            mat(p + "mix.uk", H * dq, m["kv_rank"], 2.0)
            mat(p + "mix.uv", H * m["vdim"], m["kv_rank"])
            mat(p + "mix.o", d, H * m["vdim"])
        else:
            H, KV, dim, vd, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", KV * dim), ("k", KV * dim), ("v", H * vd)):
                mat(p + "mix." + n, rows, d, 2.0)
                out[p + f"mix.{n}.conv"] = bf16(rng.standard_normal((rows, taps)) / np.sqrt(taps))
            mat(p + "mix.b", H, d)
            mat(p + "mix.a", H, d)
            out[p + "mix.A_log"] = bf16(np.log(rng.uniform(0.05, 2.0, H)))
            out[p + "mix.dt_bias"] = bf16(rng.uniform(-4.0, 0.5, H))
            vec(p + "mix.norm", vd)
            mat(p + "mix.g", H * vd, d)
            mat(p + "mix.o", d, H * vd)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            vec(p + "norm2", d)
            vec(p + "ls2", d, 0.7)
            mat(p + "mlp.gate", ff, d)
            mat(p + "mlp.up", ff, d)
            mat(p + "mlp.down", d, ff)
        if side is not None:
            mat(p + "side.gate", side["dim"], d)
            mat(p + "side.proj", d, side["dim"])
            vec(p + "side.norm", d, 0.3, 0.1)
    return out


def tensors(w):
    """The weights as the torch tensors a file would hold."""
    import torch
    return {n: torch.from_numpy(np.ascontiguousarray(a)).to(torch.bfloat16 if a.dtype.kind == "f" else torch.int32)
            for n, a in w.items()}


def write_model(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        if a.dtype.kind == "f":
            kind, raw = "BF16", (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        else:
            kind, raw = "I32", np.ascontiguousarray(a).astype("<i4").tobytes()
        header[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(len(head).to_bytes(8, "little") + head + b"".join(blobs))


def prompt(cfg, n, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]


# The mechanisms together, in sizes that share no factor: a looped block in the middle, both
# mixers with and without a feed-forward.
def mixed(size=9, loop=(1, 3, 2), **kw):
    return config([mlp(delta(), 56), mlp(attention(size=size), 88), mlp(delta(heads=4, kv_heads=4, dim=33, vdim=18, conv=5)),
                   mlp(attention(heads=17, dim=16, vdim=8, kv_rank=72, q_rank=96, size=size + 3))], loop=loop, **kw)


MODELS = {
    "delta": config([mlp(delta())], side=None),
    "delta-one-tap": config([mlp(delta(heads=2, kv_heads=1, dim=40, vdim=16, conv=1), 33)], side=None, width=50),
    "delta-wide": config([mlp(delta(heads=2, kv_heads=2, dim=260, vdim=130, conv=2))], side=None, width=96),
    "attention": config([mlp(attention())], side=None),
    "attention-wide": config([mlp(attention(heads=2, dim=144, vdim=200, kv_rank=136, q_rank=40, size=20))], side=None),
    "attention-huge-latent": config([mlp(attention(heads=2, dim=24, vdim=300, kv_rank=520, q_rank=16, size=11))], side=None),
    "attention-one-token": config([mlp(attention(size=1))], side=None),
    "mlp": config([mlp(attention(), 100)], side=None, width=65),
    "side": config([mlp(delta()), mlp(attention(), 40)], side=7),
    "loop-whole": config([mlp(delta()), mlp(attention())], side=None, loop=(0, 2, 3)),
    "loop-once": config([mlp(delta()), mlp(attention(), 30)], loop=(1, 2, 1)),
    "mixed": mixed(),
}
