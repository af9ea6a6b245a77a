"""Plain restatement of the Vogizen decoder (loop of latent-attention and gated-delta-rule
layers): one function per mechanism, written from its equation, whole sequences at a time, no
cache, no chunks.  Test infrastructure: it shares no code with the product path.

``cfg`` is the parsed config.json, ``weights`` a dict of arrays by tensor name; everything is
computed in ``ft`` (float64 unless a test says otherwise).
"""

from __future__ import annotations

import numpy as np


_operand = None   # rounding of the linears' inputs while ``rounded_operands`` is in force


class rounded_operands:
    """with rounded_operands(fn): every linear reads fn(its input), the rest stays exact - what a
    16-bit matrix product does at the least, hence a measure of a model's sensitivity to it."""

    def __init__(self, fn):
        self.fn = fn

    def __enter__(self):
        global _operand
        _operand = self.fn

    def __exit__(self, *exc):
        global _operand
        _operand = None


def linear(h, w):
    return (h if _operand is None else _operand(h).astype(h.dtype)) @ w.T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, eps):
    centred = x - x.mean(axis=-1, keepdims=True)
    return centred / np.sqrt((centred ** 2).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * w


def sinusoid(positions, width, ft=np.float64):
    """[T, width]: sine in the even entries, cosine in the odd ones."""
    entry = np.arange(width)
    angle = np.asarray(positions, ft)[:, None] * (ft(10000.0) ** (-(2.0 * (entry // 2)) / width)).astype(ft)
    return np.where(entry % 2 == 0, np.sin(angle), np.cos(angle))


def embed(table, tokens, scale, ft=np.float64):
    x = table[np.asarray(tokens)].astype(ft) * ft(scale)
    return x + sinusoid(np.arange(len(tokens)), table.shape[1], ft)


def causal_conv(x, taps):
    """x [T, channels], taps [channels, n]; the last column multiplies the current token."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1]), x.dtype), x])
    return sum(padded[j:j + len(x)] * taps[:, j] for j in range(n))


def latent_attention(h, m, w, eps, return_weights=False):
    """Windowed latent attention without positions; ``w`` holds the mixer's tensors."""
    T, H, dim, vdim = len(h), m["heads"], m["dim"], m["vdim"]
    q = linear(rms_norm(linear(h, w["dq"]), w["dq.norm"], eps), w["uq"]).reshape(T, H, dim)
    c = rms_norm(linear(h, w["dkv"]), w["dkv.norm"], eps)
    k = linear(c, w["uk"]).reshape(T, H, dim)
    v = linear(c, w["uv"]).reshape(T, H, vdim)
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = (back >= 0) & (back < m["mask"]["size"])
    out = np.zeros((T, H, vdim), h.dtype)
    probs = []
    for a in range(H):
        s = np.where(seen, (q[:, a] @ k[:, a].T) * m["scale"], -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        p /= p.sum(axis=1, keepdims=True)
        probs.append(p)
        out[:, a] = p @ v[:, a]
    y = linear(out.reshape(T, H * vdim), w["o"])
    return (y, np.stack(probs)) if return_weights else y


def delta_rule(q, k, v, beta, decay, state=None):
    """One head: q, k [T, dim], v [T, vdim], beta, decay [T]; returns (outputs, final state)."""
    S = np.zeros((q.shape[1], v.shape[1]), q.dtype) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(len(q)):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def delta_mixer(h, m, w, eps):
    T, H, KV, dim, vdim = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name, heads, size):
        return silu(causal_conv(linear(h, w[name]), w[name + ".conv"])).reshape(T, heads, size)

    def unit(x):
        return x / np.sqrt((x ** 2).sum(axis=-1, keepdims=True) + 1e-6)

    q = unit(branch("q", KV, dim)) * dim ** -0.5
    k = unit(branch("k", KV, dim))
    v = branch("v", H, vdim)
    beta = sigmoid(linear(h, w["b"]))
    decay = np.exp(-np.exp(w["A_log"]) * softplus(linear(h, w["a"]) + w["dt_bias"]))
    gate = silu(linear(h, w["g"])).reshape(T, H, vdim)
    out = np.zeros((T, H, vdim), h.dtype)
    for a in range(H):
        src = a // (H // KV)
        out[:, a], _ = delta_rule(q[:, src], k[:, src], v[:, a], beta[:, a], decay[:, a])
    y = rms_norm(out, w["norm"], eps) * gate
    return linear(y.reshape(T, H * vdim), w["o"])


def relu_mlp(h, w):
    return linear(np.maximum(linear(h, w["gate"]), 0.0) * linear(h, w["up"]), w["down"])


def token_side(x, rows, w, eps):
    """``rows`` [T, dim]: this layer's part of the tokens' side embedding."""
    y = linear(gelu_tanh(linear(x, w["gate"])) * rows, w["proj"])
    return x + rms_norm(y, w["norm"], eps)


MIXERS = {"latent_attention": latent_attention, "delta": delta_mixer}


def run_order(cfg):
    """[(layer, first of a pass?)] in the order in which the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    body = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return ([(i, False) for i in range(loop["start"])] + body * loop["times"]
            + [(i, False) for i in range(loop["stop"], n)])


def forward(cfg, weights, tokens, ft=np.float64, per_layer=None):
    """Logits [T, vocab] of a whole sequence; ``per_layer``: a list that receives the residual
    stream after every layer run."""
    W = {n: (a.astype(ft) if a.dtype.kind == "f" else a) for n, a in weights.items()}
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]

    def part(prefix):
        return {n[len(prefix):]: a for n, a in W.items() if n.startswith(prefix)}

    x = x0 = embed(W["embed"], tokens, cfg["embedding"]["scale"], ft)
    for i, starts_pass in run_order(cfg):
        layer = cfg["layers"][i]
        w = part(f"l{i}.")
        if starts_pass:
            x = linear(np.concatenate([x, x0], axis=1), W["loop.in"])
        mixed = MIXERS[layer["type"]](layer_norm(x, w["norm1"], eps), layer["mixer"], part(f"l{i}.mix."), eps)
        x = x + mixed * w["ls1"]
        if layer["mlp"] is not None:
            x = x + relu_mlp(layer_norm(x, w["norm2"], eps), part(f"l{i}.mlp.")) * w["ls2"]
        if cfg.get("token_side"):
            dim = cfg["token_side"]["dim"]
            x = token_side(x, W["side.embed"][tokens, i * dim:(i + 1) * dim], part(f"l{i}.side."), eps)
        if per_layer is not None:
            per_layer.append(x)
    return linear(layer_norm(x, W["final.norm"], eps), W["embed"])
