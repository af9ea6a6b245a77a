"""Plain restatement of the Virudra decoder (grouped attention with a learned distance bias, dense
and token-table mixture feed-forwards, norms around every sublayer): one function per mechanism,
written from its equation, whole sequences at a time, no cache, no chunks.  Test infrastructure:
it shares no code with the product path.

``cfg`` is the parsed config.json, ``weights`` a dict of arrays by tensor name; everything is
computed in ``ft`` (float64 unless a test says otherwise).
"""

from __future__ import annotations

import math

import numpy as np

_operand = None   # rounding of the linears' inputs while ``rounded_operands`` is in force


class rounded_operands:
    """with rounded_operands(fn): every linear reads fn(its input), and attention reads fn of its
    queries, keys and values, the rest stays exact - what 16-bit matrix products do at the least,
    hence a measure of a model's sensitivity to them."""

    def __init__(self, fn):
        self.fn = fn

    def __enter__(self):
        global _operand
        _operand = self.fn

    def __exit__(self, *exc):
        global _operand
        _operand = None


def operand(h):
    return h if _operand is None else _operand(h).astype(h.dtype)


def linear(h, w):
    return operand(h) @ w.T


def rms_norm(x, w, eps):
    """``w`` is an offset from one."""
    return x / np.sqrt((x ** 2).mean(axis=-1, keepdims=True) + eps) * (1.0 + w)


def silu(z):
    return z / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def query_temperature(position, coef, every):
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1)


def bucket(distance, rows, bias_max):
    """Which row of a table of ``rows`` a distance reads: the near half one by one, the rest in
    logarithmic steps up to ``bias_max``, the last row for everything beyond."""
    half = rows // 2
    if distance < half:
        return distance
    step = math.floor(math.log(distance / half) / math.log(bias_max / half) * (rows - half))
    return min(rows - 1, half + step)


def attention(h, m, w, return_weights=False):
    """Causal grouped attention with a query temperature and a distance bias; ``w`` holds the
    mixer's tensors."""
    T, H, G, dim, vdim = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w["q"]).reshape(T, H, dim)
    k = operand(linear(h, w["k"])).reshape(T, G, dim)
    v = operand(linear(h, w["v"])).reshape(T, G, vdim)
    temperature = np.array([query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(T)])
    q = operand(q * temperature[:, None, None].astype(q.dtype))
    rows = np.array([bucket(n, len(w["rel"]), m["bias_max"]) for n in range(T)])
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, vdim), h.dtype)
    probs = []
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"] + w["rel"][rows[np.maximum(back, 0)], a]
        s = np.where(back >= 0, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        p /= p.sum(axis=1, keepdims=True)
        probs.append(p)
        out[:, a] = p @ v[:, g]
    y = linear(out.reshape(T, H * vdim), w["o"])
    return (y, np.stack(probs)) if return_weights else y


def gated(h, w, act):
    return linear(act(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def table_mixture(h, tokens, router, w):
    """Every token's experts are a row of ``table``; they weigh the same."""
    out = np.zeros_like(h)
    for t, token in enumerate(tokens):
        for e in w["table"][token]:
            part = {n: w[f"e{int(e)}.{n}"] for n in ("gate", "up", "down")}
            out[t] += gated(h[t:t + 1], part, silu)[0] / router["top"]
    return out


def softcap(logits, cap):
    return cap * np.tanh(logits / cap)


def run_order(cfg):
    """The layers in the order in which they run."""
    order = list(range(len(cfg["layers"])))
    loop = cfg.get("loop")
    if not loop:
        return order
    a, b = loop["start"], loop["stop"]
    return order[:a] + order[a:b] * loop["times"] + order[b:]


def forward(cfg, weights, tokens, ft=np.float64, per_layer=None):
    """Logits [T, vocab] of a whole sequence; ``per_layer``: a list that receives the residual
    stream after every layer run."""
    W = {n: (a.astype(ft) if a.dtype.kind == "f" else a) for n, a in weights.items()}
    tokens = [int(t) for t in tokens]
    eps = cfg["norm"]["eps"]

    def part(prefix):
        return {n[len(prefix):]: a for n, a in W.items() if n.startswith(prefix)}

    x = W["embed"][tokens]
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        mixed = attention(rms_norm(x, W[p + "norm1"], eps), layer["mixer"], part(p + "mix."))
        x = x + rms_norm(mixed, W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            h = rms_norm(x, W[p + "norm2"], eps)
            if layer["mlp"]["kind"] == "moe":
                y = table_mixture(h, tokens, layer["mlp"]["router"], part(p + "mlp."))
            else:
                y = gated(h, part(p + "mlp."), gelu_tanh)
            x = x + rms_norm(y, W[p + "norm2b"], eps)
        if per_layer is not None:
            per_layer.append(x)
    return softcap(linear(rms_norm(x, W["final.norm"], eps), W["head"]), cfg["logit_softcap"])
