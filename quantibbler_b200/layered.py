"""Decoder of layered designs: a list of layers, each a mixer (``layers.py``) with an optional
feed-forward (gated, or a mixture of experts), optionally with a block of layers that runs several
times, layer scales or norms behind the sublayers, and a per-layer token input.

Slots, prompts in portions, greedy steps, graph capture and generation are ``SlotDecoder``'s; this
class adds the trunk.  Every pass of a looped layer has its own cache or state; what a sequence
leaves behind in a slot is never read by the next one (positions decide what is valid).
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import numpy as np

from . import _lib
from ._lib import QK_F32, check
from .decoder import SlotDecoder, check_cache_capacity
from .gpu import GpuContext
from .layers import (IN_CONCAT, IN_NORM, NORM_LAYER, NORM_NONE, NORM_RMS, GatedDelta, GatedMlp, GroupedAttention, Join,
                     LatentAttention, Linear, Rows, TableExperts, TokenSide, Weights, padded)

NORMS = {"layer": NORM_LAYER, "rms": NORM_RMS}
IDLE = -(1 << 30)   # position of a row without a sequence: far enough below zero to stay negative


@dataclass
class LayerSpec:
    mixer: str                      # a key of MIXERS
    sizes: dict                     # the mixer's keyword arguments
    activation: str | None = None   # feed-forward activation; None: no feed-forward
    experts: int | None = None      # a mixture of this many, chosen by a table of token ids; None: one


@dataclass
class LayeredConfig:
    vocab: int
    width: int
    layers: list
    norm: str = "layer"
    norm_eps: float = 1e-5
    norm_offset: float = 0.0                # added to the norms' weights
    post_norms: bool = False                # results join the stream through norms (norm1b, norm2b)
    logit_softcap: float | None = None      # logits <- cap tanh(logits / cap)
    embedding_scale: float = 1.0
    sinusoid_base: float | None = None      # None: no position vector
    loop: tuple | None = None               # (start, stop, times)
    side_dim: int | None = None             # per-layer token input
    serving: str = "bfloat16"
    max_seq: int = 1 << 20                  # positions; windowed layers keep only their window
    max_batch: int = 1
    prefill_min_tokens: int = 2
    prefill_chunk: int = 2048
    vector_rows: int = 4                    # portions this short keep float32 activations

    def run_order(self) -> list:
        """[(layer, starts a pass)] in running order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        body = [(i, i == start) for i in range(start, stop)]
        return [(i, False) for i in range(start)] + body * times + [(i, False) for i in range(stop, n)]


MIXERS = {"latent_attention": LatentAttention, "delta": GatedDelta, "grouped_attention": GroupedAttention}


class _Layer:
    def __init__(self, w: Weights, cfg: LayeredConfig, spec: LayerSpec, t: dict, index: int, side_table):
        def part(prefix):
            return {n[len(prefix):]: a for n, a in t.items() if n.startswith(prefix)}

        def join(which):
            if cfg.post_norms:
                return Join(norm=w.vector(t[f"norm{which}b"], cfg.norm_offset), eps=cfg.norm_eps)
            return Join(scale=w.vector(t[f"ls{which}"]) if f"ls{which}" in t else None)

        self.mixer = MIXERS[spec.mixer](w, part("mix."), eps=cfg.norm_eps, **spec.sizes)
        self.norm1, self.norm2, self.mlp, self.side = w.vector(t["norm1"], cfg.norm_offset), None, None, None
        self.join1, self.join2 = join(1), None
        if spec.activation is not None:
            self.norm2, self.join2 = w.vector(t["norm2"], cfg.norm_offset), join(2)
            if spec.experts is None:
                self.mlp = GatedMlp(w, part("mlp."), activation=spec.activation)
            else:
                self.mlp = TableExperts(w, part("mlp."), experts=spec.experts, activation=spec.activation)
        if cfg.side_dim is not None:
            self.side = TokenSide(w, part("side."), side_table, dim=cfg.side_dim, offset=index * cfg.side_dim,
                                  eps=cfg.norm_eps)


class LayeredDecoder(SlotDecoder):
    """Batched greedy decoding of a ``LayeredConfig`` model on one GPU; ``tensors`` maps tensor
    names (``embed``, ``l<i>.*``, ``loop.in``, ``side.embed``, ``final.norm``, ``head``) to torch
    tensors; without ``head`` the embedding table serves as the head, without ``loop.in`` nothing
    happens between the passes of a loop."""

    keeps_state = True

    def __init__(self, ctx: GpuContext, cfg: LayeredConfig, tensors: dict):
        import torch
        self.torch, self.ctx, self.cfg = torch, ctx, cfg
        if cfg.serving not in ("float32", "bfloat16"):
            raise ValueError(f"serving dtype must be float32 or bfloat16, got {cfg.serving!r}")
        dev = self.device = torch.device("cuda", torch.cuda.current_device())
        ctx.set_stream(torch.cuda.current_stream().cuda_stream)  # order with torch's own work
        w = self.weights = Weights(torch, dev, cfg.serving)
        self.width, self.stride = cfg.width, padded(cfg.width)
        self.norm_kind = NORMS[cfg.norm]
        if cfg.post_norms and cfg.side_dim is not None:
            raise ValueError("a token input reads the settled stream: not beside norms behind the sublayers")
        # (columns padded)
        self.embedding = w.matrix(tensors["embed"]).w
        self.lm_head = w.matrix(tensors["head"]).w if "head" in tensors else self.embedding
        self.logit_softcap = cfg.logit_softcap
        self.head_width, self.v_loc, self.vocab_offset = self.stride, cfg.vocab, 0
        self.final_norm = w.vector(tensors["final.norm"], cfg.norm_offset)
        self.inv_freq = None
        if cfg.sinusoid_base is not None:
            i = np.arange((cfg.width + 1) // 2, dtype=np.float64)
            self.inv_freq = torch.from_numpy(float(cfg.sinusoid_base) ** (-2.0 * i / cfg.width)).to(dev)
        side = w.to(tensors["side.embed"]) if cfg.side_dim is not None else None
        self.loop_in = w.halves(tensors["loop.in"], cfg.width) if "loop.in" in tensors else None
        self.layers = [
            _Layer(w, cfg, spec, {n[len(f"l{i}."):]: t for n, t in tensors.items() if n.startswith(f"l{i}.")}, i, side)
            for i, spec in enumerate(cfg.layers)]
        self.tables = [layer.mlp.table for layer in self.layers if isinstance(layer.mlp, TableExperts)]
        B = cfg.max_batch
        self.portion_rows = min(cfg.prefill_chunk, cfg.max_seq)
        self.runs = [(self.layers[i], starts,
                      self.layers[i].mixer.make_state(torch, dev, B, cfg.max_seq, max(self.portion_rows, 1)))
                     for i, starts in cfg.run_order()]
        self.rows = Rows(torch, dev, B, self.stride, w, vector=B <= cfg.vector_rows)
        self._portions = {}
        self.token_ids, self.positions = self.rows.ids, self.rows.positions
        self.positions.fill_(IDLE)
        f32 = dict(dtype=torch.float32, device=dev)
        self.h = torch.zeros(B, self.stride, **f32)
        self.logits = torch.zeros(B, cfg.vocab, **f32)
        self.best_val = torch.zeros(B, **f32)
        self.best_idx = torch.zeros(B, dtype=torch.int32, device=dev)
        self._setup_driver()
        self._host_positions = [None] * B

    # ------------------------------------------------------------------ trunk
    def _trunk(self, rows: Rows, after_layer=None) -> None:
        cfg, ctx = self.cfg, self.ctx
        rows.pending = None
        rows.route(ctx, self.tables, self.width, cfg.vocab)
        first = rows.f32("embedding", self.stride) if self.loop_in is not None else None
        check(_lib.lib().qk_embed_scaled(
            ctx.handle, self.embedding.data_ptr(), self.weights.tag, self.stride, rows.ids.data_ptr(),
            rows.positions.data_ptr(), rows.n, self.width, cfg.vocab, float(cfg.embedding_scale),
            None if self.inv_freq is None else self.inv_freq.data_ptr(), rows.x.data_ptr(),
            None if first is None else first.data_ptr(), self.stride))
        for layer, starts_pass, state in self.runs:
            if starts_pass and self.loop_in is not None:
                f = dict(rows.stream_fields(NORM_NONE, None, 0.0), input=IN_CONCAT, second=first, x_out=None)
                rows.dense(ctx, self.loop_in, **f, out=rows.x2, out_stride=self.stride)
                rows.x, rows.x2, rows.pending = rows.x2, rows.x, None
            layer.mixer.forward(ctx, rows, self.norm_kind, layer.norm1, cfg.norm_eps, layer.join1, state, cfg.max_seq)
            if layer.mlp is not None:
                layer.mlp.forward(ctx, rows, self.norm_kind, layer.norm2, cfg.norm_eps, layer.join2)
            if layer.side is not None:
                layer.side.forward(ctx, rows)
            if after_layer is not None:
                after_layer(self.stream(rows))

    def _final(self, rows: Rows, places, out) -> None:
        """Final-normed rows: all of them (``places`` None) or the given ones."""
        x, pending, n = rows.x, rows.pending, rows.n
        if places is not None:
            n = len(places)
            if n == 1 and pending is None:
                x = x[places[0]:]
            else:
                idx = self.torch.as_tensor(places, device=self.device)
                x, pending = x.index_select(0, idx), None if pending is None else pending.at(self.torch, idx)
        fields = dict(tokens=n, input=IN_NORM, x=x, x_stride=self.stride, norm=self.norm_kind,
                      norm_weight=self.final_norm, norm_eps=self.cfg.norm_eps, out=out, out_dtype=QK_F32)
        if pending is not None:
            fields.update(pending.fields())
        d = rows.call(Linear(self.lm_head, 0, self.width, self.stride), **fields)
        check(_lib.lib().qk_dense_input(self.ctx.handle, ctypes.byref(d)))

    def stream(self, rows: Rows):
        """A copy of the residual stream with what is pending added (for inspection)."""
        out = self.torch.zeros(rows.n, self.stride, dtype=self.torch.float32, device=self.device)
        f = dict(rows.stream_fields(NORM_NONE, None, 0.0), x_out=None)
        d = rows.call(Linear(self.lm_head, 0, self.width, self.stride), **f, out=out)
        check(_lib.lib().qk_dense_input(self.ctx.handle, ctypes.byref(d)))
        return out[:, :self.width]

    # ------------------------------------------------------------------ steps
    def step(self) -> None:
        """One decode step for the whole batch (idle slots change nothing); leaves the logits in
        ``logits`` and the greedy tokens in ``best_idx``."""
        rows = self.rows
        x, x2 = rows.x, rows.x2
        self._trunk(rows)
        self._final(rows, None, self.h)
        rows.x, rows.x2 = x, x2      # (every step starts in the same buffer, as its graph replays it)
        self._head(self.h, rows.n, self.logits)
        self._greedy(self.logits, rows.n, self.best_val, self.best_idx)

    def start(self, token_ids, positions) -> None:
        """Next token and position per slot; position None: the slot sits this step out."""
        live = [p for p in positions if p is not None]
        check_cache_capacity(live, 1, self.cfg.max_seq)
        torch = self.torch
        self._host_positions = [None if p is None else int(p) for p in positions]
        self.token_ids.copy_(torch.as_tensor(token_ids, dtype=torch.int32))
        self.positions.copy_(torch.as_tensor([IDLE if p is None else int(p) for p in positions], dtype=torch.int32))

    def _make_idle(self) -> None:
        self.positions.fill_(IDLE)

    def _portion_buffers(self, n: int, reserve: int) -> Rows:
        """The workspace for a portion of ``n`` rows (kept and reused)."""
        short = n <= self.cfg.vector_rows
        cap = self.cfg.vector_rows if short else max(n, reserve)
        have = self._portions.get(short)
        if have is None or have.cap < cap:
            have = Rows(self.torch, self.device, cap, self.stride, self.weights, vector=short)
            self._portions[short] = have
        return have

    def _prefill_portion(self, part, seq: int, p0: int, reserve: int) -> None:
        torch, n = self.torch, len(part)
        rows = self._portion = self._portion_buffers(n, reserve)
        rows.n, rows.segments, rows.portion = n, 1, (seq, p0)
        at = torch.arange(n, dtype=torch.int32)
        rows.ids[:n].copy_(torch.tensor(part, dtype=torch.int32))
        rows.seg_row[:n].copy_(at)
        rows.positions[:n].copy_(at + p0)
        rows.slots[:n].fill_(seq)
        rows.seg_first[:1].fill_(0)
        rows.seg_len[:1].fill_(n)
        self._trunk(rows, getattr(self, "after_layer", None))

    def _portion_hidden(self, places, out) -> None:
        self._final(self._portion, places, out)
