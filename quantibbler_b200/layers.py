"""Building blocks of layered decoders: dense linears with their fused inputs and outputs, the
mixers (windowed latent attention, grouped attention with a distance bias, gated delta rule), each
with the cache or state it keeps per sequence slot, and the feed-forwards (gated, mixture of experts).

A mixer takes the residual stream of a ``Rows`` workspace and adds its result to it; everything
it does is a C-ABI call that only launches kernels, so a step can be captured in a CUDA graph.
Sizes and constants are parameters: nothing here belongs to one design.
"""

from __future__ import annotations

import ctypes
import functools
import math
from ctypes import c_double, c_float, c_int32, c_size_t, c_uint64, c_void_p
from dataclasses import dataclass

from . import _lib
from ._lib import QK_BF16, QK_F32, check

IN_PLAIN, IN_NORM, IN_CONCAT, IN_GATED = range(4)
NORM_NONE, NORM_LAYER, NORM_RMS = range(3)
ACTIVATIONS = {"relu": 0, "silu": 1, "gelu_tanh": 2}
OUT_STORE, OUT_RESIDUAL, OUT_GLU, OUT_SIDE = range(4)
FORM_VECTOR = 0


def _struct(name, fields):
    return type(name, (ctypes.Structure,), {"_fields_": fields})


_P, _Z, _I, _F = c_void_p, c_size_t, c_int32, c_float
LatentAppend = _struct("LatentAppend", [
    ("src", _P), ("src_stride", _Z), ("width", _Z), ("weight", _P), ("eps", _F), ("cache_dtype", _I),
    ("cache", _P), ("ring", _Z), ("stride", _Z)])
DenseCall = _struct("DenseCall", [
    ("tokens", _Z), ("positions", _P), ("slots", _P), ("ids", _P), ("vocab", _Z),
    ("input", _I), ("x_dtype", _I), ("x", _P), ("x_stride", _Z), ("width", _Z), ("k", _Z),
    ("pending", _P), ("pending_stride", _Z), ("pending_weight", _P), ("pending_eps", _F), ("x_out", _P),
    ("second", _P), ("norm", _I), ("norm_eps", _F), ("norm_weight", _P), ("gate", _P), ("gate_stride", _Z),
    ("group", _Z), ("append", LatentAppend),
    ("w_dtype", _I), ("w", _P), ("rows", _Z), ("w_stride", _Z),
    ("output", _I), ("activation", _I), ("out_dtype", _I), ("out", _P), ("out_stride", _Z),
    ("residual", _P), ("residual_stride", _Z), ("out_scale", _P), ("side", _P), ("side_dtype", _I),
    ("side_stride", _Z), ("side_offset", _Z), ("scratch", _P), ("scratch_bytes", _Z),
    ("pending_rows", _P), ("pending_top", _Z), ("pending_scale", _F),
    ("experts", _Z), ("top", _Z), ("by_choice", _I), ("table", _P), ("places", _P), ("offsets", _P), ("tiles", _P)])
RouteJob = _struct("RouteJob", [("table", _P), ("places", _P), ("offsets", _P), ("tiles", _P), ("top", c_uint64),
                                ("experts", c_uint64)])
GroupedCall = _struct("GroupedCall", [
    ("tokens", _Z), ("positions", _P), ("slots", _P), ("heads", _Z), ("kv_heads", _Z), ("dim_stride", _Z),
    ("vdim_stride", _Z), ("s_max", _Z), ("n_slots", _Z), ("scale", _F), ("temp_coef", _F), ("temp_every", c_double),
    ("bias", _P), ("bias_len", _Z), ("proj", _P), ("proj_dtype", _I), ("proj_stride", _Z), ("cache_dtype", _I),
    ("cache_k", _P), ("cache_v", _P), ("n_splits", _Z), ("scratch", _P), ("out", _P), ("out_dtype", _I),
    ("out_stride", _Z), ("append", _I), ("slot", _Z), ("first_position", _Z)])
DeltaCall = _struct("DeltaCall", [
    ("tokens", _Z), ("segments", _Z), ("positions", _P), ("slots", _P), ("seg_first", _P), ("seg_len", _P),
    ("seg_row", _P), ("heads", _Z), ("kv_heads", _Z), ("dim", _Z), ("vdim", _Z), ("taps", _Z), ("proj", _P),
    ("proj_stride", _Z), ("beta_offset", _Z), ("decay_offset", _Z), ("conv_q", _P), ("conv_k", _P), ("conv_v", _P),
    ("a_log", _P), ("dt_bias", _P), ("unit_eps", _F), ("conv_state", _P), ("state", _P), ("qkv", _P), ("gates", _P),
    ("out", _P), ("out_stride", _Z)])
LatentCall = _struct("LatentCall", [
    ("tokens", _Z), ("positions", _P), ("slots", _P), ("heads", _Z), ("dim", _Z), ("dim_stride", _Z), ("vdim", _Z),
    ("vdim_stride", _Z), ("kv_rank", _Z), ("kv_stride", _Z), ("window", _Z), ("ring", _Z), ("n_slots", _Z),
    ("scale", _F), ("q", _P), ("q_dtype", _I), ("q_stride", _Z), ("w_dtype", _I), ("uk", _P), ("uv", _P),
    ("cache", _P), ("n_splits", _Z), ("scratch", _P), ("out", _P), ("out_dtype", _I), ("out_stride", _Z)])


def up_to(n: int, multiple: int) -> int:
    return -(-int(n) // multiple) * multiple


def padded(n: int) -> int:
    """Row strides: a whole number of 64-entry pieces, the matrix kernels' k step."""
    return up_to(n, 64)


@dataclass
class Linear:
    """Weight rows on the device, columns padded with zeros to ``k``."""
    w: object
    rows: int
    width: int
    k: int


@dataclass
class Join:
    """How a sublayer's result joins the residual stream: times ``scale`` (a vector), or, with
    ``norm``, through an RMS norm with that weight."""
    scale: object = None
    norm: object = None
    eps: float = 0.0


@dataclass
class Pending:
    """A result that the next norm still has to add to the stream: y / rms(y) * weight, where y is
    a row of ``rows``, or ``scale`` times the sum of ``top`` of them (``places`` [rows, top], None:
    consecutive ones)."""
    rows: object
    weight: object
    eps: float
    top: int = 0
    places: object = None
    scale: float = 1.0

    def fields(self) -> dict:
        return dict(pending=self.rows, pending_stride=self.rows.shape[1], pending_weight=self.weight,
                    pending_eps=self.eps, pending_top=self.top, pending_rows=self.places, pending_scale=self.scale)

    def at(self, torch, index) -> "Pending":
        """The same for the rows ``index`` (a device tensor)."""
        if self.top == 0:
            return Pending(self.rows.index_select(0, index), self.weight, self.eps)
        if self.places is None:
            places = index[:, None] * self.top + torch.arange(self.top, device=index.device)
        else:
            places = self.places.index_select(0, index)
        return Pending(self.rows, self.weight, self.eps, self.top, places.to(torch.int32).contiguous(), self.scale)


class Weights:
    """Packs a model's tensors for the kernels: ``dtype`` is the dtype of the linears."""

    def __init__(self, torch, device, serving: str):
        self.torch, self.device = torch, device
        self.dtype = torch.float32 if serving == "float32" else torch.bfloat16
        self.tag = QK_F32 if serving == "float32" else QK_BF16

    def to(self, t, dtype=None):
        return t.to(self.device, dtype or self.dtype).contiguous()

    def vector(self, t, offset: float = 0.0):
        """In float32, plus ``offset`` (1 for weights that are kept as offsets from one)."""
        v = self.to(t, self.torch.float32)
        return v + offset if offset else v

    def matrix(self, *mats) -> Linear:
        """The matrices' rows one after the other (they share their input)."""
        width = mats[0].shape[1]
        k = padded(width)
        rows = sum(m.shape[0] for m in mats)
        w = self.torch.zeros(rows, k, dtype=self.dtype, device=self.device)
        w[:, :width] = self.torch.cat([self.to(m) for m in mats])
        return Linear(w, rows, width, k)

    def heads(self, mat, heads: int, size: int, stride: int):
        """Head-major rows with every head's rows padded to ``stride``."""
        m = self.to(mat).reshape(heads, size, mat.shape[1])
        out = self.torch.zeros(heads, stride, mat.shape[1], dtype=self.dtype, device=self.device)
        out[:, :size] = m
        return out.reshape(heads * stride, mat.shape[1])

    def head_columns(self, mat, heads: int, size: int, stride: int):
        """The columns of every head padded to ``stride``."""
        m = self.to(mat)
        out = self.torch.zeros(m.shape[0], heads, stride, dtype=self.dtype, device=self.device)
        out[:, :, :size] = m.reshape(m.shape[0], heads, size)
        return out.reshape(m.shape[0], heads * stride)

    def halves(self, mat, width: int) -> Linear:
        """A matrix over [x ; y], each half's columns padded on their own."""
        half = padded(width)
        m = self.to(mat)
        w = self.torch.zeros(m.shape[0], 2 * half, dtype=self.dtype, device=self.device)
        w[:, :width] = m[:, :width]
        w[:, half:half + width] = m[:, width:]
        return Linear(w, m.shape[0], width, 2 * half)

    def gated_pair(self, gate, up) -> Linear:
        """Blocks of 32 gate rows and their 32 up rows, so that a kernel that has one has both."""
        ff, width = gate.shape
        k, blocks = padded(width), up_to(ff, 32) // 32
        w = self.torch.zeros(blocks, 2, 32, k, dtype=self.dtype, device=self.device)
        for which, m in enumerate((gate, up)):
            full = self.torch.zeros(blocks * 32, width, dtype=self.dtype, device=self.device)
            full[:ff] = self.to(m)
            w[:, which, :, :width] = full.reshape(blocks, 32, width)
        return Linear(w, blocks * 64, width, k)


    def stacked(self, lins) -> Linear:
        """Linears of one shape one after the other; the shape stays that of one."""
        one = lins[0]
        return Linear(self.torch.stack([m.w.reshape(one.rows, one.k) for m in lins]), one.rows, one.width, one.k)


class Rows:
    """Activation buffers and row descriptions for up to ``cap`` rows at a time.

    The residual stream alternates between ``x`` and ``x2``; ``pending`` is a result that the next
    norm still has to add to it.  ``act`` holds the dtype of what only matrix products read:
    float32 where the vector form takes the rows, else the linears' dtype."""

    def __init__(self, torch, device, cap: int, stride: int, weights: Weights, vector: bool):
        self.torch, self.device, self.cap, self.stride = torch, device, cap, stride
        i32 = dict(dtype=torch.int32, device=device)
        self.ids, self.slots = torch.zeros(cap, **i32), torch.arange(cap, **i32)
        self.positions = torch.zeros(cap, **i32)
        self.seg_first, self.seg_len = torch.arange(cap, **i32), torch.ones(cap, **i32)
        self.seg_row = torch.zeros(cap, **i32)
        self.n = self.segments = cap
        self.portion = None            # (slot, first position) when the rows are one portion
        self.act = torch.float32 if vector else weights.dtype
        self.act_tag = QK_F32 if self.act == torch.float32 else QK_BF16
        self.weights = weights
        self._buffers, self.split_floats = {}, {}
        self.x, self.x2 = self.f32("x", stride), self.f32("x2", stride)
        self.pending = None            # a Pending
        self.routes = {}               # per expert table: what qk_route leaves (Route)
        self._route_jobs = None

    def f32(self, name: str, width: int):
        return self.buffer(name, width, self.torch.float32)

    def buffer(self, name: str, width: int, dtype=None, rows: int | None = None):
        """A zeroed buffer of ``cap`` rows, shared by every layer that asks for the same one."""
        dtype = dtype or self.act
        key = (name, int(width), dtype, rows)
        if key not in self._buffers:
            self._buffers[key] = self.torch.zeros(rows or self.cap, int(width), dtype=dtype, device=self.device)
        return self._buffers[key]

    def call(self, lin: Linear, **fields) -> DenseCall:
        d = DenseCall(tokens=self.n, positions=self.positions.data_ptr(), slots=self.slots.data_ptr(),
                      ids=self.ids.data_ptr(), x_dtype=QK_F32, width=lin.width, k=lin.k,
                      w_dtype=self.weights.tag, w=lin.w.data_ptr(), rows=lin.rows, w_stride=lin.k,
                      out_dtype=QK_F32)
        for name, value in fields.items():
            if hasattr(value, "data_ptr"):
                value = value.data_ptr()
            setattr(d, name, value)
        return d

    def dense(self, ctx, lin: Linear, **fields) -> None:
        d = self.call(lin, **fields)
        plain = d.input == IN_PLAIN and d.x_dtype == self.weights.tag
        if d.experts and not d.by_choice:
            plain = False
        if not plain and _lib.lib().qk_dense_form(self.n, lin.k, self.weights.tag) != FORM_VECTOR:
            scratch = self.buffer("input", lin.k, self.weights.dtype, rows=self.cap * max(1, d.top))
            d.scratch, d.scratch_bytes = scratch.data_ptr(), scratch.numel() * scratch.element_size()
        check(_lib.lib().qk_dense(ctx.handle, ctypes.byref(d)))

    def stream_fields(self, norm: int, norm_weight, eps: float) -> dict:
        """Input fields of a linear behind a norm of the residual stream; takes ``pending`` in."""
        f = dict(input=IN_NORM, x=self.x, x_stride=self.stride, norm=norm, norm_weight=norm_weight, norm_eps=eps)
        if self.pending is not None:
            f.update(self.pending.fields(), x_out=self.x2)
        return f

    def settle(self) -> None:
        """After a linear with ``stream_fields``: the stream is where it has been written."""
        if self.pending is not None:
            self.x, self.x2 = self.x2, self.x
            self.pending = None

    def join(self, ctx, lin: Linear, join: Join | None, **fields) -> None:
        """A linear whose result joins the stream; one that joins through a norm is left pending."""
        join = join or Join()
        if join.norm is None:
            self.dense(ctx, lin, **fields, **self.residual_fields(join.scale))
            return
        y = self.f32("result", self.stride)
        self.dense(ctx, lin, **fields, out=y, out_stride=self.stride)
        self.pending = Pending(y, join.norm, join.eps)

    def residual_fields(self, scale) -> dict:
        """Output fields of a linear that adds to the stream; bfloat16 rows also keep a copy for
        the plain linear that may follow."""
        f = dict(output=OUT_RESIDUAL, residual=self.x, residual_stride=self.stride, out_scale=scale)
        if self.act != self.torch.float32:
            f.update(out=self.buffer("stream", self.stride), out_stride=self.stride, out_dtype=self.act_tag)
        return f

    def stream_rows(self):
        """The stream as a plain input (after ``residual_fields``): (buffer, dtype tag)."""
        if self.act != self.torch.float32:
            return self.buffer("stream", self.stride), self.act_tag
        return self.x, QK_F32

    def route(self, ctx, tables, width: int, vocab: int) -> None:
        """Sorts these rows' choices by expert for every table (one launch), where a matrix form will
        read them (``width``: the width of the stream)."""
        if not tables or _lib.lib().qk_dense_form(self.n, padded(width), self.weights.tag) == FORM_VECTOR:
            return
        torch = self.torch
        if self._route_jobs is None:
            jobs = (RouteJob * len(tables))()
            for job, table in zip(jobs, tables):
                r = self.routes[id(table)] = Route(torch, self.device, self.cap, table)
                job.table, job.places, job.offsets, job.tiles = (x.data_ptr() for x in (table.rows, r.places, r.offsets, r.tiles))
                job.top, job.experts = table.top, table.experts
            self._route_jobs = torch.frombuffer(bytearray(jobs), dtype=torch.uint8).to(self.device)
        lib = _lib.lib()
        tile = lib.qk_route_tile_rows(self.n, padded(width), self.weights.tag)
        check(lib.qk_route(ctx.handle, self._route_jobs.data_ptr(), len(tables), max(t.experts for t in tables),
                           self.ids.data_ptr(), self.n, vocab, tile))


class ExpertTable:
    """Every token id's experts: [vocab, top] on the device."""

    def __init__(self, weights: Weights, table, experts: int):
        self.rows = weights.to(table, weights.torch.int32)
        self.experts, self.top = int(experts), int(table.shape[1])


class Route:
    """Room for the choices of up to ``cap`` rows, sorted by expert."""

    def __init__(self, torch, device, cap: int, table: ExpertTable):
        i32 = dict(dtype=torch.int32, device=device)
        n = cap * table.top
        self.places = torch.zeros(cap, table.top, **i32)
        self.offsets = torch.zeros(table.experts + 1, **i32)
        self.tiles = torch.zeros(1 + 5 * (-(-n // 64) + table.experts), **i32)


class RingCache:
    """The last ``rows`` latents of every slot: position p of a slot lies in row p mod rows."""

    def __init__(self, torch, device, slots: int, rows: int, stride: int, dtype):
        self.rows, self.stride = int(rows), int(stride)
        self.data = torch.zeros(slots, self.rows, self.stride, dtype=dtype, device=device)


class KeyValueCache:
    """Keys and values of every position of every slot, head by head.  A row reads no position
    beyond its own, so a slot needs no clearing between sequences."""

    def __init__(self, torch, device, slots: int, kv_heads: int, rows: int, dim_stride: int, vdim_stride: int, dtype):
        self.rows = int(rows)
        self.k = torch.zeros(slots, kv_heads, self.rows, dim_stride, dtype=dtype, device=device)
        self.v = torch.zeros(slots, kv_heads, self.rows, vdim_stride, dtype=dtype, device=device)


class RecurrentState:
    """Per slot: the heads' float32 state matrices and the convolution's last inputs.  A portion
    that starts at position 0 starts from zero, so a slot needs no clearing between sequences."""

    def __init__(self, torch, device, slots: int, heads: int, dim: int, vdim: int, taps: int, channels: int):
        f32 = dict(dtype=torch.float32, device=device)
        self.matrix = torch.zeros(slots, heads, vdim, dim, **f32)
        self.conv = torch.zeros(slots, taps, channels, **f32)


class LatentAttention:
    """Latent attention without positions under a sliding window (None: no window).

    Portions of more than ``absorbed_rows`` rows (bfloat16, head sizes up to 256) expand the
    window's latents into keys and values by a matrix product; everything else works on the
    latents themselves."""

    absorbed_rows = 16

    def __init__(self, weights: Weights, tensors: dict, *, heads: int, dim: int, vdim: int, kv_rank: int,
                 q_rank: int, scale: float, window: int | None, eps: float):
        self.heads, self.dim, self.vdim, self.kv_rank, self.q_rank = heads, dim, vdim, kv_rank, q_rank
        self.scale, self.window, self.eps, self.weights = float(scale), window, float(eps), weights
        self.dim_stride, self.vdim_stride, self.kv_stride = up_to(dim, 16), up_to(vdim, 16), padded(kv_rank)
        t, w = tensors, weights
        self.down = w.matrix(t["dq"], t["dkv"])
        self.q_norm, self.kv_norm = w.vector(t["dq.norm"]), w.vector(t["dkv.norm"])
        self.uq = w.matrix(w.heads(t["uq"], heads, dim, self.dim_stride))
        self.ukv = w.matrix(w.heads(t["uk"], heads, dim, self.dim_stride),
                            w.heads(t["uv"], heads, vdim, self.vdim_stride))
        self.out = w.matrix(t["o"])
        self.expands = w.tag == QK_BF16 and max(self.dim_stride, self.vdim_stride) <= 256

    def make_state(self, torch, device, slots: int, max_seq: int, portion: int) -> RingCache:
        # a portion is appended before its first row is read, so the ring holds a window beside it
        window = min(self.window or max_seq, max_seq)
        return RingCache(torch, device, slots, min(window - 1 + portion, max(max_seq, window)), self.kv_stride,
                         self.weights.dtype)

    def n_splits(self, rows: int, window: int) -> int:
        """Key splits of the absorbed form: about two blocks per SM, 32 keys or more each."""
        groups = -(-self.heads // 16) if self.weights.tag == QK_BF16 else self.heads
        want = max(1, min(64, 296 // max(1, rows * groups), -(-window // 32)))
        return want // 8 * 8 if want >= 8 else want   # (clusters of eight merge their splits)

    def _split_floats(self, rows: Rows, window: int) -> int:
        """Scratch of the absorbed form for any number of rows it may get in this workspace."""
        key = (self.heads, self.kv_stride, window)
        if key not in rows.split_floats:
            most = min(rows.cap, self.absorbed_rows) if self.expands and rows.portion is not None else rows.cap
            rows.split_floats[key] = max(_lib.lib().qk_latent_scratch(
                m, self.heads, self.kv_stride, self.n_splits(m, window)) for m in range(1, most + 1)) // 4
        return rows.split_floats[key]

    def forward(self, ctx, rows: Rows, norm: int, norm_weight, norm_eps: float, join, state: RingCache,
                max_seq: int) -> None:
        lib, n = _lib.lib(), rows.n
        window = min(self.window or max_seq, max_seq, state.rows)
        lat_stride = up_to(self.q_rank + self.kv_rank, 4)
        lat = rows.f32("latents", lat_stride)
        rows.dense(ctx, self.down, **rows.stream_fields(norm, norm_weight, norm_eps), out=lat, out_stride=lat_stride)
        rows.settle()
        expanded = self.expands and rows.portion is not None and n > self.absorbed_rows
        q_stride = padded(self.heads * self.dim_stride)
        q = rows.buffer("query", q_stride, self.weights.dtype if expanded else rows.torch.float32)
        append = LatentAppend(src=lat.data_ptr() + 4 * self.q_rank, src_stride=lat_stride, width=self.kv_rank,
                              weight=self.kv_norm.data_ptr(), eps=self.eps, cache_dtype=self.weights.tag,
                              cache=state.data.data_ptr(), ring=state.rows, stride=state.stride)
        rows.dense(ctx, self.uq, input=IN_NORM, x=lat, x_stride=lat_stride, norm=NORM_RMS, norm_weight=self.q_norm,
                   norm_eps=self.eps, append=append, out=q, out_stride=q_stride,
                   out_dtype=self.weights.tag if expanded else QK_F32)
        o_stride = padded(self.heads * self.vdim)
        att = rows.buffer("attention", o_stride)
        if expanded:
            self._expanded(ctx, rows, q, q_stride, att, o_stride, state, window)
        else:
            splits = self.n_splits(n, window)
            scratch = rows.buffer("splits", self._split_floats(rows, window), rows.torch.float32, rows=1)
            c = LatentCall(
                tokens=n, positions=rows.positions.data_ptr(), slots=rows.slots.data_ptr(), heads=self.heads,
                dim=self.dim, dim_stride=self.dim_stride, vdim=self.vdim, vdim_stride=self.vdim_stride,
                kv_rank=self.kv_rank, kv_stride=self.kv_stride, window=window, ring=state.rows,
                n_slots=state.data.shape[0], scale=self.scale, q=q.data_ptr(), q_dtype=QK_F32, q_stride=q_stride,
                w_dtype=self.weights.tag, uk=self.ukv.w.data_ptr(),
                uv=self.ukv.w[self.heads * self.dim_stride:].data_ptr(), cache=state.data.data_ptr(),
                n_splits=splits, scratch=scratch.data_ptr(), out=att.data_ptr(), out_dtype=rows.act_tag,
                out_stride=o_stride)
            check(lib.qk_latent_attention(ctx.handle, ctypes.byref(c)))
        rows.join(ctx, self.out, join, input=IN_PLAIN, x=att, x_dtype=rows.act_tag, x_stride=o_stride)

    def _expanded(self, ctx, rows: Rows, q, q_stride, att, o_stride, state: RingCache, window: int) -> None:
        lib = _lib.lib()
        slot, p0 = rows.portion
        first = max(0, p0 - window + 1)
        keys = p0 + rows.n - first
        kv_row = padded(self.ukv.rows)
        lat = rows.buffer("window", self.kv_stride, self.weights.dtype, rows=state.rows)
        kv = rows.buffer("keys", kv_row, self.weights.dtype, rows=state.rows)
        check(lib.qk_latent_gather(ctx.handle, c_void_p(state.data.data_ptr()), self.weights.tag, state.rows,
                                   state.stride, slot, first, keys, c_void_p(lat.data_ptr())))
        d = rows.call(self.ukv, tokens=keys, input=IN_PLAIN, x=lat, x_dtype=self.weights.tag, x_stride=self.kv_stride,
                      out=kv, out_stride=kv_row, out_dtype=self.weights.tag)
        check(lib.qk_dense(ctx.handle, ctypes.byref(d)))
        check(lib.qk_window_attention(ctx.handle, c_void_p(q.data_ptr()), q_stride, c_void_p(kv.data_ptr()), kv_row,
                                      first, keys, p0, rows.n, self.heads, self.dim_stride, self.vdim,
                                      self.vdim_stride, window, self.scale, c_void_p(att.data_ptr()), o_stride))


@functools.lru_cache(maxsize=64)
def distance_buckets(rows: int, bias_max: float, most: int = 1 << 24) -> tuple:
    """The table row of every distance, up to the first one from which on it is the last row: the
    near half one by one, then logarithmic steps that reach the end at ``bias_max``."""
    half = rows // 2
    if half < 1 or bias_max <= half:
        raise ValueError(f"a distance bias of {rows} rows cannot reach to a distance of {bias_max}")
    out, n = [], 0
    while not out or out[-1] < rows - 1:
        if n >= most:
            raise ValueError(f"a distance bias that reaches to {bias_max} is not supported")
        out.append(n if n < half else
                   min(rows - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (rows - half))))
        n += 1
    return tuple(out)


class GroupedAttention:
    """Causal attention with ``heads / kv_heads`` query heads per key/value head over the whole
    sequence.  Positions enter through a factor on the queries, 1 + coef ln(floor((p + 1) / every) + 1)
    (``temperature``: (coef, every) or None), and a learned bias per head and distance bucket
    (``bias_max``: where the last bucket begins; None: no bias).

    bfloat16 portions of more than ``row_rows`` rows take the portion kernel, everything else the
    kernel that serves rows one by one."""

    row_rows = 16

    def __init__(self, weights: Weights, tensors: dict, *, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 temperature: tuple | None, bias_max: float | None, eps: float):
        del eps   # (no norm inside)
        t, w = tensors, weights
        self.heads, self.kv_heads, self.dim, self.vdim, self.weights = heads, kv_heads, dim, vdim, weights
        self.scale, self.temperature = float(scale), temperature
        self.dim_stride, self.vdim_stride = up_to(dim, 16), up_to(vdim, 16)
        self.proj = w.matrix(w.heads(t["q"], heads, dim, self.dim_stride), w.heads(t["k"], kv_heads, dim, self.dim_stride),
                             w.heads(t["v"], kv_heads, vdim, self.vdim_stride))
        self.out = w.matrix(w.head_columns(t["o"], heads, vdim, self.vdim_stride))
        self.bias = None
        if bias_max is not None:   # [heads, distances]: the bias of every distance until it stops changing
            rel = w.vector(t["rel"])
            buckets = w.torch.tensor(distance_buckets(rel.shape[0], bias_max), device=rel.device)
            self.bias = rel.index_select(0, buckets).t().contiguous()
        self.tiled = w.tag == QK_BF16 and max(self.dim_stride, self.vdim_stride) <= 256

    def make_state(self, torch, device, slots: int, max_seq: int, portion: int) -> KeyValueCache:
        return KeyValueCache(torch, device, slots, self.kv_heads, max_seq, self.dim_stride, self.vdim_stride,
                             self.weights.dtype)

    def n_splits(self, rows: int, max_seq: int) -> int:
        """Key splits: about two blocks per SM, 64 keys or more each."""
        group = self.heads // self.kv_heads
        blocks = rows * (self.kv_heads * -(-group // 8) if self.tiled else self.heads)
        return max(1, min(24, 296 // blocks, -(-max_seq // 64)))

    def _scratch(self, rows: Rows, n_splits: int):
        """Partial results and counters (zero between calls) for this number of rows and splits."""
        floats = _lib.lib().qk_grouped_scratch(rows.n, self.heads, self.kv_heads, self.vdim_stride, n_splits) // 4
        return rows.buffer(f"grouped splits {rows.n} {self.heads} {self.vdim_stride} {n_splits}", floats,
                           rows.torch.float32, rows=1)

    def forward(self, ctx, rows: Rows, norm: int, norm_weight, norm_eps: float, join, state: KeyValueCache,
                max_seq: int) -> None:
        lib, n = _lib.lib(), rows.n
        tiled = self.tiled and rows.portion is not None and n > self.row_rows
        dtype, tag = (rows.weights.dtype, self.weights.tag) if tiled else (rows.torch.float32, QK_F32)
        stride = up_to(self.proj.rows, 8)
        proj = rows.buffer("heads", stride, dtype)
        rows.dense(ctx, self.proj, **rows.stream_fields(norm, norm_weight, norm_eps), out=proj, out_stride=stride, out_dtype=tag)
        rows.settle()
        o_stride = self.out.k
        att = rows.buffer("attention", o_stride)
        coef, every = self.temperature or (0.0, 0.0)
        c = GroupedCall(
            tokens=n, positions=rows.positions.data_ptr(), slots=rows.slots.data_ptr(), heads=self.heads,
            kv_heads=self.kv_heads, dim_stride=self.dim_stride, vdim_stride=self.vdim_stride, s_max=state.rows,
            n_slots=state.k.shape[0], scale=self.scale, temp_coef=coef, temp_every=every,
            bias=None if self.bias is None else self.bias.data_ptr(), bias_len=0 if self.bias is None else self.bias.shape[1],
            proj=proj.data_ptr(), proj_dtype=tag, proj_stride=stride, cache_dtype=self.weights.tag,
            cache_k=state.k.data_ptr(), cache_v=state.v.data_ptr(), out=att.data_ptr(), out_dtype=rows.act_tag,
            out_stride=o_stride)
        if rows.portion is not None:
            check(lib.qk_grouped_append(ctx.handle, ctypes.byref(c)))
        if tiled:
            c.slot, c.first_position = rows.portion
            check(lib.qk_grouped_portion(ctx.handle, ctypes.byref(c)))
        else:
            c.append = int(rows.portion is None)   # (a step has one row per slot)
            c.n_splits = self.n_splits(n, state.rows)
            c.scratch = self._scratch(rows, c.n_splits).data_ptr()
            check(lib.qk_grouped_attention(ctx.handle, ctypes.byref(c)))
        rows.join(ctx, self.out, join, input=IN_PLAIN, x=att, x_dtype=rows.act_tag, x_stride=o_stride)


class GatedDelta:
    """Gated delta rule with short causal convolutions and one decay per head."""

    def __init__(self, weights: Weights, tensors: dict, *, heads: int, kv_heads: int, dim: int, vdim: int, taps: int,
                 eps: float, unit_eps: float):
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = heads, kv_heads, dim, vdim, taps
        self.eps, self.unit_eps = float(eps), float(unit_eps)
        t, w = tensors, weights
        self.proj = w.matrix(t["q"], t["k"], t["v"], t["g"], t["b"], t["a"])
        self.channels = 2 * kv_heads * dim + heads * vdim
        self.gate_at = self.channels
        self.beta_at = self.gate_at + heads * vdim
        self.decay_at = self.beta_at + heads
        self.conv = [w.vector(t[n + ".conv"]) for n in ("q", "k", "v")]
        self.a_log, self.dt_bias, self.norm = w.vector(t["A_log"]), w.vector(t["dt_bias"]), w.vector(t["norm"])
        self.out = w.matrix(t["o"])

    def make_state(self, torch, device, slots: int, max_seq: int, portion: int) -> RecurrentState:
        return RecurrentState(torch, device, slots, self.heads, self.dim, self.vdim, self.taps, self.channels)

    def forward(self, ctx, rows: Rows, norm: int, norm_weight, norm_eps: float, join, state: RecurrentState,
                max_seq: int) -> None:
        stride = up_to(self.proj.rows, 8)
        proj = rows.f32("projections", stride)
        rows.dense(ctx, self.proj, **rows.stream_fields(norm, norm_weight, norm_eps), out=proj, out_stride=stride)
        rows.settle()
        o_stride = padded(self.heads * self.vdim)
        out = rows.f32("readout", o_stride)
        qkv, gates = rows.f32("qkv", self.channels), rows.buffer("gates", self.heads * 20, rows.torch.float32, rows=up_to(rows.cap, 8))
        c = DeltaCall(tokens=rows.n, segments=rows.segments, positions=rows.positions.data_ptr(),
                      slots=rows.slots.data_ptr(), seg_first=rows.seg_first.data_ptr(),
                      seg_len=rows.seg_len.data_ptr(), seg_row=rows.seg_row.data_ptr(), heads=self.heads,
                      kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, taps=self.taps, proj=proj.data_ptr(),
                      proj_stride=stride, beta_offset=self.beta_at, decay_offset=self.decay_at,
                      conv_q=self.conv[0].data_ptr(), conv_k=self.conv[1].data_ptr(), conv_v=self.conv[2].data_ptr(),
                      a_log=self.a_log.data_ptr(), dt_bias=self.dt_bias.data_ptr(), unit_eps=self.unit_eps,
                      conv_state=state.conv.data_ptr(), state=state.matrix.data_ptr(), qkv=qkv.data_ptr(),
                      gates=gates.data_ptr(), out=out.data_ptr(), out_stride=o_stride)
        check(_lib.lib().qk_delta(ctx.handle, ctypes.byref(c)))
        rows.join(ctx, self.out, join, input=IN_GATED, x=out, x_stride=o_stride, gate=proj.data_ptr() + 4 * self.gate_at,
                  gate_stride=stride, group=self.vdim, norm_weight=self.norm, norm_eps=self.eps)


class GatedMlp:
    """W_down (act(W_gate h) * (W_up h))."""

    def __init__(self, weights: Weights, tensors: dict, *, activation: str):
        self.pair = weights.gated_pair(tensors["gate"], tensors["up"])
        self.down = weights.matrix(tensors["down"])
        self.act = ACTIVATIONS[activation]

    def forward(self, ctx, rows: Rows, norm: int, norm_weight, norm_eps: float, join) -> None:
        stride = self.down.k
        ff = rows.buffer("ff", stride)
        rows.dense(ctx, self.pair, **rows.stream_fields(norm, norm_weight, norm_eps), output=OUT_GLU,
                   activation=self.act, out=ff, out_stride=stride, out_dtype=rows.act_tag)
        rows.settle()
        rows.join(ctx, self.down, join, input=IN_PLAIN, x=ff, x_dtype=rows.act_tag, x_stride=stride)


class TableExperts:
    """Gated feed-forwards of which every token id has ``top``, named by a table, that weigh the
    same.  Their sum is formed where it joins the stream, through a norm."""

    def __init__(self, weights: Weights, tensors: dict, *, experts: int, activation: str):
        t = tensors
        self.table = ExpertTable(weights, t["table"], experts)
        self.pair = weights.stacked([weights.gated_pair(t[f"e{e}.gate"], t[f"e{e}.up"]) for e in range(experts)])
        self.down = weights.stacked([weights.matrix(t[f"e{e}.down"]) for e in range(experts)])
        self.act = ACTIVATIONS[activation]

    def forward(self, ctx, rows: Rows, norm: int, norm_weight, norm_eps: float, join) -> None:
        if join is None or join.norm is None:
            raise ValueError("the experts' results join the stream through a norm")
        top, stride = self.table.top, self.down.k
        chosen = dict(experts=self.table.experts, top=top, table=self.table.rows, vocab=self.table.rows.shape[0])
        places = None   # the vector form: consecutive
        if _lib.lib().qk_dense_form(rows.n, self.pair.k, rows.weights.tag) != FORM_VECTOR:
            r = rows.routes[id(self.table)]
            places = r.places
            chosen.update(places=places, offsets=r.offsets, tiles=r.tiles)
        ff = rows.buffer("expert ff", stride, rows=rows.cap * top)
        rows.dense(ctx, self.pair, **rows.stream_fields(norm, norm_weight, norm_eps), output=OUT_GLU,
                   activation=self.act, out=ff, out_stride=stride, out_dtype=rows.act_tag, **chosen)
        rows.settle()
        y = rows.buffer("expert result", rows.stride, rows.torch.float32, rows=rows.cap * top)
        rows.dense(ctx, self.down, input=IN_PLAIN, x=ff, x_dtype=rows.act_tag, x_stride=stride, by_choice=1, out=y,
                   out_stride=rows.stride, **chosen)
        rows.pending = Pending(y, join.norm, join.eps, top, places, 1.0 / top)


class TokenSide:
    """Per-layer token input: norm(W_proj (gelu(W_gate x) * e)) is left pending on the stream, e
    being ``dim`` columns of the token's row of ``table`` from ``offset`` on."""

    def __init__(self, weights: Weights, tensors: dict, table, *, dim: int, offset: int, eps: float):
        self.gate, self.proj = weights.matrix(tensors["gate"]), weights.matrix(tensors["proj"])
        self.norm, self.table, self.dim, self.offset, self.eps = (weights.vector(tensors["norm"]), table, dim, offset,
                                                                  float(eps))

    def forward(self, ctx, rows: Rows) -> None:
        x, tag = rows.stream_rows()
        s = rows.buffer("side", self.proj.k)
        rows.dense(ctx, self.gate, input=IN_PLAIN, x=x, x_dtype=tag, x_stride=rows.stride, output=OUT_SIDE,
                   activation=ACTIVATIONS["gelu_tanh"], side=self.table, side_dtype=rows.weights.tag,
                   side_stride=self.table.shape[1], side_offset=self.offset, vocab=self.table.shape[0], out=s,
                   out_stride=self.proj.k, out_dtype=rows.act_tag)
        y = rows.f32("side result", rows.stride)
        rows.dense(ctx, self.proj, input=IN_PLAIN, x=s, x_dtype=rows.act_tag, x_stride=self.proj.k, out=y,
                   out_stride=rows.stride)
        rows.pending = Pending(y, self.norm, self.eps)
