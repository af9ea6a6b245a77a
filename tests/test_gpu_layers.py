"""The building blocks of layered decoders one call at a time, against float64: every form of
the dense linear with every input and output, the latent append, the two attention forms."""

import ctypes

import numpy as np
import pytest

from quantibbler_b200 import _lib
from quantibbler_b200._lib import QK_BF16, QK_F32, KernelError, check

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def dev(gpu_ctx):
    import torch
    from quantibbler_b200 import layers
    gpu_ctx.set_stream(torch.cuda.current_stream().cuda_stream)
    return gpu_ctx, torch, layers


def rel(got, want):
    return float((got.double() - want).abs().max() / want.abs().max())


def silu(z):
    return z / (1 + (-z).exp())


TOKENS = [1, 2, 3, 4, 5, 8, 9, 33, 64, 65, 128, 129, 300]


@pytest.mark.parametrize("serving,tol", [("float32", 4e-6), ("bfloat16", 1e-2)])
@pytest.mark.parametrize("tokens", TOKENS)
def test_dense_inputs_and_outputs(dev, tokens, serving, tol):
    ctx, torch, L = dev
    g = torch.Generator(device="cuda").manual_seed(tokens)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    w = L.Weights(torch, torch.device("cuda"), serving)
    bf = lambda t: t.bfloat16().float()   # weights both dtypes hold exactly
    for width, rows_out in ((72, 40), (200, 257), (1000, 96)):
        stride = L.padded(width)
        rows = L.Rows(torch, torch.device("cuda"), tokens, stride, w, vector=tokens <= 4)
        x = rows.x
        x[:, :width] = rnd(tokens, width) * 2 + 1
        xd = x[:, :width].double()
        y = rnd(tokens, stride) * 3
        y[:, width:] = 0
        yd = y[:, :width].double()
        pw, nw = rnd(width) * 0.5 + 1, rnd(width) * 0.3 + 1
        m = bf(rnd(rows_out, width) / width ** 0.5)
        lin = w.matrix(m)
        out = torch.zeros(tokens, L.up_to(rows_out, 8), device="cuda")
        o = dict(out=out, out_stride=out.shape[1])

        def ran(**f):
            out.zero_()
            rows.dense(ctx, lin, **f, **o)
            return out[:, :rows_out]

        # plain
        assert rel(ran(input=L.IN_PLAIN, x=x, x_stride=stride), xd @ m.double().T) < tol
        # pending residual, layer norm and rms norm
        h = xd + yd / (yd.pow(2).mean(1, keepdim=True) + 1e-3).sqrt() * pw.double()
        pend = dict(pending=y, pending_stride=stride, pending_weight=pw, pending_eps=1e-3, x_out=rows.x2)
        c = h - h.mean(1, keepdim=True)
        ln = c / (c.pow(2).mean(1, keepdim=True) + 1e-4).sqrt() * nw.double()
        rn = h / (h.pow(2).mean(1, keepdim=True) + 1e-4).sqrt() * nw.double()
        base = dict(input=L.IN_NORM, x=x, x_stride=stride, norm_weight=nw, norm_eps=1e-4)
        assert rel(ran(**base, **pend, norm=L.NORM_LAYER), ln @ m.double().T) < tol
        assert rel(rows.x2[:, :width], h) < 2e-6
        assert rel(ran(**base, **pend, norm=L.NORM_RMS), rn @ m.double().T) < tol
        # residual output with a scale
        res, s = rnd(tokens, out.shape[1]), rnd(rows_out)
        want = res[:, :rows_out].double() + (xd @ m.double().T) * s.double()
        rows.dense(ctx, lin, input=L.IN_PLAIN, x=x, x_stride=stride, output=L.OUT_RESIDUAL, residual=res,
                   residual_stride=out.shape[1], out_scale=s, **o)
        assert rel(res[:, :rows_out], want) < tol
        assert torch.equal(out[:, :rows_out], res[:, :rows_out])
        # gated pair
        up = bf(rnd(rows_out, width) / width ** 0.5)
        pair = w.gated_pair(m, up)
        act = torch.zeros(tokens, pair.rows // 2, device="cuda")
        for name, fn in (("relu", torch.relu), ("silu", silu)):
            rows.dense(ctx, pair, input=L.IN_PLAIN, x=x, x_stride=stride, output=L.OUT_GLU,
                       activation=L.ACTIVATIONS[name], out=act, out_stride=act.shape[1])
            want = fn(xd @ m.double().T) * (xd @ up.double().T)
            assert rel(act[:, :rows_out], want) < tol
            assert not act[:, rows_out:].any()
        # token-side product
        table = w.to(bf(rnd(11, rows_out + 9)))
        rows.ids.copy_(torch.arange(tokens) % 11)
        rows.dense(ctx, lin, input=L.IN_PLAIN, x=x, x_stride=stride, output=L.OUT_SIDE,
                   activation=L.ACTIVATIONS["gelu_tanh"], side=table, side_dtype=w.tag, side_stride=table.shape[1],
                   side_offset=5, vocab=11, **o)
        z = xd @ m.double().T
        want = torch.nn.functional.gelu(z, approximate="tanh") * table[rows.ids.long()][:, 5:5 + rows_out].double()
        assert rel(out[:, :rows_out], want) < tol


@pytest.mark.parametrize("serving,tol", [("float32", 4e-6), ("bfloat16", 1e-2)])
@pytest.mark.parametrize("tokens", [1, 4, 6, 70])
def test_dense_concatenated_and_gated_inputs(dev, tokens, serving, tol):
    ctx, torch, L = dev
    g = torch.Generator(device="cuda").manual_seed(7)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    w = L.Weights(torch, torch.device("cuda"), serving)
    width, stride = 90, 128
    rows = L.Rows(torch, torch.device("cuda"), tokens, stride, w, vector=tokens <= 4)
    rows.x[:, :width] = rnd(tokens, width)
    second = torch.zeros(tokens, stride, device="cuda")
    second[:, :width] = rnd(tokens, width)
    m = (rnd(70, 2 * width) / 13).bfloat16().float()
    out = torch.zeros(tokens, 72, device="cuda")
    rows.dense(ctx, w.halves(m, width), input=L.IN_CONCAT, x=rows.x, x_stride=stride, second=second, out=out, out_stride=72)
    both = torch.cat([rows.x[:, :width], second[:, :width]], 1).double()
    assert rel(out[:, :70], both @ m.double().T) < tol
    # groups of 18: rms norm, weight, silu gate
    gate, nw = rnd(tokens, 96), rnd(18)
    m = (rnd(33, width) / 9).bfloat16().float()
    rows.dense(ctx, w.matrix(m), input=L.IN_GATED, x=rows.x, x_stride=stride, gate=gate, gate_stride=96, group=18,
               norm_weight=nw, norm_eps=1e-3, out=out, out_stride=72)
    v = rows.x[:, :width].double().reshape(tokens, 5, 18)
    v = v / (v.pow(2).mean(2, keepdim=True) + 1e-3).sqrt() * nw.double()
    v = v.reshape(tokens, width) * silu(gate[:, :width].double())
    assert rel(out[:, :33], v @ m.double().T) < tol


def test_dense_results_do_not_depend_on_the_rest_of_the_batch(dev):
    """Within a form, the bits of a row are the same whatever rows lie beside it."""
    ctx, torch, L = dev
    w = L.Weights(torch, torch.device("cuda"), "bfloat16")
    g = torch.Generator(device="cuda").manual_seed(1)
    m = w.matrix(torch.randn(192, 256, device="cuda", generator=g))
    x = torch.randn(300, 256, device="cuda", generator=g)
    got = {}
    for n in (65, 128, 300):
        rows = L.Rows(torch, torch.device("cuda"), n, 256, w, vector=False)
        out = torch.zeros(n, 192, device="cuda")
        rows.dense(ctx, m, input=L.IN_PLAIN, x=x, x_stride=256, out=out, out_stride=192)
        got[n] = out[:65].clone()
    assert torch.equal(got[65], got[128]) and torch.equal(got[65], got[300])


def test_dense_refusals(dev):
    ctx, torch, L = dev
    w = L.Weights(torch, torch.device("cuda"), "float32")
    lin = w.matrix(torch.randn(8, 16))
    rows = L.Rows(torch, torch.device("cuda"), 2, 64, w, vector=True)
    out = torch.zeros(2, 8, device="cuda")
    for bad, text in ((dict(k=63), "multiple of 8"), (dict(x_out=rows.x), "another buffer"), (dict(out=None), "no output"),
                      (dict(output=L.OUT_GLU), "blocks of 64"), (dict(input=L.IN_CONCAT), "second vector"),
                      (dict(input=L.IN_NORM, norm=1), "needs its weight"), (dict(w_dtype=7), "weight dtype")):
        with pytest.raises(KernelError, match=text):
            rows.dense(ctx, lin, **dict(dict(x=rows.x, x_stride=64, out=out, out_stride=8), **bad))


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("heads,dim,vdim,kv,window,splits", [
    (1, 16, 16, 64, 5, 1), (5, 20, 12, 100, 40, 3), (16, 32, 64, 128, 33, 4), (33, 48, 24, 256, 200, 16),
    (3, 128, 128, 512, 300, 7), (2, 64, 16, 576, 90, 2)])
def test_latent_attention_absorbed(dev, heads, dim, vdim, kv, window, splits, bf16):
    """Rows of several slots at positions around the window's and the ring's edges, one idle; one
    key of every row stands out by its score."""
    ctx, torch, L = dev
    g = torch.Generator(device="cuda").manual_seed(heads)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    dtype = torch.bfloat16 if bf16 else torch.float32
    ds, vs, ks = L.up_to(dim, 16), L.up_to(vdim, 16), L.padded(kv)
    ring, slots = window + 7, 3
    uk, uv = torch.zeros(heads, ds, ks, device="cuda"), torch.zeros(heads, vs, ks, device="cuda")
    uk[:, :dim, :kv], uv[:, :vdim, :kv] = rnd(heads, dim, kv) / kv ** 0.5, rnd(heads, vdim, kv) / kv ** 0.5
    uk, uv = uk.to(dtype), uv.to(dtype)
    last = window * 2 + 11
    cache = torch.full((slots, ring, ks), 1e4, device="cuda", dtype=dtype)   # stale rows would show
    lat = torch.zeros(slots, last + 1, ks, device="cuda")
    lat[:, :, :kv] = rnd(slots, last + 1, kv)
    lat = lat.to(dtype)
    positions = [0, 1, window - 2, window - 1, window, last, -5]
    positions = [min(max(p, 0), last) if p >= 0 else p for p in positions]
    out = torch.zeros(1, L.padded(heads * vdim), device="cuda")
    n = len(positions)
    rows_slot = [i % slots for i in range(n)]
    q = torch.zeros(n, heads, ds, device="cuda")
    for i, (p, s) in enumerate(zip(positions, rows_slot)):
        if p < 0:
            continue
        lo = max(0, p - window + 1)
        target = lo if i % 2 else max(lo, p - window // 2)
        k = torch.einsum("hdc,c->hd", uk.float()[:, :dim], lat[s, target].float())
        q[i, :, :dim] = rnd(heads, dim) + 6 * k / k.norm(dim=1, keepdim=True)
    scale = 1.7 / dim ** 0.5
    for i in range(n):    # one row per call: each needs the ring as it was at its position
        p, s = positions[i], rows_slot[i]
        cache.fill_(1e4)
        for j in range(max(0, p - window + 1), p + 1):
            cache[s, j % ring] = lat[s, j]
        pos = torch.tensor([p], dtype=torch.int32, device="cuda")
        slot = torch.tensor([s], dtype=torch.int32, device="cuda")
        scratch = torch.full((_lib.lib().qk_latent_scratch(1, heads, ks, splits) // 4,), float("nan"), device="cuda")
        c = L.LatentCall(tokens=1, positions=pos.data_ptr(), slots=slot.data_ptr(), heads=heads, dim=dim, dim_stride=ds,
                         vdim=vdim, vdim_stride=vs, kv_rank=kv, kv_stride=ks, window=window, ring=ring, n_slots=slots,
                         scale=scale, q=q[i].data_ptr(), q_dtype=QK_F32, q_stride=heads * ds,
                         w_dtype=QK_BF16 if bf16 else QK_F32, uk=uk.data_ptr(), uv=uv.data_ptr(), cache=cache.data_ptr(),
                         n_splits=splits, scratch=scratch.data_ptr(), out=out.data_ptr(), out_dtype=QK_F32,
                         out_stride=out.shape[1])
        check(_lib.lib().qk_latent_attention(ctx.handle, ctypes.byref(c)))
        ctx.synchronize()
        got = out[0, :heads * vdim].reshape(heads, vdim).double()
        if p < 0:
            assert not got.any()
            continue
        L_ = lat[s, max(0, p - window + 1):p + 1].double()
        kk = torch.einsum("hdc,jc->hjd", uk.double()[:, :dim], L_)
        vv = torch.einsum("hdc,jc->hjd", uv.double()[:, :vdim], L_)
        pr = torch.softmax(torch.einsum("hd,hjd->hj", q[i, :, :dim].double(), kk) * scale, dim=1)
        want = torch.einsum("hj,hjd->hd", pr, vv)
        assert float((got - want).abs().max() / want.abs().max()) < (1e-4 if bf16 else 1e-5), (i, p)


@pytest.mark.parametrize("dim,vdim,window,p0,tokens", [
    (16, 16, 1, 0, 20), (32, 64, 7, 3, 64), (48, 32, 64, 100, 65), (64, 128, 65, 10, 200), (128, 16, 130, 0, 300),
    (128, 128, 63, 500, 129), (160, 256, 40, 33, 70), (256, 96, 1000, 70, 100)])
def test_window_attention_expanded(dev, dim, vdim, window, p0, tokens):
    """Keys in tiles of 64: bands that start and end anywhere, the farthest visible key standing
    out for every third row."""
    ctx, torch, L = dev
    heads = 3
    g = torch.Generator(device="cuda").manual_seed(dim + window)
    key0 = max(0, p0 - window + 1)
    n = p0 + tokens - key0
    ds, vs = L.up_to(dim, 16), L.up_to(vdim, 16)
    kv = torch.randn(n, heads * (ds + vs), device="cuda", generator=g).bfloat16()
    k = kv[:, :heads * ds].reshape(n, heads, ds)
    v = kv[:, heads * ds:].reshape(n, heads, vs)
    q = torch.randn(tokens, heads, ds, device="cuda", generator=g) * 0.5
    for t in range(0, tokens, 3):
        far = max(0, p0 + t - window + 1) - key0
        q[t] += 0.6 * k[far].float()
    q = q.bfloat16()
    out = torch.zeros(tokens, L.padded(heads * vdim), device="cuda", dtype=torch.bfloat16)
    scale = 1.0 / dim ** 0.5
    P = ctypes.c_void_p
    check(_lib.lib().qk_window_attention(ctx.handle, P(q.data_ptr()), heads * ds, P(kv.data_ptr()), kv.shape[1], key0, n,
                                         p0, tokens, heads, ds, vdim, vs, window, scale, P(out.data_ptr()), out.shape[1]))
    ctx.synchronize()
    i = torch.arange(tokens, device="cuda")[:, None] + p0
    back = i - (torch.arange(n, device="cuda")[None] + key0)
    s = torch.einsum("thd,jhd->htj", q.double(), k.double()) * scale
    s = s.masked_fill(((back < 0) | (back >= window))[None], float("-inf"))
    want = torch.einsum("htj,jhd->thd", torch.softmax(s, -1), v.double()[:, :, :vdim])
    got = out[:, :heads * vdim].reshape(tokens, heads, vdim).double()
    assert float((got - want).abs().max() / want.abs().max()) < 1e-2
    assert not out[:, heads * vdim:].any()


def test_late_positions_keep_their_angles(dev):
    """Sinusoidal positions near 10^6: float32 angles would be wrong in the second digit."""
    ctx, torch, L = dev
    width, vocab = 11, 3
    table = torch.zeros(vocab, 64, device="cuda")
    pos = torch.tensor([0, 5, 999_983, -7], dtype=torch.int32, device="cuda")
    ids = torch.zeros(4, dtype=torch.int32, device="cuda")
    freq = torch.tensor([10000.0 ** (-2 * i / width) for i in range(6)], dtype=torch.float64, device="cuda")
    x = torch.full((4, 64), 9.0, device="cuda")
    P = ctypes.c_void_p
    check(_lib.lib().qk_embed_scaled(ctx.handle, P(table.data_ptr()), QK_F32, 64, P(ids.data_ptr()), P(pos.data_ptr()), 4,
                                     width, vocab, 2.0, P(freq.data_ptr()), P(x.data_ptr()), None, 64))
    ctx.synchronize()
    got = x.cpu().numpy()[:, :width]
    for r, p in enumerate((0, 5, 999_983)):
        angle = p * 10000.0 ** (-2 * (np.arange(width) // 2) / width)
        want = np.where(np.arange(width) % 2 == 0, np.sin(angle), np.cos(angle))
        np.testing.assert_allclose(got[r], want, atol=1e-6)
    assert not got[3].any()


def grouped_problem(torch, heads, kv_heads, dim, vdim, s_max, dtype, seed, bias_len=37):
    """A cache of three slots, queries of which every third has one key that stands out."""
    from quantibbler_b200 import layers as L
    g = torch.Generator(device="cuda").manual_seed(seed)
    ds, vs = L.up_to(dim, 16), L.up_to(vdim, 16)
    k, v = torch.zeros(3, kv_heads, s_max, ds, device="cuda"), torch.zeros(3, kv_heads, s_max, vs, device="cuda")
    k[..., :dim] = torch.randn(3, kv_heads, s_max, dim, device="cuda", generator=g)
    v[..., :vdim] = torch.randn(3, kv_heads, s_max, vdim, device="cuda", generator=g)
    bias = torch.randn(heads, bias_len, device="cuda", generator=g)
    return g, ds, vs, k.to(dtype), v.to(dtype), bias


def grouped_reference(torch, q, k, v, bias, scale, coef, every, p):
    """One row at position p: q [heads, dim], k and v [kv_heads, p + 1, ..], float64."""
    H, G = q.shape[0], k.shape[0]
    q, k, v = q.double(), k.double().repeat_interleave(H // G, 0), v.double().repeat_interleave(H // G, 0)
    factor = scale * (1 + coef * np.log(np.floor((p + 1) / every) + 1)) if every else scale
    s = torch.einsum("hd,hjd->hj", q, k) * factor
    back = (p - torch.arange(p + 1, device="cuda")).clamp(max=bias.shape[1] - 1)
    return torch.einsum("hj,hjd->hd", torch.softmax(s + bias.double()[:, back], 1), v)


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("append", [False, True])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,splits", [
    (1, 1, 16, 16, 1), (6, 2, 20, 44, 3), (8, 1, 64, 64, 4), (24, 2, 40, 24, 2), (4, 2, 128, 96, 7), (5, 5, 100, 128, 5),
    (3, 1, 256, 250, 3), (2, 2, 300, 270, 4)])
def test_grouped_attention_of_rows(dev, heads, kv_heads, dim, vdim, splits, append, bf16):
    """Rows of three slots at positions around the edges of key tiles and splits, one idle, one
    outside the cache; nothing behind a row's position is read.  With ``append`` the newest key and
    value come from the projections and end up in the cache, without it every row is cached."""
    ctx, torch, L = dev
    dtype, tag = (torch.bfloat16, QK_BF16) if bf16 else (torch.float32, QK_F32)
    s_max = 700
    g, ds, vs, ck, cv, bias = grouped_problem(torch, heads, kv_heads, dim, vdim, s_max, dtype, heads + dim)
    positions = [0, 1, 14, 15, 16, 17, 31, 32, 63, 64, 65, 127, 128, 129, 191, 192, 300, 511, 512, 699, -3, 36, 37, 38]
    rows = len(positions)
    stride = L.up_to(heads * ds + kv_heads * (ds + vs), 8) + 8
    proj = torch.zeros(rows, stride, device="cuda")
    q = torch.zeros(rows, heads, ds, device="cuda")
    q[..., :dim] = torch.randn(rows, heads, dim, device="cuda", generator=g) * 0.3
    nk, nv = torch.zeros(rows, kv_heads, ds, device="cuda"), torch.zeros(rows, kv_heads, vs, device="cuda")
    nk[..., :dim] = torch.randn(rows, kv_heads, dim, device="cuda", generator=g)
    nv[..., :vdim] = torch.randn(rows, kv_heads, vdim, device="cuda", generator=g)
    scale, coef, every = 1.3 / dim ** 0.5, 0.4, 60.0
    out = torch.zeros(rows, heads * vs + 4, device="cuda")
    for r in range(0, rows, 3):   # (position 0 or the middle stands out)
        p, s = positions[r], r % 3
        if p > 0:
            far = ck[s, :, 0 if r % 2 else p // 2].float().repeat_interleave(heads // kv_heads, 0)
            q[r] += 2.5 * far / far.norm(dim=1, keepdim=True) * dim ** 0.25
    proj[:, :heads * ds] = q.reshape(rows, -1)
    proj[:, heads * ds:(heads + kv_heads) * ds] = nk.reshape(rows, -1)
    proj[:, (heads + kv_heads) * ds:(heads + kv_heads) * ds + kv_heads * vs] = nv.reshape(rows, -1)
    for r in range(rows):       # one row per call: each needs the cache as it was at its position
        p, s = positions[r], r % 3
        k, v = ck.clone(), cv.clone()
        n = max(p, 0) + (0 if append else 1)
        k[:, :, n:], v[:, :, n:] = float("nan"), float("nan")
        pos = torch.tensor([p], dtype=torch.int32, device="cuda")
        slot = torch.tensor([s], dtype=torch.int32, device="cuda")
        scratch = torch.zeros(_lib.lib().qk_grouped_scratch(1, heads, kv_heads, vs, splits) // 4, device="cuda")
        out.fill_(7.0)
        c = L.GroupedCall(tokens=1, positions=pos.data_ptr(), slots=slot.data_ptr(), heads=heads, kv_heads=kv_heads,
                          dim_stride=ds, vdim_stride=vs, s_max=s_max, n_slots=3, scale=scale, temp_coef=coef,
                          temp_every=every, bias=bias.data_ptr(), bias_len=bias.shape[1], proj=proj[r].data_ptr(),
                          proj_dtype=QK_F32, proj_stride=stride, cache_dtype=tag, cache_k=k.data_ptr(),
                          cache_v=v.data_ptr(), n_splits=splits, scratch=scratch.data_ptr(), out=out[r].data_ptr(),
                          out_dtype=QK_F32, out_stride=heads * vs, append=int(append))
        check(_lib.lib().qk_grouped_attention(ctx.handle, ctypes.byref(c)))
        ctx.synchronize()
        assert not scratch[-heads:].view(torch.int32).any(), "the counters are zero again"
        if p < 0:
            assert (out[r] == 7.0).all()
            continue
        if append:
            assert torch.equal(k[s, :, p], nk[r].to(dtype)) and torch.equal(v[s, :, p], nv[r].to(dtype))
            k[s, :, p], v[s, :, p] = nk[r].to(dtype), nv[r].to(dtype)
        want = grouped_reference(torch, q[r], k[s, :, :p + 1], v[s, :, :p + 1], bias, scale, coef, every, p)
        got = out[r, :heads * vs].reshape(heads, vs).double()
        assert float((got - want).abs().max() / want.abs().max()) < (1e-4 if bf16 else 2e-5), (r, p)


def test_grouped_attention_of_a_batch(dev):
    """All rows of a step at once equal each alone, bit for bit; a row outside the cache is reported."""
    ctx, torch, L = dev
    heads, kv_heads, dim, s_max, slots = 8, 2, 64, 256, 9
    g = torch.Generator(device="cuda").manual_seed(3)
    k = torch.randn(slots, kv_heads, s_max, dim, device="cuda", generator=g).bfloat16()
    v = torch.randn(slots, kv_heads, s_max, dim, device="cuda", generator=g).bfloat16()
    stride = (heads + 2 * kv_heads) * dim
    proj = torch.randn(slots, stride, device="cuda", generator=g)
    pos = torch.tensor([0, 255, 17, -1, 128, 63, 200, 1, 90], dtype=torch.int32, device="cuda")
    slot = torch.tensor([4, 2, 0, 1, 3, 8, 7, 6, 5], dtype=torch.int32, device="cuda")

    def ran(first, n, positions=pos):
        kk, vv, out = k.clone(), v.clone(), torch.zeros(n, heads * dim, device="cuda")
        scratch = torch.zeros(_lib.lib().qk_grouped_scratch(n, heads, kv_heads, dim, 3) // 4, device="cuda")
        c = L.GroupedCall(tokens=n, positions=positions[first:].data_ptr(), slots=slot[first:].data_ptr(), heads=heads,
                          kv_heads=kv_heads, dim_stride=dim, vdim_stride=dim, s_max=s_max, n_slots=slots, scale=0.125,
                          proj=proj[first:].data_ptr(), proj_dtype=QK_F32, proj_stride=stride, cache_dtype=QK_BF16,
                          cache_k=kk.data_ptr(), cache_v=vv.data_ptr(), n_splits=3, scratch=scratch.data_ptr(),
                          out=out.data_ptr(), out_dtype=QK_F32, out_stride=heads * dim, append=1)
        check(_lib.lib().qk_grouped_attention(ctx.handle, ctypes.byref(c)))
        torch.cuda.synchronize()
        return out, kk, vv

    whole = ran(0, slots)
    ctx.synchronize()
    for r in range(slots):
        alone = ran(r, 1)
        assert torch.equal(alone[0][0], whole[0][r])
        assert torch.equal(alone[1][slot[r]], whole[1][slot[r]]) and torch.equal(alone[2][slot[r]], whole[2][slot[r]])
    ctx.synchronize()
    late = pos.clone()
    late[2] = s_max
    out, kk, _ = ran(0, slots, late)
    assert not out[2].any() and torch.equal(kk[slot[2]], k[slot[2]])
    with pytest.raises(Exception, match="cache"):
        ctx.synchronize()


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,p0,tokens", [
    (1, 1, 16, 16, 0, 20), (4, 2, 32, 64, 3, 64), (6, 3, 48, 20, 100, 65), (3, 1, 64, 128, 10, 200), (2, 2, 128, 16, 0, 300),
    (4, 1, 128, 128, 500, 129), (3, 1, 80, 112, 0, 300), (6, 2, 96, 64, 130, 260), (1, 1, 112, 80, 1000, 17),
    (9, 3, 64, 64, 7, 385), (4, 2, 128, 128, 3000, 150), (2, 1, 160, 256, 33, 70), (2, 2, 250, 96, 70, 100), (8, 2, 128, 128, 0, 513)])
def test_grouped_attention_of_a_portion(dev, heads, kv_heads, dim, vdim, p0, tokens):
    """Portions that start and end anywhere between key tiles, with the append in front; cache rows
    behind the portion hold no numbers."""
    ctx, torch, L = dev
    s_max = p0 + tokens + 5
    g, ds, vs, k, v, bias = grouped_problem(torch, heads, kv_heads, dim, vdim, s_max, torch.bfloat16, dim + p0)
    stride = heads * ds + kv_heads * (ds + vs)
    q = torch.zeros(tokens, heads, ds, device="cuda")
    q[..., :dim] = torch.randn(tokens, heads, dim, device="cuda", generator=g) * 0.5
    for t in range(0, tokens, 3):
        q[t] += 1.5 * k[1, :, max(0, p0 + t - 90)].float().repeat_interleave(heads // kv_heads, 0) / dim ** 0.25
    proj = torch.cat([q.reshape(tokens, -1), k[1, :, p0:p0 + tokens].transpose(0, 1).reshape(tokens, -1).float(),
                      v[1, :, p0:p0 + tokens].transpose(0, 1).reshape(tokens, -1).float()], 1).bfloat16()
    assert proj.shape[1] == stride
    full_k, full_v = k.clone(), v.clone()
    k[:, :, p0:], v[:, :, p0:] = float("nan"), float("nan")
    out = torch.zeros(tokens, heads * vs, device="cuda", dtype=torch.bfloat16)
    pos = torch.arange(p0, p0 + tokens, dtype=torch.int32, device="cuda")
    slot = torch.ones(tokens, dtype=torch.int32, device="cuda")
    scale, coef, every = 1.0 / dim ** 0.5, 0.35, 48.0
    c = L.GroupedCall(tokens=tokens, positions=pos.data_ptr(), slots=slot.data_ptr(), heads=heads, kv_heads=kv_heads,
                      dim_stride=ds, vdim_stride=vs, s_max=s_max, n_slots=3, scale=scale, temp_coef=coef, temp_every=every,
                      bias=bias.data_ptr(), bias_len=bias.shape[1], proj=proj.data_ptr(), proj_dtype=QK_BF16,
                      proj_stride=stride, cache_dtype=QK_BF16, cache_k=k.data_ptr(), cache_v=v.data_ptr(),
                      out=out.data_ptr(), out_dtype=QK_BF16, out_stride=heads * vs, slot=1, first_position=p0)
    check(_lib.lib().qk_grouped_append(ctx.handle, ctypes.byref(c)))
    check(_lib.lib().qk_grouped_portion(ctx.handle, ctypes.byref(c)))
    ctx.synchronize()
    assert torch.equal(k[1, :, :p0 + tokens], full_k[1, :, :p0 + tokens])
    assert torch.equal(v[1, :, :p0 + tokens], full_v[1, :, :p0 + tokens])
    assert k[1, :, p0 + tokens:].isnan().all() and k[0, :, p0:].isnan().all()
    qb = proj[:, :heads * ds].reshape(tokens, heads, ds)
    for t in sorted({0, 1, 15, 16, 63, 64, 65, tokens // 2, tokens - 2, tokens - 1} & set(range(tokens))):
        p = p0 + t
        want = grouped_reference(torch, qb[t], k[1, :, :p + 1], v[1, :, :p + 1], bias, scale, coef, every, p)
        got = out[t].reshape(heads, vs).double()
        assert float((got - want).abs().max() / want.abs().max()) < 1.2e-2, t


@pytest.mark.parametrize("serving,tol", [("float32", 4e-6), ("bfloat16", 1e-2)])
@pytest.mark.parametrize("tokens", [1, 2, 4, 5, 16, 70, 128, 129, 400])
@pytest.mark.parametrize("experts,top,width,ff", [(1, 1, 72, 40), (5, 2, 200, 33), (3, 3, 64, 130), (40, 3, 136, 64)])
def test_experts(dev, tokens, experts, top, width, ff, serving, tol):
    """Every form of a linear with experts: choices sorted by expert, rows per choice, and the next
    norm's pending sum, against one product per token and choice."""
    ctx, torch, L = dev
    g = torch.Generator(device="cuda").manual_seed(tokens + experts)
    rnd = lambda *s: torch.randn(*s, device="cuda", generator=g)
    bf = lambda t: t.bfloat16().float()
    w = L.Weights(torch, torch.device("cuda"), serving)
    vocab, eps = 50, 1e-3
    table = torch.stack([torch.randperm(experts)[:top] for _ in range(vocab)]).to(torch.int32)
    if experts > 4:   # (two experts that nobody has, one that most have)
        table[table == 1] = experts - 1
        table = torch.where((table == experts - 1).sum(1, keepdim=True) > 1, torch.arange(2, 2 + top, dtype=torch.int32), table)
    t = {"table": table}
    for e in range(experts):
        t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"] = (
            bf(rnd(ff, width) / width ** 0.5), bf(rnd(ff, width) / width ** 0.5), bf(rnd(width, ff) / ff ** 0.5))
    mlp = L.TableExperts(w, t, experts=experts, activation="silu")
    stride = L.padded(width)
    rows = L.Rows(torch, torch.device("cuda"), tokens, stride, w, vector=tokens <= 4)
    x = rnd(tokens, width) * 2
    rows.x[:, :width] = x
    ids = torch.randint(0, vocab, (tokens,), device="cuda", generator=g)
    rows.ids.copy_(ids)
    nw, pw = rnd(width) * 0.2 + 1, rnd(width) * 0.2 + 1
    rows.route(ctx, [mlp.table], width, vocab)
    mlp.forward(ctx, rows, L.NORM_RMS, nw, eps, L.Join(norm=pw, eps=eps))
    # what is pending, added by a linear that copies its input
    eye = w.matrix(torch.eye(width, device="cuda"))
    out = torch.zeros(tokens, L.up_to(width, 8), device="cuda")
    rows.dense(ctx, eye, **rows.stream_fields(L.NORM_NONE, None, 0.0), out=out, out_stride=out.shape[1])
    rows.settle()
    ctx.synchronize()
    xd = x.double()
    h = xd / (xd.pow(2).mean(1, keepdim=True) + eps).sqrt() * nw.double()
    y = torch.zeros_like(h)
    for i in range(tokens):
        for e in table[ids[i].item()].tolist():
            a = silu(t[f"e{e}.gate"].double() @ h[i]) * (t[f"e{e}.up"].double() @ h[i])
            y[i] += t[f"e{e}.down"].double() @ a / top
    want = xd + y / (y.pow(2).mean(1, keepdim=True) + eps).sqrt() * pw.double()
    assert rel(rows.x[:, :width], want) < tol * 3   # (rms norms of sums of few terms)
    if tokens > 4:
        r = rows.routes[id(mlp.table)]
        chosen = table.cuda()[ids.long()].flatten()
        assert sorted(r.places.flatten().tolist()) == list(range(tokens * top))
        assert torch.equal(chosen[r.places.flatten().argsort()], chosen.sort().values)
        counts = torch.bincount(chosen.long(), minlength=experts)
        assert r.offsets.tolist() == [0] + counts.cumsum(0).tolist()
        covered = []
        for n in range(int(r.tiles[0])):
            e, first, end, tile0, tiles = r.tiles[1 + 5 * n:6 + 5 * n].tolist()
            assert tile0 <= n < tile0 + tiles and all(int(r.tiles[1 + 5 * i]) == e for i in range(tile0, tile0 + tiles))
            assert r.offsets[e] <= first < end <= r.offsets[e + 1] and end - first <= 128
            covered += range(first, end)
        assert covered == list(range(tokens * top))


@pytest.mark.parametrize("tokens", [1, 5, 9, 70])
@pytest.mark.parametrize("bf16", [False, True])
def test_soft_capped_head(dev, tokens, bf16):
    ctx, torch, L = dev
    g = torch.Generator(device="cuda").manual_seed(tokens)
    h = torch.randn(tokens, 128, device="cuda", generator=g)
    m = torch.randn(301, 128, device="cuda", generator=g).to(torch.bfloat16 if bf16 else torch.float32)
    P = ctypes.c_void_p
    for cap in (0.0, 4.0):
        out = torch.zeros(tokens, 301, device="cuda")
        check(_lib.lib().qk_lm_head_capped(ctx.handle, P(h.data_ptr()), P(m.data_ptr()), QK_BF16 if bf16 else QK_F32, tokens,
                                           301, 128, 301, cap, P(out.data_ptr())))
        ctx.synchronize()
        want = h.double() @ m.double().T
        if cap:
            want = cap * torch.tanh(want / cap)
        assert rel(out, want) < 1e-4
