// Row kernels of the layered decoders that are not attention or a linear: the scaled embedding
// with sinusoidal positions, and the gated delta rule.
//
// The delta rule per head, with a state S [dim][vdim] in float32:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// Column j of S meets only v_j, so the columns are independent recurrences: eight lanes hold one
// column in registers, a warp four columns, and a block walks its sixteen columns of one head
// through all tokens of a sequence portion while the next tokens' k, q and v arrive by cp.async.
// Both dot products of a token read the OLD state, so that only one reduction lies between two
// tokens: S^T k after the decay is g (S_old^T k), and o = g (S_old^T q) + (k . q) u.
#include "qk_dense_dev.cuh"

namespace {

// ------------------------------------------------------------------ embedding
template <typename W>
__global__ void __launch_bounds__(256)
embed_scaled_kernel(const W *__restrict__ table, uint32_t table_stride, const int32_t *__restrict__ ids,
                    const int32_t *__restrict__ positions, uint32_t width, uint32_t vocab, float scale,
                    const double *__restrict__ inv_freq, float *__restrict__ x, float *__restrict__ x_copy,
                    uint32_t x_stride) {
    qk::pdl_launch();
    qk::pdl_wait();
    const uint32_t t = blockIdx.x;
    const int pos = positions[t];
    const uint32_t id = (uint32_t)min(max(ids[t], 0), (int)vocab - 1);
    for (uint32_t i = blockIdx.y * blockDim.x + threadIdx.x; i < width; i += gridDim.y * blockDim.x) {
        float v = 0.f;
        if (pos >= 0) {
            v = load_as_float(table, (size_t)id * table_stride + i) * scale;
            if (inv_freq) {
                // the angle to float64 accuracy, brought to one turn before it is rounded: a
                // float32 angle of a late position would lose its last digits
                const double a = (double)pos * inv_freq[i / 2];
                const float r = (float)(a - 6.283185307179586476925 * rint(a * 0.15915494309189533577));
                v += i % 2 ? cosf(r) : sinf(r);
            }
        }
        x[(size_t)t * x_stride + i] = v;
        if (x_copy) x_copy[(size_t)t * x_stride + i] = v;
    }
}

// ------------------------------------------------------------------ delta rule: inputs of the recurrence
struct DeltaArgs {
    const int32_t *positions, *slots, *seg_first, *seg_len, *seg_row;
    const float *proj, *conv_q, *conv_k, *conv_v, *a_log, *dt_bias;
    float *conv_state, *state, *qkv, *gates, *out;
    uint32_t heads, kv_heads, dim, vdim, taps, channels, proj_stride, beta_offset, decay_offset, out_stride;
    float unit_eps;
};

// Convolution and silu of channel c (of q | k | v, as the projection lays them out) at row t.
__device__ __forceinline__ float conv_silu(const DeltaArgs &a, uint32_t t, int pos, uint32_t in_seg, uint32_t slot,
                                           const float *__restrict__ taps, uint32_t c) {
    float y = 0.f;
    for (uint32_t back = 0; back < a.taps; ++back) {
        float v = 0.f;
        if (in_seg >= back) v = a.proj[(size_t)(t - back) * a.proj_stride + c];
        else if (pos >= (int)back)
            v = a.conv_state[((size_t)slot * a.taps + (uint32_t)(pos - (int)back) % a.taps) * a.channels + c];
        y = fmaf(taps[a.taps - 1 - back], v, y);
    }
    return silu_f(y);
}

constexpr int kPrepThreads = 256, kMaxLane = 16;  // dim up to 32 * kMaxLane
__global__ void __launch_bounds__(kPrepThreads)
delta_inputs_kernel(DeltaArgs a) {
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ float kq[];  // [kv heads of this block]
    const uint32_t t = blockIdx.x, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int pos = a.positions[t];
    if (pos < 0) return;
    const uint32_t in_seg = (uint32_t)a.seg_row[t], slot = (uint32_t)a.slots[t];
    const uint32_t n_local = (a.kv_heads - blockIdx.y + gridDim.y - 1) / gridDim.y;  // kv heads y, y + parts, ..
    const uint32_t ratio = a.heads / a.kv_heads, key0 = a.kv_heads * a.dim, val0 = 2 * key0;
    float *row = a.qkv + (size_t)t * a.channels;
    for (uint32_t i = warp; i < n_local; i += kPrepThreads / 32) {
        const uint32_t c0 = (blockIdx.y + i * gridDim.y) * a.dim;
        float q[kMaxLane], k[kMaxLane], sq = 0.f, sk = 0.f;
#pragma unroll
        for (int j = 0; j < kMaxLane; ++j) {
            const uint32_t d = lane + 32 * j;
            q[j] = k[j] = 0.f;
            if (d < a.dim) {
                q[j] = conv_silu(a, t, pos, in_seg, slot, a.conv_q + (size_t)(c0 + d) * a.taps, c0 + d);
                k[j] = conv_silu(a, t, pos, in_seg, slot, a.conv_k + (size_t)(c0 + d) * a.taps, key0 + c0 + d);
            }
            sq += q[j] * q[j];
            sk += k[j] * k[j];
        }
        for (int off = 16; off > 0; off >>= 1) {
            sq += __shfl_xor_sync(0xffffffffu, sq, off);
            sk += __shfl_xor_sync(0xffffffffu, sk, off);
        }
        const float iq = 1.0f / sqrtf(sq + a.unit_eps) * (1.0f / sqrtf((float)a.dim));
        const float ik = 1.0f / sqrtf(sk + a.unit_eps);
        float dot = 0.f;
#pragma unroll
        for (int j = 0; j < kMaxLane; ++j) {
            const uint32_t d = lane + 32 * j;
            const float qv = q[j] * iq, kv = k[j] * ik;
            if (d < a.dim) {
                row[c0 + d] = qv;
                row[key0 + c0 + d] = kv;
            }
            dot += qv * kv;
        }
        for (int off = 16; off > 0; off >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, off);
        if (lane == 0) kq[i] = dot;
    }
    // values: the channels of the heads that belong to these kv heads
    const uint32_t per = ratio * a.vdim;
    for (uint32_t i = threadIdx.x; i < n_local * per; i += kPrepThreads) {
        const uint32_t c = (blockIdx.y + i / per * gridDim.y) * per + i % per;
        row[val0 + c] = conv_silu(a, t, pos, in_seg, slot, a.conv_v + (size_t)c * a.taps, val0 + c);
    }
    __syncthreads();
    const float *pr = a.proj + (size_t)t * a.proj_stride;
    for (uint32_t i = threadIdx.x; i < n_local * ratio; i += kPrepThreads) {
        const uint32_t h = (blockIdx.y + i / ratio * gridDim.y) * ratio + i % ratio;
        const float z = pr[a.decay_offset + h] + a.dt_bias[h];
        const float sp = z > 20.f ? z : log1pf(expf(z));
        float *g = a.gates + ((size_t)t * a.heads + h) * 4;
        g[0] = sigmoid_f(pr[a.beta_offset + h]);
        g[1] = expf(-expf(a.a_log[h]) * sp);
        g[2] = kq[i / ratio];
    }
}

// ------------------------------------------------------------------ delta rule: the recurrence
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float &a, float &b) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ void copy_async4(float *smem, const float *gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem)
                 : "memory");
}
__device__ __forceinline__ void copy_async16(float *smem, const float *gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem)
                 : "memory");
}

constexpr int kScanThreads = 128, kScanCols = kScanThreads / 8;  // columns per block

// kPer: state entries per lane (dim <= 8 * kPer).  Lane l of a column's eight holds entries
// 32 i + 4 l .. + 3.
template <int kPer>
__global__ void __launch_bounds__(kScanThreads)
delta_scan_kernel(DeltaArgs a, int vec) {
    constexpr int kDim = 8 * kPer;
    constexpr int kScanTokens = kPer > 32 ? 4 : 8;  // tokens per staged chunk
    qk::pdl_launch();
    qk::pdl_wait();
    __shared__ __align__(16) float ks[2][kScanTokens][kDim], qs[2][kScanTokens][kDim];
    __shared__ float vs[2][kScanTokens][kScanCols];
    __shared__ __align__(16) float gs[2][kScanTokens][4];
    const uint32_t h = blockIdx.y, seg = blockIdx.z;
    const uint32_t first = (uint32_t)a.seg_first[seg], len = (uint32_t)a.seg_len[seg];
    const int pos0 = len ? a.positions[first] : -1;
    if (pos0 < 0) return;
    const uint32_t slot = (uint32_t)a.slots[first];
    const uint32_t lane8 = threadIdx.x % 8, col_in = threadIdx.x / 8, col0 = blockIdx.x * kScanCols;
    const uint32_t col = col0 + col_in;
    const bool live = col < a.vdim;
    const uint32_t kvh = h / (a.heads / a.kv_heads), key0 = a.kv_heads * a.dim;
    float *st = a.state + (((size_t)slot * a.heads + h) * a.vdim + min(col, a.vdim - 1)) * a.dim;

    // entries past dim stay zero in both buffers
    if (a.dim < (uint32_t)kDim) {
        for (uint32_t i = threadIdx.x; i < 2 * kScanTokens * kDim; i += kScanThreads) {
            (&ks[0][0][0])[i] = 0.f;
            (&qs[0][0][0])[i] = 0.f;
        }
        __syncthreads();
    }
    auto stage = [&](uint32_t t0, uint32_t buf) {
        const uint32_t n = min((uint32_t)kScanTokens, len - t0);
        const float *base = a.qkv + (size_t)(first + t0) * a.channels;
        if (vec) {
            const uint32_t per = a.dim / 4;
            for (uint32_t i = threadIdx.x; i < n * per; i += kScanThreads) {
                const uint32_t t = i / per, d = (i % per) * 4;
                const float *src = base + (size_t)t * a.channels + kvh * a.dim + d;
                copy_async16(&qs[buf][t][d], src);
                copy_async16(&ks[buf][t][d], src + key0);
            }
        } else {
            for (uint32_t i = threadIdx.x; i < n * a.dim; i += kScanThreads) {
                const uint32_t t = i / a.dim, d = i % a.dim;
                const float *src = base + (size_t)t * a.channels + kvh * a.dim + d;
                copy_async4(&qs[buf][t][d], src);
                copy_async4(&ks[buf][t][d], src + key0);
            }
        }
        for (uint32_t i = threadIdx.x; i < n * kScanCols; i += kScanThreads) {
            const uint32_t t = i / kScanCols, j = i % kScanCols;
            if (col0 + j < a.vdim)
                copy_async4(&vs[buf][t][j], base + (size_t)t * a.channels + 2 * key0 + h * a.vdim + col0 + j);
        }
        if (threadIdx.x < n)
            copy_async16(&gs[buf][threadIdx.x][0], a.gates + ((size_t)(first + t0 + threadIdx.x) * a.heads + h) * 4);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    f32x2 s[kPer / 2];
#pragma unroll
    for (int i = 0; i < kPer / 4; ++i) {
        const uint32_t d = 32 * i + 4 * lane8;
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (pos0 != 0 && live) {
            if (vec && d < a.dim) {
                const float4 f = *reinterpret_cast<const float4 *>(st + d);
                v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < a.dim) v[e] = st[d + e];
            }
        }
        s[2 * i] = pack2(v[0], v[1]);
        s[2 * i + 1] = pack2(v[2], v[3]);
    }
    for (uint32_t t0 = 0, buf = 0; t0 < len; t0 += kScanTokens, buf ^= 1) {
        if (t0 + kScanTokens < len) {
            stage(t0 + kScanTokens, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const uint32_t n = min((uint32_t)kScanTokens, len - t0);
        for (uint32_t t = 0; t < n; ++t) {
            const float4 gt = *reinterpret_cast<const float4 *>(&gs[buf][t][0]);
            const float v = vs[buf][t][col_in];
            f32x2 k[kPer / 2];
            f32x2 dk0 = 0, dk1 = 0, dq0 = 0, dq1 = 0;  // (two zero floats)
#pragma unroll
            for (int i = 0; i < kPer / 4; ++i) {
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2 *>(&ks[buf][t][32 * i + 4 * lane8]);
                const ulonglong2 qq = *reinterpret_cast<const ulonglong2 *>(&qs[buf][t][32 * i + 4 * lane8]);
                k[2 * i] = kk.x;
                k[2 * i + 1] = kk.y;
                dk0 = fma2(s[2 * i], kk.x, dk0);
                dk1 = fma2(s[2 * i + 1], kk.y, dk1);
                dq0 = fma2(s[2 * i], qq.x, dq0);
                dq1 = fma2(s[2 * i + 1], qq.y, dq1);
            }
            float a0, a1, a2, a3;
            unpack2(dk0, a0, a1);
            unpack2(dk1, a2, a3);
            float dk = (a0 + a1) + (a2 + a3);
            unpack2(dq0, a0, a1);
            unpack2(dq1, a2, a3);
            float dq = (a0 + a1) + (a2 + a3);
#pragma unroll
            for (int off = 1; off < 8; off <<= 1) {
                dk += __shfl_xor_sync(0xffffffffu, dk, off);
                dq += __shfl_xor_sync(0xffffffffu, dq, off);
            }
            const float u = gt.x * (v - gt.y * dk);
            const f32x2 g2 = pack2(gt.y, gt.y), u2 = pack2(u, u);
#pragma unroll
            for (int i = 0; i < kPer / 2; ++i) s[i] = fma2(k[i], u2, mul2(g2, s[i]));
            if (lane8 == 0 && live)
                a.out[(size_t)(first + t0 + t) * a.out_stride + h * a.vdim + col] = gt.y * dq + gt.z * u;
        }
        __syncthreads();
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < kPer / 4; ++i) {
            const uint32_t d = 32 * i + 4 * lane8;
            float v[4];
            unpack2(s[2 * i], v[0], v[1]);
            unpack2(s[2 * i + 1], v[2], v[3]);
            if (vec && d < a.dim) {
                *reinterpret_cast<float4 *>(st + d) = make_float4(v[0], v[1], v[2], v[3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (d + e < a.dim) st[d + e] = v[e];
            }
        }
    }
    // the convolution's last taps - 1 inputs (their readers, the inputs kernel, have finished)
    const uint32_t keep = min(a.taps - 1, len);
    const uint32_t n_blocks = gridDim.x * gridDim.y, block = blockIdx.y * gridDim.x + blockIdx.x;
    for (uint32_t i = block * kScanThreads + threadIdx.x; i < keep * a.channels; i += n_blocks * kScanThreads) {
        const uint32_t back = i / a.channels, c = i % a.channels, r = len - 1 - back;
        a.conv_state[((size_t)slot * a.taps + (uint32_t)(pos0 + (int)r) % a.taps) * a.channels + c] =
            a.proj[(size_t)(first + r) * a.proj_stride + c];
    }
}

qk_status enter(qk_ctx *ctx, qk_ctx **c) {
    qk_status st = qk::resolve_ctx(ctx, c);
    if (st != QK_OK) return st;
    QK_CUDA(cudaSetDevice((*c)->device));
    return QK_OK;
}

}  // namespace

extern "C" {

qk_status qk_embed_scaled(qk_ctx *ctx, const void *table, int32_t table_dtype, size_t table_stride,
                          const int32_t *ids, const int32_t *positions, size_t tokens, size_t width, size_t vocab,
                          float scale, const double *inv_freq, float *x, float *x_copy, size_t x_stride) {
    qk_ctx *c;
    qk_status st = enter(ctx, &c);
    if (st != QK_OK) return st;
    if (!table || !ids || !positions || !x || vocab == 0 || width > table_stride || width > x_stride)
        return qk::fail(QK_ERR_VALUE, "qk_embed_scaled: bad arguments");
    if (tokens == 0) return QK_OK;
    const dim3 grid((unsigned)tokens, tokens < 64 ? (unsigned)qk::ceil_div(width, 256) : 1);
    if (table_dtype == QK_F32)
        (void)qk::launch_pdl(c->pdl, embed_scaled_kernel<float>, grid, dim3(256), 0, c->stream, (const float *)table,
                             (uint32_t)table_stride, ids, positions, (uint32_t)width, (uint32_t)vocab, scale, inv_freq,
                             x, x_copy, (uint32_t)x_stride);
    else if (table_dtype == QK_BF16)
        (void)qk::launch_pdl(c->pdl, embed_scaled_kernel<uint16_t>, grid, dim3(256), 0, c->stream,
                             (const uint16_t *)table, (uint32_t)table_stride, ids, positions, (uint32_t)width,
                             (uint32_t)vocab, scale, inv_freq, x, x_copy, (uint32_t)x_stride);
    else
        return qk::fail(QK_ERR_VALUE, "embedding dtype must be float32 or bfloat16, got tag %d", table_dtype);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
}

qk_status qk_delta(qk_ctx *ctx, const qk_delta_call *d) {
    qk_ctx *c;
    qk_status st = enter(ctx, &c);
    if (st != QK_OK) return st;
    if (!d || !d->proj || !d->state || !d->conv_state || !d->qkv || !d->gates || !d->out)
        return qk::fail(QK_ERR_VALUE, "qk_delta: null argument");
    if (d->kv_heads == 0 || d->heads % d->kv_heads || d->dim == 0 || d->vdim == 0 || d->taps == 0)
        return qk::fail(QK_ERR_VALUE, "qk_delta: %zu heads over %zu key heads, dim %zu, vdim %zu, %zu taps", d->heads,
                        d->kv_heads, d->dim, d->vdim, d->taps);
    if (d->dim > 512) return qk::fail(QK_ERR_VALUE, "qk_delta: dim above 512 is not supported, got %zu", d->dim);
    if (d->tokens == 0) return QK_OK;
    DeltaArgs a{};
    a.positions = d->positions;
    a.slots = d->slots;
    a.seg_first = d->seg_first;
    a.seg_len = d->seg_len;
    a.seg_row = d->seg_row;
    a.proj = d->proj;
    a.conv_q = d->conv_q;
    a.conv_k = d->conv_k;
    a.conv_v = d->conv_v;
    a.a_log = d->a_log;
    a.dt_bias = d->dt_bias;
    a.conv_state = d->conv_state;
    a.state = d->state;
    a.qkv = d->qkv;
    a.gates = d->gates;
    a.out = d->out;
    a.heads = (uint32_t)d->heads;
    a.kv_heads = (uint32_t)d->kv_heads;
    a.dim = (uint32_t)d->dim;
    a.vdim = (uint32_t)d->vdim;
    a.taps = (uint32_t)d->taps;
    a.channels = (uint32_t)(2 * d->kv_heads * d->dim + d->heads * d->vdim);
    a.proj_stride = (uint32_t)d->proj_stride;
    a.beta_offset = (uint32_t)d->beta_offset;
    a.decay_offset = (uint32_t)d->decay_offset;
    a.out_stride = (uint32_t)d->out_stride;
    a.unit_eps = d->unit_eps;
    // few rows: a block per key head and row; many rows: a block for a few key heads
    const size_t parts = d->tokens <= 64 ? d->kv_heads : qk::ceil_div(d->kv_heads, 8);
    (void)qk::launch_pdl(c->pdl, delta_inputs_kernel, dim3((unsigned)d->tokens, (unsigned)parts), dim3(kPrepThreads),
                         d->kv_heads * sizeof(float), c->stream, a);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    const dim3 grid((unsigned)qk::ceil_div(d->vdim, kScanCols), (unsigned)d->heads, (unsigned)d->segments);
    const int vec = d->dim % 4 == 0 && a.channels % 4 == 0 && ((uintptr_t)d->qkv & 15) == 0 &&
                    ((uintptr_t)d->state & 15) == 0;
#define QK_SCAN(per) \
    (void)qk::launch_pdl(c->pdl, delta_scan_kernel<per>, grid, dim3(kScanThreads), 0, c->stream, a, vec)
    if (d->dim <= 32) QK_SCAN(4);
    else if (d->dim <= 64) QK_SCAN(8);
    else if (d->dim <= 128) QK_SCAN(16);
    else if (d->dim <= 256) QK_SCAN(32);
    else QK_SCAN(64);
#undef QK_SCAN
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
}

}  // extern "C"
