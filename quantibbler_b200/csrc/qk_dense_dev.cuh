// Device code shared by the forms of the dense linear (qk_dense.cu): how the input vector of a
// row is formed (plain, normed with a pending residual, concatenated, gated) and what happens
// to a result (store, residual, gated pair, token-side product).  The matrix-vector form calls
// these inside its own kernel; the matrix forms call the same functions from a kernel in front
// of the product and from their epilogues.
#pragma once

#include <cstdint>

#include "qk_common.h"
#include "qk_decoder_dev.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return __fdividef(z, 1.0f + expf(-z)); }
// 0.5 z (1 + tanh u) = z sigmoid(2 u)
__device__ __forceinline__ float gelu_tanh_f(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.0f + expf(-2.0f * u));
}
__device__ __forceinline__ float activate(int kind, float z) {
    return kind == QK_ACT_RELU ? fmaxf(z, 0.f) : kind == QK_ACT_SILU ? silu_f(z) : gelu_tanh_f(z);
}

struct AppendArgs {
    const float *src, *weight;
    void *cache;
    uint32_t src_stride, width, ring, stride;
    float eps;
    int bf16;
};
struct InputArgs {
    const float *x, *pending, *pending_weight, *second, *norm_weight, *gate;
    float *x_out;
    const int32_t *positions, *slots;
    uint32_t x_stride, pending_stride, gate_stride, width, k, group;
    float pending_eps, norm_eps;
    int kind, norm;
    AppendArgs append;
    // the pending value's y is a sum of pending_top rows times pending_scale (0: row t itself)
    const int32_t *pending_rows;
    uint32_t pending_top;
    float pending_scale;
    // the input rows of the matrix forms are stored once per choice, at places[t][..] (null: at t)
    const int32_t *places;
    uint32_t top;
};
// The choices of a linear with experts, for the vector form.
struct ChoiceArgs {
    const int32_t *table, *ids;
    uint32_t top, vocab, by_choice;
};
__device__ __forceinline__ const float *pending_row(const InputArgs &a, uint32_t t, uint32_t j) {
    const uint32_t at = t * a.pending_top + j;
    return a.pending + (size_t)(a.pending_rows ? (uint32_t)a.pending_rows[at] : at) * a.pending_stride;
}
struct OutputArgs {
    void *out;
    float *residual;
    const float *scale;
    const void *side;
    const int32_t *ids;
    uint32_t out_stride, residual_stride, side_stride, side_offset, vocab;
    int kind, act, out_bf16, side_bf16;
};

// The sum over a block of `kInThreads` threads; `red` holds one float per warp.
__device__ __forceinline__ float in_block_sum(float v, float *red) { return block_sum(v, red); }

// kInBatch values per thread are requested together before any of them is used: these loops are
// pure latency when a step has one row.
template <int kInBatch = 8, typename F>
__device__ __forceinline__ void in_load(const float *__restrict__ p, uint32_t n, F &&use) {
    for (uint32_t base = threadIdx.x; base < n; base += kInBatch * blockDim.x) {
        float v[kInBatch];
#pragma unroll
        for (int j = 0; j < kInBatch; ++j) v[j] = p[min(base + j * blockDim.x, n - 1)];
#pragma unroll
        for (int j = 0; j < kInBatch; ++j) {
            const uint32_t i = base + j * blockDim.x;
            if (i < n) use(i, v[j]);
        }
    }
}

// Forms the input vector of row t: `at(i)` is a reference to the shared-memory place of entry i
// (0 <= i < k).  Ends with the whole vector visible to the block.  `writer`: this block stores
// x_out.
template <typename At>
__device__ __forceinline__ void build_input(const InputArgs &a, uint32_t t, bool writer, At &&at, float *red) {
    const uint32_t n = a.width;
    const float *xr = a.x + (size_t)t * a.x_stride;
    if (a.kind == QK_INPUT_PLAIN) {
        in_load<16>(xr, n, [&](uint32_t i, float v) { at(i) = v; });
        for (uint32_t i = n + threadIdx.x; i < a.k; i += blockDim.x) at(i) = 0.f;
        __syncthreads();
        return;
    }
    if (a.kind == QK_INPUT_GATED) {
        in_load(xr, n, [&](uint32_t i, float v) { at(i) = v; });
        for (uint32_t i = n + threadIdx.x; i < a.k; i += blockDim.x) at(i) = 0.f;
        __syncthreads();
        const float *gr = a.gate + (size_t)t * a.gate_stride;
        const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, nw = blockDim.x / 32, g = a.group;
        for (uint32_t h = warp; h < n / g; h += nw) {
            float ss = 0.f;
            for (uint32_t i = lane; i < g; i += 32) {
                const float v = at(h * g + i);
                ss += v * v;
            }
            for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
            const float inv = 1.0f / sqrtf(ss / (float)g + a.norm_eps);
            for (uint32_t i = lane; i < g; i += 32)
                at(h * g + i) = at(h * g + i) * inv * a.norm_weight[i] * silu_f(gr[h * g + i]);
        }
        __syncthreads();
        return;
    }
    // h = x + pending
    float sum = 0.f, sq = 0.f;
    if (a.pending) {
        float ps = 0.f;
        if (a.pending_top) {
            for (uint32_t j = 0; j < a.pending_top; ++j)
                in_load(pending_row(a, t, j), n, [&](uint32_t i, float v) { at(i) = j ? at(i) + v : v; });
            for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
                const float v = at(i) * a.pending_scale;
                at(i) = v;
                ps += v * v;
            }
        } else {
            in_load(a.pending + (size_t)t * a.pending_stride, n, [&](uint32_t i, float v) {
                at(i) = v;
                ps += v * v;
            });
        }
        const float inv = 1.0f / sqrtf(in_block_sum(ps, red) / (float)n + a.pending_eps);
        const float *pw = a.pending_weight;
        in_load(xr, n, [&](uint32_t i, float v) {
            const float h = v + at(i) * inv * pw[i];
            at(i) = h;
            if (writer && a.x_out) a.x_out[(size_t)t * a.x_stride + i] = h;
            sum += h;
            sq += h * h;
        });
    } else {
        in_load(xr, n, [&](uint32_t i, float v) {
            at(i) = v;
            if (writer && a.x_out) a.x_out[(size_t)t * a.x_stride + i] = v;
            sum += v;
            sq += v * v;
        });
    }
    // (every thread goes on with the entries it has written itself)
    if (a.norm == QK_NORM_LAYER) {
        const float mean = in_block_sum(sum, red) / (float)n;
        float dev = 0.f;
        for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
            const float d = at(i) - mean;
            dev += d * d;
        }
        const float inv = 1.0f / sqrtf(in_block_sum(dev, red) / (float)n + a.norm_eps);
        in_load(a.norm_weight, n, [&](uint32_t i, float w) { at(i) = (at(i) - mean) * inv * w; });
    } else if (a.norm == QK_NORM_RMS) {
        const float inv = 1.0f / sqrtf(in_block_sum(sq, red) / (float)n + a.norm_eps);
        in_load(a.norm_weight, n, [&](uint32_t i, float w) { at(i) = at(i) * inv * w; });
    }
    if (a.kind == QK_INPUT_CONCAT) {
        const uint32_t half = a.k / 2;
        for (uint32_t i = n + threadIdx.x; i < half; i += blockDim.x) at(i) = 0.f;
        in_load(a.second + (size_t)t * a.x_stride, n, [&](uint32_t i, float v) { at(half + i) = v; });
        for (uint32_t i = half + n + threadIdx.x; i < a.k; i += blockDim.x) at(i) = 0.f;
    } else {
        for (uint32_t i = n + threadIdx.x; i < a.k; i += blockDim.x) at(i) = 0.f;
    }
    __syncthreads();
}

// The same for a normed row of up to 1024 kNormPieces aligned entries, for 256 threads: all loads of the
// row go out together, the norms' weights have been staged by stage_norm_weights (which depends on no
// other kernel).  `at4(p)` is the shared-memory place of entries 4 p .. 4 p + 3.
constexpr int kNormPieces = 4;
__device__ __forceinline__ void stage16(float *smem, const float *gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
// staged: [2][width] floats (every thread reads back only what it has copied itself)
__device__ __forceinline__ void stage_norm_weights(const InputArgs &a, float *staged) {
    for (uint32_t p = threadIdx.x; p < a.width / 4; p += 256) {
        if (a.norm != QK_NORM_NONE) stage16(staged + 4 * p, a.norm_weight + 4 * p);
        if (a.pending) stage16(staged + a.width + 4 * p, a.pending_weight + 4 * p);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}
template <typename At4>
__device__ __forceinline__ void build_norm_row(const InputArgs &a, uint32_t t, bool writer, const float *staged, At4 &&at4,
                                               float *red) {
    const uint32_t n = a.width, pieces = n / 4;
    const float4 *xr = reinterpret_cast<const float4 *>(a.x + (size_t)t * a.x_stride);
    const float4 *nw = reinterpret_cast<const float4 *>(staged), *pw = nw + pieces;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 h[kNormPieces];
#pragma unroll
    for (int j = 0; j < kNormPieces; ++j) {
        const uint32_t p = threadIdx.x + 256 * j;
        h[j] = p < pieces ? xr[p] : zero;
    }
    if (a.pending) {
        const uint32_t parts = a.pending_top ? a.pending_top : 1;
        float4 y[kNormPieces];
        for (uint32_t c = 0; c < parts; ++c) {
            const float4 *pr = reinterpret_cast<const float4 *>(
                a.pending_top ? pending_row(a, t, c) : a.pending + (size_t)t * a.pending_stride);
#pragma unroll
            for (int j = 0; j < kNormPieces; ++j) {
                const uint32_t p = threadIdx.x + 256 * j;
                const float4 v = p < pieces ? pr[p] : zero;
                y[j] = c ? make_float4(y[j].x + v.x, y[j].y + v.y, y[j].z + v.z, y[j].w + v.w) : v;
            }
        }
        const float share = a.pending_top ? a.pending_scale : 1.f;
        float ps = 0.f;
#pragma unroll
        for (int j = 0; j < kNormPieces; ++j) {
            y[j] = make_float4(y[j].x * share, y[j].y * share, y[j].z * share, y[j].w * share);
            ps += y[j].x * y[j].x + y[j].y * y[j].y + y[j].z * y[j].z + y[j].w * y[j].w;
        }
        const float inv = 1.0f / sqrtf(in_block_sum(ps, red) / (float)n + a.pending_eps);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        float4 *xo = writer && a.x_out ? reinterpret_cast<float4 *>(a.x_out + (size_t)t * a.x_stride) : nullptr;
#pragma unroll
        for (int j = 0; j < kNormPieces; ++j) {
            const uint32_t p = threadIdx.x + 256 * j;
            if (p >= pieces) continue;
            const float4 w = pw[p];
            h[j].x += y[j].x * inv * w.x;
            h[j].y += y[j].y * inv * w.y;
            h[j].z += y[j].z * inv * w.z;
            h[j].w += y[j].w * inv * w.w;
            if (xo) xo[p] = h[j];
        }
    } else if (writer && a.x_out) {
        float4 *xo = reinterpret_cast<float4 *>(a.x_out + (size_t)t * a.x_stride);
#pragma unroll
        for (int j = 0; j < kNormPieces; ++j)
            if (threadIdx.x + 256 * j < pieces) xo[threadIdx.x + 256 * j] = h[j];
    }
    float mean = 0.f, inv = 1.f;
    if (a.norm == QK_NORM_LAYER) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < kNormPieces; ++j) s += h[j].x + h[j].y + h[j].z + h[j].w;
        mean = in_block_sum(s, red) / (float)n;
    }
    if (a.norm != QK_NORM_NONE) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < kNormPieces; ++j) {
            if (threadIdx.x + 256 * j >= pieces) continue;
            const float b = h[j].x - mean, c = h[j].y - mean, d = h[j].z - mean, e = h[j].w - mean;
            s += b * b + c * c + d * d + e * e;
        }
        inv = 1.0f / sqrtf(in_block_sum(s, red) / (float)n + a.norm_eps);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int j = 0; j < kNormPieces; ++j) {
        const uint32_t p = threadIdx.x + 256 * j;
        if (p >= pieces) continue;
        float4 v = h[j];
        if (a.norm != QK_NORM_NONE) {
            const float4 w = nw[p];
            v = make_float4((v.x - mean) * inv * w.x, (v.y - mean) * inv * w.y, (v.z - mean) * inv * w.z, (v.w - mean) * inv * w.w);
        }
        at4(p) = v;
    }
    for (uint32_t p = pieces + threadIdx.x; p < a.k / 4; p += 256) at4(p) = zero;
    __syncthreads();
}
// A plain row in aligned pieces.
template <typename At4>
__device__ __forceinline__ void build_plain_row(const InputArgs &a, uint32_t t, At4 &&at4) {
    const uint32_t pieces = a.width / 4;
    const float4 *xr = reinterpret_cast<const float4 *>(a.x + (size_t)t * a.x_stride);
    for (uint32_t base = threadIdx.x; base < pieces; base += 8 * 256) {
        float4 v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = xr[min(base + 256 * j, pieces - 1)];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (base + 256 * j < pieces) at4(base + 256 * j) = v[j];
    }
    for (uint32_t p = pieces + threadIdx.x; p < a.k / 4; p += 256) at4(p) = make_float4(0.f, 0.f, 0.f, 0.f);
    __syncthreads();
}

// The RMS-normed latent of row t into its slot's ring; nothing for an idle row.
__device__ __forceinline__ void append_latent(const InputArgs &a, uint32_t t, float *red) {
    const AppendArgs &p = a.append;
    const int pos = a.positions[t];
    if (pos < 0) return;  // (uniform over the block)
    const float *src = p.src + (size_t)t * p.src_stride;
    float ss = 0.f;
    in_load(src, p.width, [&](uint32_t, float v) { ss += v * v; });
    const float inv = 1.0f / sqrtf(in_block_sum(ss, red) / (float)p.width + p.eps);
    const size_t row = ((size_t)a.slots[t] * p.ring + (uint32_t)pos % p.ring) * p.stride;
    for (uint32_t i = threadIdx.x; i < p.stride; i += blockDim.x) {
        const float v = i < p.width ? src[i] * inv * p.weight[i] : 0.f;
        if (p.bf16) static_cast<uint16_t *>(p.cache)[row + i] = float_to_bf16_bits(v);
        else static_cast<float *>(p.cache)[row + i] = v;
    }
}

__device__ __forceinline__ void put(void *p, int bf16, size_t i, float v) {
    if (bf16) static_cast<uint16_t *>(p)[i] = float_to_bf16_bits(v);
    else static_cast<float *>(p)[i] = v;
}
__device__ __forceinline__ float side_value(const OutputArgs &o, uint32_t t, uint32_t n) {
    const uint32_t id = (uint32_t)min(max(o.ids[t], 0), (int)o.vocab - 1);
    const size_t at = (size_t)id * o.side_stride + o.side_offset + n;
    return o.side_bf16 ? bf16_bits_to_float(static_cast<const uint16_t *>(o.side)[at])
                       : static_cast<const float *>(o.side)[at];
}
// One finished element (not the gated pair).
__device__ __forceinline__ void finish(const OutputArgs &o, uint32_t t, uint32_t n, float v) {
    if (o.kind == QK_OUTPUT_RESIDUAL) {
        float *r = o.residual + (size_t)t * o.residual_stride + n;
        v = *r + (o.scale ? v * o.scale[n] : v);
        *r = v;
        if (!o.out) return;
    } else if (o.kind == QK_OUTPUT_SIDE) {
        v = activate(o.act, v) * side_value(o, t, n);
    }
    put(o.out, o.out_bf16, (size_t)t * o.out_stride + n, v);
}
// Output j of a gated pair.
__device__ __forceinline__ void finish_pair(const OutputArgs &o, uint32_t t, uint32_t j, float gate, float up) {
    put(o.out, o.out_bf16, (size_t)t * o.out_stride + j, activate(o.act, gate) * up);
}
// Gated pairs are stored as alternating blocks of 32 gate rows and 32 up rows.
__device__ __forceinline__ uint32_t pair_row(uint32_t j) { return (j / 32) * 64 + j % 32; }

}  // namespace
