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
#include <algorithm>

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

// The convolution's last taps - 1 inputs of a segment (their readers, the inputs kernel, have
// finished), shared out over the blocks of a segment (grid x and y).
__device__ __forceinline__ void keep_conv_inputs(const DeltaArgs &a, uint32_t slot, int pos0, uint32_t first,
                                                 uint32_t len, uint32_t threads) {
    const uint32_t keep = min(a.taps - 1, len);
    const uint32_t n_blocks = gridDim.x * gridDim.y, block = blockIdx.y * gridDim.x + blockIdx.x;
    for (uint32_t i = block * threads + threadIdx.x; i < keep * a.channels; i += n_blocks * threads) {
        const uint32_t back = i / a.channels, c = i % a.channels, r = len - 1 - back;
        a.conv_state[((size_t)slot * a.taps + (uint32_t)(pos0 + (int)r) % a.taps) * a.channels + c] =
            a.proj[(size_t)(first + r) * a.proj_stride + c];
    }
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
    keep_conv_inputs(a, slot, pos0, first, len, kScanThreads);
}

// ------------------------------------------------------------------ delta rule: a portion, eight tokens at a time
// For eight tokens from a state S0 on, with P_t = g_1 .. g_t and R_ti = g_i+1 .. g_t:
//   u_t = beta_t (v_t - P_t S0^T k_t - sum_{i<t} R_ti (k_i . k_t) u_i)
//   o_t = P_t S0^T q_t + sum_{i<=t} R_ti (k_i . q_t) u_i
//   S8  = P_8 S0 + sum_i R_8i k_i u_i^T
// so all sixteen products with the state are independent, and only an 8 x 8 triangular solve of
// scalars per column is sequential.  The scalars depend on the head alone: the inputs kernel
// writes them once, 20 floats per token: beta R (k . k) [8], R (k . q) [8], beta, beta P, P, R_8.
constexpr int kMini = 8, kCoef = 20;

// A block takes kTok rows and one key head with the heads it serves.  Thread per channel: convolution
// and silu of the rows from one window of loads (kTaps bounds the taps), then a warp per row for
// the unit norms, then the scalars.  kTok = 8: rows of one portion, kCoef scalars per row and
// head; kTok = 1: any row, {beta, g, k . q} per row and head.
template <int kTaps, int kTok>
__global__ void __launch_bounds__(256, kTaps <= 4 ? 4 : 2)
delta_inputs_kernel(DeltaArgs a, uint32_t n_tokens) {
    qk::pdl_launch();
    extern __shared__ float ci_smem[];  // q, k [kTok][dim + 1], then products, then [ratio][kTok][2] gates
    const uint32_t t0 = blockIdx.x * kTok, kvh = blockIdx.y, pitch = a.dim + 1, ratio = a.heads / a.kv_heads;
    float *qs = ci_smem, *ks = qs + kTok * pitch, *prod = ks + kTok * pitch, *gate = prod + 2 * kTok * kTok;
    const uint32_t n = min((uint32_t)kTok, n_tokens - t0), warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    qk::pdl_wait();
    const int pos = a.positions[t0];
    if (pos < 0) return;
    const int in_seg = a.seg_row[t0];
    const uint32_t slot = (uint32_t)a.slots[t0], key0 = a.kv_heads * a.dim, per = ratio * a.vdim;
#pragma unroll 1
    for (uint32_t c = threadIdx.x; c < 2 * a.dim + per; c += 256) {
        const uint32_t which = c < a.dim ? 0 : c < 2 * a.dim ? 1 : 2;
        const uint32_t in = which == 0 ? c : which == 1 ? c - a.dim : c - 2 * a.dim;   // place in this head's part
        const uint32_t own = which == 2 ? kvh * per + in : kvh * a.dim + in;          // row of the taps
        const uint32_t ch = which == 0 ? own : which == 1 ? key0 + own : 2 * key0 + own;
        const float *taps = (which == 0 ? a.conv_q : which == 1 ? a.conv_k : a.conv_v) + (size_t)own * a.taps;
        float w[kTaps], x[kTaps - 1 + kTok];
        if (in_seg >= kTaps - 1) {  // (uniform over the block) every earlier input is a row
            const float *src = a.proj + (size_t)(t0 - (kTaps - 1)) * a.proj_stride + ch;
#pragma unroll
            for (int j = 0; j < kTaps - 1 + kTok; ++j)
                x[j] = j - (kTaps - 1) < (int)n ? src[(size_t)j * a.proj_stride] : 0.f;
        } else
#pragma unroll
        for (int j = 0; j < kTaps - 1 + kTok; ++j) {
            const int r = j - (kTaps - 1), p = pos + r;  // row t0 + r at position p
            const bool row = r < (int)n && r >= -in_seg, kept = r < -in_seg && p >= 0 && -r < (int)a.taps;
            const float *src = row ? a.proj + (size_t)((int)t0 + r) * a.proj_stride + ch
                                   : a.conv_state + ((size_t)slot * a.taps + (uint32_t)(kept ? p : 0) % a.taps) * a.channels + ch;
            x[j] = row || kept ? *src : 0.f;
        }
#pragma unroll
        for (int j = 0; j < kTaps; ++j) w[j] = j < (int)a.taps ? taps[a.taps - 1 - j] : 0.f;   // w[j]: j tokens back
#pragma unroll
        for (int t = 0; t < kTok; ++t) {
            float y = 0.f;
#pragma unroll
            for (int j = 0; j < kTaps; ++j) y = fmaf(w[j], x[kTaps - 1 + t - j], y);
            y = silu_f(y);
            if (which == 2) {
                if (t < (int)n) a.qkv[(size_t)(t0 + t) * a.channels + ch] = y;
            } else {
                (which == 0 ? qs : ks)[t * pitch + in] = t < (int)n ? y : 0.f;
            }
        }
    }
    for (uint32_t i = threadIdx.x; i < ratio * kTok; i += 256) {
        const uint32_t h = kvh * ratio + i / kTok, t = i % kTok;
        float beta = 0.f, g = 1.f;
        if (t < n) {
            const float *pr = a.proj + (size_t)(t0 + t) * a.proj_stride;
            const float z = pr[a.decay_offset + h] + a.dt_bias[h];
            beta = sigmoid_f(pr[a.beta_offset + h]);
            g = expf(-expf(a.a_log[h]) * (z > 20.f ? z : log1pf(expf(z))));
        }
        gate[2 * i] = beta;
        gate[2 * i + 1] = g;
    }
    __syncthreads();
    if (warp < (uint32_t)kTok) {   // unit vectors: warp = row
        float sq = 0.f, sk = 0.f;
        for (uint32_t d = lane; d < a.dim; d += 32) {
            sq += qs[warp * pitch + d] * qs[warp * pitch + d];
            sk += ks[warp * pitch + d] * ks[warp * pitch + d];
        }
        for (int off = 16; off > 0; off >>= 1) {
            sq += __shfl_xor_sync(0xffffffffu, sq, off);
            sk += __shfl_xor_sync(0xffffffffu, sk, off);
        }
        const float iq = 1.0f / sqrtf(sq + a.unit_eps) * (1.0f / sqrtf((float)a.dim));
        const float ik = 1.0f / sqrtf(sk + a.unit_eps);
        float *row = a.qkv + (size_t)(t0 + warp) * a.channels + kvh * a.dim;
        float dot = 0.f;
        for (uint32_t d = lane; d < a.dim; d += 32) {
            const float q = qs[warp * pitch + d] * iq, k = ks[warp * pitch + d] * ik;
            qs[warp * pitch + d] = q;
            ks[warp * pitch + d] = k;
            dot += q * k;
            if (warp < n) {
                row[d] = q;
                row[key0 + d] = k;
            }
        }
        if constexpr (kTok == 1) {
            for (int off = 16; off > 0; off >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, off);
            for (uint32_t r = lane; r < ratio; r += 32) {
                float *dst = a.gates + ((size_t)t0 * a.heads + kvh * ratio + r) * 4;
                dst[0] = gate[2 * r];
                dst[1] = gate[2 * r + 1];
                dst[2] = dot;
            }
        }
    }
    if constexpr (kTok == 1) return;
    __syncthreads();
    {   // k_i . k_t and k_i . q_t: two threads per product
        const uint32_t pair = threadIdx.x / 2, half = threadIdx.x % 2, t = pair / kTok % kTok, i = pair % kTok;
        const float *x = (pair < kTok * kTok ? ks : qs) + t * pitch, *y = ks + i * pitch;
        float v = 0.f;
        for (uint32_t d = half; d < a.dim; d += 2) v = fmaf(x[d], y[d], v);
        v += __shfl_xor_sync(0xffffffffu, v, 1);
        if (half == 0 && pair < 2 * kTok * kTok) prod[pair] = v;
    }
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < ratio * kTok; i += 256) {
        const uint32_t r = i / kTok, t = i % kTok;
        const float *g = gate + r * kTok * 2;
        float *dst = a.gates + (((size_t)blockIdx.x * a.heads + kvh * ratio + r) * kTok + t) * kCoef;
        const float beta = g[2 * t];
        float decay = 1.f;  // R_ti, from i = t downwards
        for (int j = kTok - 1; j >= 0; --j) {
            float kk = 0.f, kq = 0.f;
            if (j <= (int)t) {
                if (j < (int)t) {
                    decay *= g[2 * (j + 1) + 1];
                    kk = beta * decay * prod[t * kTok + j];
                }
                kq = decay * prod[kTok * kTok + t * kTok + j];
            }
            dst[j] = kk;
            dst[kTok + j] = kq;
        }
        const float from_start = decay * g[1];  // (R_t0 g_0)
        float to_end = 1.f;
        for (uint32_t j = t + 1; j < (uint32_t)kTok; ++j) to_end *= g[2 * j + 1];
        dst[16] = beta;
        dst[17] = beta * from_start;
        dst[18] = from_start;
        dst[19] = to_end;
    }
}

// Sums over the lanes of 32 values each of two kinds, value (token, column): lane 4 t + c ends
// with token t, column c.  The lanes' register slot i holds token i ^ lane / 4, so that in the
// first three rounds every lane sends the upper half of its slots and keeps the lower.
__device__ __forceinline__ void scatter_sums(float (&x)[32], float (&y)[32], uint32_t lane) {
#pragma unroll
    for (int half = 16; half > 2; half >>= 1)
#pragma unroll
        for (int j = 0; j < half; ++j) {
            x[j] += __shfl_xor_sync(0xffffffffu, x[j + half], half);
            y[j] += __shfl_xor_sync(0xffffffffu, y[j + half], half);
        }
#pragma unroll
    for (int half = 2; half > 0; half >>= 1) {
        const bool up = (lane & half) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
            const float sx = up ? x[j] : x[j + half], kx = up ? x[j + half] : x[j];
            const float sy = up ? y[j] : y[j + half], ky = up ? y[j + half] : y[j];
            x[j] = kx + __shfl_xor_sync(0xffffffffu, sx, half);
            y[j] = ky + __shfl_xor_sync(0xffffffffu, sy, half);
        }
    }
}

constexpr int kChunkWarps = 4, kChunkCols = 4;  // columns per warp
template <int kE> struct ChunkShape {
    static constexpr int kDim = 32 * kE, kStages = kE > 4 ? 3 : 4, kCols = kChunkWarps * kChunkCols;
    static constexpr int kFloats = 2 * kMini * kDim + kMini * kCols + kMini * kCoef;  // per stage
    static constexpr size_t kSmem = ((size_t)kStages * kFloats + kChunkWarps * kMini * kChunkCols) * 4;
};
// kE: state entries per lane and column (dim <= 32 * kE): entry e of lane l is 128 (e / 4) + 4 l + e % 4
// (kE = 2: 2 l + e).  A warp owns four columns of one head.
template <int kE>
__global__ void __launch_bounds__(kChunkWarps * 32)
delta_chunk_scan_kernel(DeltaArgs a, uint32_t n_tokens, int vec) {
    using S = ChunkShape<kE>;
    constexpr int kPairs = kE / 2, kPiece = kE < 4 ? 2 : 4;
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) float cs_smem[];
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, h = blockIdx.y;
    const int pos0 = a.positions[0];
    if (pos0 < 0) return;
    const uint32_t slot = (uint32_t)a.slots[0], kvh = h / (a.heads / a.kv_heads), key0 = a.kv_heads * a.dim;
    const uint32_t col0 = blockIdx.x * S::kCols, n_chunks = (n_tokens + kMini - 1) / kMini;
    float *us = cs_smem + S::kStages * S::kFloats + warp * kMini * kChunkCols;
    if (a.dim < (uint32_t)S::kDim) {  // entries past dim stay zero
        for (uint32_t i = threadIdx.x; i < S::kStages * S::kFloats; i += kChunkWarps * 32) cs_smem[i] = 0.f;
        __syncthreads();
    }
    auto stage = [&](uint32_t chunk) {
        if (chunk < n_chunks) {
            float *q = cs_smem + (chunk % S::kStages) * S::kFloats, *k = q + kMini * S::kDim, *v = k + kMini * S::kDim;
            float *cf = v + kMini * S::kCols;
            const uint32_t t0 = chunk * kMini;
            if (vec) {
                const uint32_t per = a.dim / 4;
                for (uint32_t i = threadIdx.x; i < kMini * per; i += kChunkWarps * 32) {
                    const uint32_t t = i / per, d = (i % per) * 4;
                    const uint32_t bytes = t0 + t < n_tokens ? 16 : 0;
                    const float *src = a.qkv + (size_t)min(t0 + t, n_tokens - 1) * a.channels + kvh * a.dim + d;
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(
                                     (uint32_t)__cvta_generic_to_shared(q + t * S::kDim + d)), "l"(src), "r"(bytes) : "memory");
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(
                                     (uint32_t)__cvta_generic_to_shared(k + t * S::kDim + d)), "l"(src + key0), "r"(bytes) : "memory");
                }
            } else {
                for (uint32_t i = threadIdx.x; i < kMini * a.dim; i += kChunkWarps * 32) {
                    const uint32_t t = i / a.dim, d = i % a.dim;
                    const uint32_t bytes = t0 + t < n_tokens ? 4 : 0;
                    const float *src = a.qkv + (size_t)min(t0 + t, n_tokens - 1) * a.channels + kvh * a.dim + d;
                    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(
                                     (uint32_t)__cvta_generic_to_shared(q + t * S::kDim + d)), "l"(src), "r"(bytes) : "memory");
                    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(
                                     (uint32_t)__cvta_generic_to_shared(k + t * S::kDim + d)), "l"(src + key0), "r"(bytes) : "memory");
                }
            }
            for (uint32_t i = threadIdx.x; i < kMini * S::kCols; i += kChunkWarps * 32) {
                const uint32_t t = i / S::kCols, j = i % S::kCols;
                const uint32_t bytes = t0 + t < n_tokens && col0 + j < a.vdim ? 4 : 0;
                const float *src = a.qkv + (size_t)min(t0 + t, n_tokens - 1) * a.channels + 2 * key0 + h * a.vdim +
                                   min(col0 + j, a.vdim - 1);
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(
                                 (uint32_t)__cvta_generic_to_shared(v + t * S::kCols + j)), "l"(src), "r"(bytes) : "memory");
            }
            if (threadIdx.x < kMini * kCoef / 4)
                copy_async16(cf + threadIdx.x * 4, a.gates + ((size_t)chunk * a.heads + h) * kMini * kCoef + threadIdx.x * 4);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < S::kStages - 1; ++i) stage(i);

    f32x2 s[kChunkCols][kPairs];
    auto entry = [&](int pair) -> uint32_t {  // first entry of a pair
        return kE < 4 ? 2 * lane : 128 * (pair / 2) + 4 * lane + 2 * (pair % 2);
    };
#pragma unroll
    for (int c = 0; c < kChunkCols; ++c) {
        const uint32_t col = col0 + warp * kChunkCols + c;
        const float *st = a.state + (((size_t)slot * a.heads + h) * a.vdim + min(col, a.vdim - 1)) * a.dim;
#pragma unroll
        for (int p = 0; p < kPairs; ++p) {
            const uint32_t d = entry(p);
            const float x = pos0 != 0 && d < a.dim ? st[d] : 0.f, y = pos0 != 0 && d + 1 < a.dim ? st[d + 1] : 0.f;
            s[c][p] = pack2(x, y);
        }
    }
    const uint32_t my_t = lane / kChunkCols, my_c = lane % kChunkCols;
    const uint32_t my_col = col0 + warp * kChunkCols + my_c;
    for (uint32_t chunk = 0; chunk < n_chunks; ++chunk) {
        asm volatile("cp.async.wait_group %0;" ::"n"(S::kStages - 2) : "memory");
        __syncthreads();  // chunk has landed; the stage before it may be filled again
        stage(chunk + S::kStages - 1);
        const float *q = cs_smem + (chunk % S::kStages) * S::kFloats, *k = q + kMini * S::kDim, *v = k + kMini * S::kDim;
        const float *cf = v + kMini * S::kCols + my_t * kCoef;
        auto piece = [&](const float *row, f32x2 (&x)[kPairs]) {
#pragma unroll
            for (int p = 0; p < kE / kPiece; ++p) {
                if constexpr (kE < 4) {
                    x[0] = *reinterpret_cast<const f32x2 *>(row + 2 * lane);
                } else {
                    const ulonglong2 w = *reinterpret_cast<const ulonglong2 *>(row + 128 * p + 4 * lane);
                    x[2 * p] = w.x;
                    x[2 * p + 1] = w.y;
                }
            }
        };
        float dk[32], dq[32];
#pragma unroll
        for (int i = 0; i < kMini; ++i) {
            f32x2 x[kPairs], y[kPairs];
            const uint32_t at = ((uint32_t)i ^ my_t) * S::kDim;
            piece(k + at, x);
            piece(q + at, y);
#pragma unroll
            for (int c = 0; c < kChunkCols; ++c) {
                f32x2 ak = mul2(s[c][0], x[0]), aq = mul2(s[c][0], y[0]);
#pragma unroll
                for (int p = 1; p < kPairs; ++p) {
                    ak = fma2(s[c][p], x[p], ak);
                    aq = fma2(s[c][p], y[p], aq);
                }
                float lo, hi;
                unpack2(ak, lo, hi);
                dk[i * kChunkCols + c] = lo + hi;
                unpack2(aq, lo, hi);
                dq[i * kChunkCols + c] = lo + hi;
            }
        }
        scatter_sums(dk, dq, lane);
        const float sk = dk[0], sq = dq[0];
        // lane (t, c): the triangular solve over the tokens of column c
        float kk[kMini], kq[kMini];
#pragma unroll
        for (int i = 0; i < kMini; i += 4) {
            const float4 x = *reinterpret_cast<const float4 *>(cf + i), y = *reinterpret_cast<const float4 *>(cf + kMini + i);
            kk[i] = x.x; kk[i + 1] = x.y; kk[i + 2] = x.z; kk[i + 3] = x.w;
            kq[i] = y.x; kq[i + 1] = y.y; kq[i + 2] = y.z; kq[i + 3] = y.w;
        }
        const float4 g = *reinterpret_cast<const float4 *>(cf + 16);  // beta, beta P, P, R_8
        float u = g.x * v[my_t * S::kCols + warp * kChunkCols + my_c] - g.y * sk, o = g.z * sq;
#pragma unroll
        for (int i = 0; i < kMini; ++i) {
            const float ui = __shfl_sync(0xffffffffu, u, i * kChunkCols + my_c);
            u = fmaf(-kk[i], ui, u);
            o = fmaf(kq[i], ui, o);
        }
        const uint32_t t = chunk * kMini + my_t;
        if (t < n_tokens && my_col < a.vdim) a.out[(size_t)t * a.out_stride + h * a.vdim + my_col] = o;
        const float p8 = __shfl_sync(0xffffffffu, g.z, 31);  // P of the last token
        us[lane] = u * g.w;
        __syncwarp();
        const f32x2 p2 = pack2(p8, p8);
#pragma unroll
        for (int c = 0; c < kChunkCols; ++c)
#pragma unroll
            for (int p = 0; p < kPairs; ++p) s[c][p] = mul2(p2, s[c][p]);
#pragma unroll
        for (int i = 0; i < kMini; ++i) {
            const float4 w = *reinterpret_cast<const float4 *>(us + i * kChunkCols);
            const float uw[4] = {w.x, w.y, w.z, w.w};
            f32x2 x[kPairs];
            piece(k + i * S::kDim, x);
#pragma unroll
            for (int c = 0; c < kChunkCols; ++c) {
                const f32x2 u2 = pack2(uw[c], uw[c]);
#pragma unroll
                for (int p = 0; p < kPairs; ++p) s[c][p] = fma2(x[p], u2, s[c][p]);
            }
        }
        __syncwarp();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int c = 0; c < kChunkCols; ++c) {
        const uint32_t col = col0 + warp * kChunkCols + c;
        if (col >= a.vdim) break;
        float *st = a.state + (((size_t)slot * a.heads + h) * a.vdim + col) * a.dim;
#pragma unroll
        for (int p = 0; p < kPairs; ++p) {
            const uint32_t d = entry(p);
            float x, y;
            unpack2(s[c][p], x, y);
            if (d < a.dim) st[d] = x;
            if (d + 1 < a.dim) st[d + 1] = y;
        }
    }
    keep_conv_inputs(a, slot, pos0, 0, n_tokens, kChunkWarps * 32);
}

template <int kE>
qk_status launch_chunk_scan(qk_ctx *c, const DeltaArgs &a, size_t tokens, int vec) {
    using S = ChunkShape<kE>;
    QK_CUDA(cudaFuncSetAttribute(delta_chunk_scan_kernel<kE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::kSmem));
    // (no early launch: blocks that came in while the inputs kernel drains would crowd on the few
    // SMs that are free first, and stay there)
    (void)qk::launch_pdl(false, delta_chunk_scan_kernel<kE>, dim3((a.vdim + S::kCols - 1) / S::kCols, a.heads),
                         dim3(kChunkWarps * 32), S::kSmem, c->stream, a, (uint32_t)tokens, vec);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
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
    if (d->taps > 16) return qk::fail(QK_ERR_VALUE, "qk_delta: more than 16 taps are not supported, got %zu", d->taps);
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
    const int vec = d->dim % 4 == 0 && a.channels % 4 == 0 && ((uintptr_t)d->qkv & 15) == 0 &&
                    ((uintptr_t)d->state & 15) == 0;
    const bool portion = d->segments == 1 && d->tokens >= (size_t)kMini;  // eight tokens at a time
    const size_t tok = portion ? kMini : 1;
    const dim3 ig((unsigned)qk::ceil_div(d->tokens, tok), a.kv_heads);
    const size_t smem = (2 * tok * (d->dim + 1) + 2 * tok * tok + d->heads / d->kv_heads * tok * 2) * 4;
    if (smem > 200 * 1024) return qk::fail(QK_ERR_VALUE, "qk_delta: %zu heads over %zu key heads", d->heads, d->kv_heads);
#define QK_INPUTS(taps, tok)                                                                                    \
    do {                                                                                                        \
        QK_CUDA(cudaFuncSetAttribute(delta_inputs_kernel<taps, tok>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                     (int)std::max(smem, (size_t)48 * 1024)));                                  \
        (void)qk::launch_pdl(c->pdl, delta_inputs_kernel<taps, tok>, ig, dim3(256), smem, c->stream, a,         \
                             (uint32_t)d->tokens);                                                              \
    } while (0)
    if (portion) {
        if (d->taps <= 4) QK_INPUTS(4, kMini);
        else QK_INPUTS(16, kMini);
    } else {
        if (d->taps <= 4) QK_INPUTS(4, 1);
        else QK_INPUTS(16, 1);
    }
#undef QK_INPUTS
    QK_CUDA(cudaGetLastError());
    c->launches++;
    if (portion)
        return d->dim <= 64 ? launch_chunk_scan<2>(c, a, d->tokens, vec)
               : d->dim <= 128 ? launch_chunk_scan<4>(c, a, d->tokens, vec)
               : d->dim <= 256 ? launch_chunk_scan<8>(c, a, d->tokens, vec)
                               : launch_chunk_scan<16>(c, a, d->tokens, vec);
    const dim3 grid((unsigned)qk::ceil_div(d->vdim, kScanCols), (unsigned)d->heads, (unsigned)d->segments);
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
