// Windowed attention over latents: k = W_uk c and v = W_uv c of one cached latent c per token, no
// positions.  Two forms:
//   * absorbed (decoding, short portions, float32): the scores of a head are (W_uk^T q) . c, the
//     output is W_uv (sum p c), so a row touches only the latents in its window.  Three launches:
//     W_uk^T q per head; the window's keys split over blocks, each with its own running maximum
//     (bfloat16: mma.sync with q and p split into two bfloat16 terms; otherwise float32); the
//     splits combined and W_uv applied.
//   * expanded (long portions, bfloat16): a matrix product has turned the window's latents into k
//     and v; flash attention over a band of keys on the tensor cores.
// The latents live in a ring per slot: position p in row p mod ring.
#include <algorithm>

#include "qk_dense_dev.cuh"
#include "qk_mma.cuh"

namespace {

// eight consecutive weights as floats
__device__ __forceinline__ void lt_load8(const uint16_t *p, float (&w)[8]) {
    const uint4 v = *reinterpret_cast<const uint4 *>(p);
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        w[2 * i] = __uint_as_float(u[i] << 16);
        w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void lt_load8(const float *p, float (&w)[8]) {
    const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
    w[0] = a.x; w[1] = a.y; w[2] = a.z; w[3] = a.w;
    w[4] = b.x; w[5] = b.y; w[6] = b.z; w[7] = b.w;
}

struct LatentArgs {
    const int32_t *positions, *slots;
    const float *q;
    float *absorbed;   // [tokens][heads][kv_stride]
    float *partial;    // [tokens][heads][n_splits][kv_stride + 8]: sums, then maximum and weight
    void *out;
    uint32_t tokens, heads, dim, dim_stride, vdim, vdim_stride, kv_stride, window, ring, n_splits, q_stride, out_stride;
    float scale;
    int out_bf16;
};

// The keys of one split of one row: first position and count.
struct SplitKeys {
    uint32_t first, count;
};
__device__ __forceinline__ SplitKeys split_keys(const LatentArgs &a, int pos, uint32_t split) {
    const uint32_t n = min(a.window, (uint32_t)pos + 1u), lo = (uint32_t)pos + 1u - n;
    const uint32_t per = (n + a.n_splits - 1) / a.n_splits;
    const uint32_t b = min(split * per, n), e = min(b + per, n);
    return {lo + b, e - b};
}

// ------------------------------------------------------------------ absorbed: W_uk^T q
constexpr int kAbsRows = 4, kAbsWarps = 8, kAbsAhead = 8;
__device__ __forceinline__ void lt_fetch8(const uint16_t *p, uint4 (&w)[1]) { w[0] = *reinterpret_cast<const uint4 *>(p); }
__device__ __forceinline__ void lt_fetch8(const float *p, uint4 (&w)[2]) {
    w[0] = *reinterpret_cast<const uint4 *>(p);
    w[1] = *reinterpret_cast<const uint4 *>(p + 4);
}
__device__ __forceinline__ void lt_open8(const uint4 (&v)[1], float (&w)[8]) {
    const uint32_t u[4] = {v[0].x, v[0].y, v[0].z, v[0].w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        w[2 * i] = __uint_as_float(u[i] << 16);
        w[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void lt_open8(const uint4 (&v)[2], float (&w)[8]) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        w[4 * i] = __uint_as_float(v[i].x);
        w[4 * i + 1] = __uint_as_float(v[i].y);
        w[4 * i + 2] = __uint_as_float(v[i].z);
        w[4 * i + 3] = __uint_as_float(v[i].w);
    }
}
template <typename W>
__global__ void __launch_bounds__(kAbsWarps * 32)
absorb_query_kernel(LatentArgs a, const W *__restrict__ uk) {
    qk::pdl_launch();
    extern __shared__ float ab_smem[];  // [kAbsRows][dim] queries, [kAbsWarps][256] sums
    float *qs = ab_smem, *sums = ab_smem + kAbsRows * a.dim;
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, h = blockIdx.y;
    const uint32_t c0 = blockIdx.x * 256 + lane * 8, t0 = blockIdx.z * kAbsRows;
    const bool live = c0 < a.kv_stride;
    const W *base = uk + (size_t)h * a.dim_stride * a.kv_stride + (live ? c0 : 0);
    uint4 ahead[kAbsAhead][sizeof(W) / 2];
    auto fetch = [&](uint32_t d0) {
#pragma unroll
        for (int i = 0; i < kAbsAhead; ++i)
            lt_fetch8(base + (size_t)min(d0 + i * kAbsWarps, a.dim - 1) * a.kv_stride, ahead[i]);
    };
    fetch(warp);  // (weights depend on no other kernel)
    qk::pdl_wait();
    for (uint32_t i = threadIdx.x; i < kAbsRows * a.dim; i += kAbsWarps * 32)
        qs[i] = a.q[(size_t)min(t0 + i / a.dim, a.tokens - 1) * a.q_stride + h * a.dim_stride + i % a.dim];
    __syncthreads();
    float acc[kAbsRows][8];
#pragma unroll
    for (int r = 0; r < kAbsRows; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = 0.f;
    for (uint32_t d0 = warp; d0 < a.dim; d0 += kAbsAhead * kAbsWarps) {
        if (d0 != warp) fetch(d0);
#pragma unroll
        for (int i = 0; i < kAbsAhead; ++i) {
            const uint32_t d = d0 + i * kAbsWarps;
            if (d >= a.dim) break;
            float w[8];
            lt_open8(ahead[i], w);
#pragma unroll
            for (int r = 0; r < kAbsRows; ++r) {
                const float q = qs[r * a.dim + d];
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(q, w[e], acc[r][e]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < kAbsRows; ++r) {
        if (t0 + r >= a.tokens) break;
#pragma unroll
        for (int e = 0; e < 8; ++e) sums[warp * 256 + lane * 8 + e] = acc[r][e];
        __syncthreads();
        const uint32_t c = blockIdx.x * 256 + threadIdx.x;
        if (c < a.kv_stride) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < kAbsWarps; ++w) v += sums[w * 256 + threadIdx.x];
            a.absorbed[((size_t)(t0 + r) * a.heads + h) * a.kv_stride + c] = v * a.scale;
        }
        __syncthreads();
    }
}

// ------------------------------------------------------------------ absorbed: scores and sums, float32
constexpr int kPlainThreads = 128, kPlainKeys = 64;
template <typename C>
__global__ void __launch_bounds__(kPlainThreads)
latent_plain_kernel(LatentArgs a, const C *__restrict__ cache) {
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ float lp_smem[];  // [kv_stride] query, [kv_stride] sums
    __shared__ float p[kPlainKeys];
    float *qv = lp_smem, *o = lp_smem + a.kv_stride;
    const uint32_t split = blockIdx.x, h = blockIdx.y, t = blockIdx.z, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const int pos = a.positions[t];
    if (pos < 0) return;
    const SplitKeys keys = split_keys(a, pos, split);
    const C *base = cache + (size_t)a.slots[t] * a.ring * a.kv_stride;
    float *dst = a.partial + (((size_t)t * a.heads + h) * a.n_splits + split) * (a.kv_stride + 8);
    for (uint32_t i = threadIdx.x; i < a.kv_stride; i += kPlainThreads) {
        qv[i] = a.absorbed[((size_t)t * a.heads + h) * a.kv_stride + i];
        o[i] = 0.f;
    }
    __syncthreads();
    float m = -INFINITY, l = 0.f;
    for (uint32_t k0 = 0; k0 < keys.count; k0 += kPlainKeys) {
        const uint32_t n = min((uint32_t)kPlainKeys, keys.count - k0);
        for (uint32_t j = warp; j < n; j += kPlainThreads / 32) {
            const C *row = base + (size_t)((keys.first + k0 + j) % a.ring) * a.kv_stride;
            float s = 0.f;
            for (uint32_t i = lane; i < a.kv_stride; i += 32) s = fmaf(qv[i], load_as_float(row, i), s);
            for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
            if (lane == 0) p[j] = s;
        }
        __syncthreads();
        float mx = m;
        for (uint32_t j = 0; j < n; ++j) mx = fmaxf(mx, p[j]);
        const float alpha = m == -INFINITY ? 0.f : expf(m - mx);
        m = mx;
        l *= alpha;
        __syncthreads();  // every thread has read the scores
        if (threadIdx.x < n) p[threadIdx.x] = expf(p[threadIdx.x] - m);
        __syncthreads();
        for (uint32_t j = 0; j < n; ++j) l += p[j];
        for (uint32_t i = threadIdx.x; i < a.kv_stride; i += kPlainThreads) {
            float acc = o[i] * alpha;
            for (uint32_t j = 0; j < n; ++j)
                acc = fmaf(p[j], load_as_float(base, (size_t)((keys.first + k0 + j) % a.ring) * a.kv_stride + i), acc);
            o[i] = acc;
        }
        __syncthreads();
    }
    for (uint32_t i = threadIdx.x; i < a.kv_stride; i += kPlainThreads) dst[i] = o[i];
    if (threadIdx.x == 0) {
        dst[a.kv_stride] = m;
        dst[a.kv_stride + 1] = l;
    }
}

// ------------------------------------------------------------------ absorbed: scores and sums, tensor cores
// A block of four warps takes up to 16 heads (the M side) of one row and one split of its keys,
// 32 keys at a time.  Each warp owns a quarter of the latent channels: it stages that quarter of
// the keys for itself, keeps the query's fragments of it in registers, multiplies the scores'
// share of its channels and later sums the same channels; only the scores meet in shared
// memory.  KV: staged channels per key (kv_stride <= KV).
constexpr int kLatKeys = 32;
template <int KV> struct LatShape {
    static constexpr int kQuarter = KV / 4, kPitch = kQuarter + 8, kBufs = 2;
    static constexpr int kScorePitch = kLatKeys + 4;
    static constexpr size_t kTileBytes = kLatKeys * kPitch * 2;             // one warp's quarter of 32 keys
    static constexpr size_t kRing = 4 * kBufs * kTileBytes, kScores = 2 * 4 * 16 * kScorePitch * 4;
    static constexpr size_t kSums = (16 * (KV + 4) + 32) * 4;               // after the last tile
    static constexpr size_t kSmem = (kRing > kSums ? kRing : kSums) + kScores;
};
__device__ __forceinline__ void lat_cluster_sync() {
    __syncwarp();
    asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t lat_map(const float *p, uint32_t cta) {
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(cta));
    return r;
}
__device__ __forceinline__ float lat_peer(const float *p, uint32_t cta) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(lat_map(p, cta)) : "memory");
    return v;
}
__device__ __forceinline__ float4 lat_peer4(const float *p, uint32_t cta) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];"
                 : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w)
                 : "r"(lat_map(p, cta))
                 : "memory");
    return v;
}
// TERMS: bfloat16 terms of the query and of the weights (two keep float32 accuracy).
template <int KV, int TERMS>
__global__ void __launch_bounds__(128)
latent_mma_kernel(LatentArgs a, const uint16_t *__restrict__ cache, uint32_t cluster) {
    using S = LatShape<KV>;
    constexpr int kQ = S::kQuarter, kSteps = kQ / 16, kTilesPerWarp = kQ / 8;
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) uint8_t lat_smem[];
    const uint32_t split = blockIdx.x, h0 = blockIdx.y * 16, t = blockIdx.z;
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane >> 2, c4 = lane & 3;
    const int pos = a.positions[t];
    if (pos < 0) return;  // (the whole cluster works on one row)
    uint8_t *ring = lat_smem + warp * S::kBufs * S::kTileBytes;
    float *scores = reinterpret_cast<float *>(lat_smem + S::kSmem - S::kScores);  // [2][warp][16][pitch]
    const SplitKeys keys = split_keys(a, pos, split);
    const uint16_t *base = cache + (size_t)a.slots[t] * a.ring * a.kv_stride + warp * kQ;
    const uint32_t ring0 = keys.first % a.ring, n_tiles = (keys.count + kLatKeys - 1) / kLatKeys;
    auto fetch = [&](uint32_t tile) {
        if (tile < n_tiles) {
            uint8_t *dst = ring + (tile % S::kBufs) * S::kTileBytes;
#pragma unroll 8
            for (uint32_t i = lane; i < kLatKeys * (kQ / 8); i += 32) {
                const uint32_t key = i / (kQ / 8), piece = i % (kQ / 8), j = tile * kLatKeys + key;
                uint32_t r = ring0 + j;
                if (r >= a.ring) r -= a.ring;  // (a window is no longer than the ring)
                const bool live = j < keys.count && warp * kQ + piece * 8 < a.kv_stride;
                copy16(dst + (key * S::kPitch + piece * 8) * 2, live ? base + (size_t)r * a.kv_stride + piece * 8 : cache,
                          live ? 16u : 0u);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    // this warp's quarter of the query, as A fragments in two bfloat16 terms
    uint32_t qh[kSteps][4], ql[kSteps][4];
#pragma unroll
    for (int ks = 0; ks < kSteps; ++ks)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const uint32_t r = g + (e & 1) * 8, c = warp * kQ + ks * 16 + 2 * c4 + (e >> 1) * 8;
            float2 v = make_float2(0.f, 0.f);
            if (h0 + r < a.heads && c < a.kv_stride)  // (kv_stride is even)
                v = *reinterpret_cast<const float2 *>(a.absorbed + ((size_t)t * a.heads + h0 + r) * a.kv_stride + c);
            split_bf16(v.x, v.y, qh[ks][e], ql[ks][e]);
        }
    float o[kTilesPerWarp][4];
#pragma unroll
    for (int n = 0; n < kTilesPerWarp; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll 1
    for (uint32_t tile_i = 0; tile_i < n_tiles; ++tile_i) {
        const uint32_t k0 = tile_i * kLatKeys;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncwarp();  // the warp's tile is in place, and it is done with the one before
        fetch(tile_i + 1);
        const uint32_t tile = (uint32_t)__cvta_generic_to_shared(ring + (tile_i % S::kBufs) * S::kTileBytes);
        float s[4][4], s2[4][4];  // (a chain per term)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[n][e] = s2[n][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < kSteps; ++ks)
#pragma unroll
            for (int pr = 0; pr < 2; ++pr) {
                uint32_t b[4];  // two tiles of eight keys x 16 channels
                ldsm4(b, tile + (((2 * pr + (lane >> 4)) * 8 + (lane & 7)) * S::kPitch + ks * 16 +
                                    ((lane >> 3) & 1) * 8) * 2);
                mma16(s[2 * pr], qh[ks], b[0], b[1]);
                mma16(s[2 * pr + 1], qh[ks], b[2], b[3]);
                if constexpr (TERMS == 2) {
                    mma16(s2[2 * pr], ql[ks], b[0], b[1]);
                    mma16(s2[2 * pr + 1], ql[ks], b[2], b[3]);
                }
            }
        float *sc = scores + (tile_i & 1) * 4 * 16 * S::kScorePitch;
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float2 *>(sc + (warp * 16 + g + 8 * r) * S::kScorePitch + n * 8 + 2 * c4) =
                    make_float2(s[n][2 * r] + s2[n][2 * r], s[n][2 * r + 1] + s2[n][2 * r + 1]);
        __syncthreads();  // (the other of the two score buffers is free: every warp is past its reads)
        // every warp forms the weights of all 32 keys for rows g and g + 8
        float v[2][2][4];  // [row][16-key step][2 c4, 2 c4 + 1, 2 c4 + 8, 2 c4 + 9]
        float alpha[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float mx = m[r];
#pragma unroll
            for (int kk = 0; kk < 2; ++kk)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const uint32_t key = kk * 16 + half * 8 + 2 * c4;
                    float2 x = make_float2(0.f, 0.f);
#pragma unroll
                    for (int w = 0; w < 4; ++w) {
                        const float2 y = *reinterpret_cast<const float2 *>(sc + (w * 16 + g + 8 * r) * S::kScorePitch + key);
                        x.x += y.x;
                        x.y += y.y;
                    }
                    v[r][kk][2 * half] = k0 + key < keys.count ? x.x : -INFINITY;
                    v[r][kk][2 * half + 1] = k0 + key + 1 < keys.count ? x.y : -INFINITY;
                    mx = fmaxf(mx, fmaxf(v[r][kk][2 * half], v[r][kk][2 * half + 1]));
                }
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            alpha[r] = m[r] == -INFINITY ? 0.f : expf(m[r] - mx);  // (every tile has a live key: mx is finite)
            m[r] = mx;
            l[r] *= alpha[r];
#pragma unroll
            for (int kk = 0; kk < 2; ++kk)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    v[r][kk][e] = expf(v[r][kk][e] - mx);
                    l[r] += v[r][kk][e];
                }
        }
#pragma unroll
        for (int n = 0; n < kTilesPerWarp; ++n) {
            o[n][0] *= alpha[0];
            o[n][1] *= alpha[0];
            o[n][2] *= alpha[1];
            o[n][3] *= alpha[1];
        }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
            uint32_t ph[4], pl[4];
            split_bf16(v[0][kk][0], v[0][kk][1], ph[0], pl[0]);
            split_bf16(v[1][kk][0], v[1][kk][1], ph[1], pl[1]);
            split_bf16(v[0][kk][2], v[0][kk][3], ph[2], pl[2]);
            split_bf16(v[1][kk][2], v[1][kk][3], ph[3], pl[3]);
#pragma unroll
            for (int n = 0; n < kTilesPerWarp; n += 2) {
                uint32_t b[4];
                ldsm4_trans(b, tile + ((kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * S::kPitch +
                                          (n + (lane >> 4)) * 8) * 2);
                mma16(o[n], ph, b[0], b[1]);
                mma16(o[n + 1], ph, b[2], b[3]);
                if constexpr (TERMS == 2) {
                    mma16(o[n], pl, b[0], b[1]);
                    mma16(o[n + 1], pl, b[2], b[3]);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // The splits of a cluster are merged here: every CTA leaves its sums, maxima and weights in its
    // shared memory (the tiles are idle) and each finishes a share of the channels.
    float *sums = reinterpret_cast<float *>(lat_smem);  // [16][KV + 4]
    constexpr int kSumPitch = KV + 4;
    float *stat = sums + 16 * kSumPitch;                // [2][16]: maximum, weight
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
#pragma unroll
        for (int n = 0; n < kTilesPerWarp; ++n)
            *reinterpret_cast<float2 *>(sums + (g + 8 * r) * kSumPitch + warp * (KV / 4) + n * 8 + 2 * c4) =
                make_float2(o[n][2 * r], o[n][2 * r + 1]);
        if (warp == 0 && c4 == 0) {
            stat[g + 8 * r] = m[r];
            stat[16 + g + 8 * r] = l[r];
        }
    }
    const uint32_t n_cta = cluster, rank = split % n_cta;
    if (n_cta > 1) lat_cluster_sync();
    else __syncthreads();
    const uint32_t share = (KV / 4 + n_cta - 1) / n_cta, p0 = rank * share, p1 = min(p0 + share, (uint32_t)KV / 4);
    for (uint32_t i = threadIdx.x; i < 16 * share; i += 128) {
        const uint32_t r = i / share, piece = p0 + i % share, h = h0 + r;
        if (h >= a.heads || piece >= p1) continue;
        float mc[8], mx = -INFINITY;
#pragma unroll
        for (int p = 0; p < 8; ++p) {
            mc[p] = (uint32_t)p < n_cta ? lat_peer(stat + r, p) : -INFINITY;
            mx = fmaxf(mx, mc[p]);
        }
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        float w = 0.f;
#pragma unroll
        for (int p = 0; p < 8; ++p) {
            if ((uint32_t)p >= n_cta || mc[p] == -INFINITY) continue;
            const float e = expf(mc[p] - mx);
            const float4 x = lat_peer4(sums + r * kSumPitch + piece * 4, p);
            v.x = fmaf(e, x.x, v.x);
            v.y = fmaf(e, x.y, v.y);
            v.z = fmaf(e, x.z, v.z);
            v.w = fmaf(e, x.w, v.w);
            w = fmaf(e, lat_peer(stat + 16 + r, p), w);
        }
        float *dst = a.partial + (((size_t)t * a.heads + h) * (a.n_splits / n_cta) + split / n_cta) * (a.kv_stride + 8);
        if (piece * 4 < a.kv_stride) *reinterpret_cast<float4 *>(dst + piece * 4) = v;
        if (piece == 0) {
            dst[a.kv_stride] = mx;
            dst[a.kv_stride + 1] = w;
        }
    }
    if (n_cta > 1) lat_cluster_sync();  // no CTA leaves while another still reads its shared memory
}

// ------------------------------------------------------------------ absorbed: combine, W_uv
// A block takes kRows rows of one head: the weights are read once for all of them.
constexpr int kOutThreads = 256;
template <typename W, int kRows>
__global__ void __launch_bounds__(kOutThreads)
latent_output_kernel(LatentArgs a, const W *__restrict__ uv, uint32_t per_block) {
    qk::pdl_launch();
    {   // the weights depend on no other kernel: on their way to L2 before the dependency wait
        const uint32_t first = blockIdx.y * per_block, n = min(per_block, a.vdim - min(first, a.vdim));
        const uint8_t *w = reinterpret_cast<const uint8_t *>(uv + ((size_t)blockIdx.x * a.vdim_stride + first) * a.kv_stride);
        for (uint32_t i = threadIdx.x * 128; i < n * a.kv_stride * (uint32_t)sizeof(W); i += kOutThreads * 128)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(w + i));
    }
    qk::pdl_wait();
    extern __shared__ __align__(16) float lo_smem[];  // [kRows][kv_stride] combined latents, [kRows][n_splits] weights
    float *lat = lo_smem, *wt = lo_smem + kRows * a.kv_stride;
    const uint32_t h = blockIdx.x, t0 = blockIdx.z * kRows, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const uint32_t j0 = blockIdx.y * per_block, j1 = min(j0 + per_block, a.vdim), pitch = a.kv_stride + 8;
    // a warp per row forms its splits' weights (and with several rows its combined latent as well)
    for (uint32_t r = warp; r < (uint32_t)kRows; r += kOutThreads / 32) {
        const uint32_t t = t0 + r;
        const bool live = t < a.tokens && a.positions[t] >= 0;  // (an idle row's output is zero)
        const float *src = a.partial + ((size_t)min(t, a.tokens - 1) * a.heads + h) * a.n_splits * pitch;
        float m = -INFINITY, l = 0.f;
        for (uint32_t s = lane; s < a.n_splits && live; s += 32) m = fmaxf(m, src[(size_t)s * pitch + a.kv_stride]);
        for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
        for (uint32_t s = lane; s < a.n_splits; s += 32) {
            const float ms = live ? src[(size_t)s * pitch + a.kv_stride] : -INFINITY;
            const float e = ms == -INFINITY ? 0.f : expf(ms - m);
            wt[r * a.n_splits + s] = e;
            if (e != 0.f) l += e * src[(size_t)s * pitch + a.kv_stride + 1];
        }
        for (int off = 16; off > 0; off >>= 1) l += __shfl_xor_sync(0xffffffffu, l, off);
        for (uint32_t s = lane; s < a.n_splits && live; s += 32) wt[r * a.n_splits + s] /= l;
        __syncwarp();
        if constexpr (kRows > 1)
#pragma unroll 4
            for (uint32_t i = lane * 4; i < a.kv_stride; i += 128) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                for (uint32_t s = 0; s < a.n_splits; ++s) {
                    const float e = wt[r * a.n_splits + s];
                    if (e == 0.f) continue;  // (an empty split holds no sums)
                    const float4 x = *reinterpret_cast<const float4 *>(src + (size_t)s * pitch + i);
                    v = make_float4(fmaf(e, x.x, v.x), fmaf(e, x.y, v.y), fmaf(e, x.z, v.z), fmaf(e, x.w, v.w));
                }
                *reinterpret_cast<float4 *>(lat + r * a.kv_stride + i) = v;
            }
    }
    __syncthreads();
    if constexpr (kRows == 1) {  // one row: the whole block combines it
        const float *src = a.partial + ((size_t)t0 * a.heads + h) * a.n_splits * pitch;
        for (uint32_t i = threadIdx.x; i < a.kv_stride; i += kOutThreads) {
            float v = 0.f;
#pragma unroll 8
            for (uint32_t s = 0; s < a.n_splits; ++s) {
                const float e = wt[s];
                if (e != 0.f) v = fmaf(e, src[(size_t)s * pitch + i], v);
            }
            lat[i] = v;
        }
        __syncthreads();
    }
    for (uint32_t j = j0 + warp; j < j1; j += kOutThreads / 32) {
        const W *row = uv + ((size_t)h * a.vdim_stride + j) * a.kv_stride;
        float v[kRows];
#pragma unroll
        for (int r = 0; r < kRows; ++r) v[r] = 0.f;
#pragma unroll 2
        for (uint32_t i = lane * 8; i < a.kv_stride; i += 256) {
            float w[8];
            lt_load8(row + i, w);
#pragma unroll
            for (int r = 0; r < kRows; ++r) {
                const float4 x = *reinterpret_cast<const float4 *>(lat + r * a.kv_stride + i);
                const float4 y = *reinterpret_cast<const float4 *>(lat + r * a.kv_stride + i + 4);
                v[r] = fmaf(w[0], x.x, fmaf(w[1], x.y, fmaf(w[2], x.z, fmaf(w[3], x.w, v[r]))));
                v[r] = fmaf(w[4], y.x, fmaf(w[5], y.y, fmaf(w[6], y.z, fmaf(w[7], y.w, v[r]))));
            }
        }
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            for (int off = 16; off > 0; off >>= 1) v[r] += __shfl_xor_sync(0xffffffffu, v[r], off);
            if (lane == 0 && t0 + r < a.tokens)
                put(a.out, a.out_bf16, (size_t)(t0 + r) * a.out_stride + h * a.vdim + j, v[r]);
        }
    }
}

// The same for 16 rows of one head on the tensor cores (bfloat16 weights): the combined latents, in
// two bfloat16 terms, are the M side, the value channels the N side, 16 per warp.
template <int TERMS>
__global__ void __launch_bounds__(kOutThreads)
latent_output_mma_kernel(LatentArgs a, const uint16_t *__restrict__ uv) {
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) uint8_t om_smem[];  // [TERMS][16][kv_stride + 8] bfloat16
    uint16_t *lat = reinterpret_cast<uint16_t *>(om_smem);
    const uint32_t h = blockIdx.x, t0 = blockIdx.y * 16, warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const uint32_t g = lane >> 2, c4 = lane & 3, lp = a.kv_stride + 8, pitch = a.kv_stride + 8;
    for (uint32_t r = warp; r < 16; r += kOutThreads / 32) {
        const uint32_t t = t0 + r;
        const bool live = t < a.tokens && a.positions[t] >= 0;  // (an idle row's output is zero)
        const float *src = a.partial + ((size_t)min(t, a.tokens - 1) * a.heads + h) * a.n_splits * pitch;
        float m = -INFINITY, l = 0.f;
        for (uint32_t s = 0; s < a.n_splits && live; ++s) m = fmaxf(m, src[(size_t)s * pitch + a.kv_stride]);
        for (uint32_t s = 0; s < a.n_splits && live; ++s) {
            const float ms = src[(size_t)s * pitch + a.kv_stride];
            if (ms != -INFINITY) l += expf(ms - m) * src[(size_t)s * pitch + a.kv_stride + 1];
        }
        for (uint32_t i = lane * 2; i < a.kv_stride; i += 64) {
            float x = 0.f, y = 0.f;
            for (uint32_t s = 0; s < a.n_splits && live; ++s) {
                const float ms = src[(size_t)s * pitch + a.kv_stride];
                if (ms == -INFINITY) continue;  // (an empty split holds no sums)
                const float e = expf(ms - m) / l;
                const float2 v = *reinterpret_cast<const float2 *>(src + (size_t)s * pitch + i);
                x = fmaf(e, v.x, x);
                y = fmaf(e, v.y, y);
            }
            uint32_t hi, lo;
            split_bf16(x, y, hi, lo);
            *reinterpret_cast<uint32_t *>(lat + r * lp + i) = hi;
            if constexpr (TERMS == 2) *reinterpret_cast<uint32_t *>(lat + (16 + r) * lp + i) = lo;
        }
    }
    __syncthreads();
    const uint32_t a_addr = (uint32_t)__cvta_generic_to_shared(lat + ((lane & 7) + ((lane >> 3) & 1) * 8) * lp + (lane >> 4) * 8);
    for (uint32_t j0 = warp * 16; j0 < a.vdim; j0 += kOutThreads / 32 * 16) {
        const uint32_t *row[2];
#pragma unroll
        for (int n = 0; n < 2; ++n)
            row[n] = reinterpret_cast<const uint32_t *>(
                uv + ((size_t)h * a.vdim_stride + min(j0 + n * 8 + g, a.vdim_stride - 1)) * a.kv_stride) + c4;
        float acc[2][4] = {};
#pragma unroll 8
        for (uint32_t k = 0; k < a.kv_stride; k += 16) {  // (kv_stride is a multiple of 16 here)
            uint32_t x[4], y[4];
            ldsm4(x, a_addr + k * 2);
            if constexpr (TERMS == 2) ldsm4(y, a_addr + (16 * lp + k) * 2);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t b0 = row[n][k / 2], b1 = row[n][k / 2 + 4];
                mma16(acc[n], x, b0, b1);
                if constexpr (TERMS == 2) mma16(acc[n], y, b0, b1);
            }
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t t = t0 + g + (e >> 1) * 8, j = j0 + n * 8 + 2 * c4 + (e & 1);
                if (t < a.tokens && j < a.vdim) put(a.out, a.out_bf16, (size_t)t * a.out_stride + h * a.vdim + j, acc[n][e]);
            }
    }
}

// ------------------------------------------------------------------ ring -> consecutive rows
__global__ void __launch_bounds__(128)
latent_gather_kernel(const uint4 *__restrict__ cache, uint32_t ring, uint32_t pieces, uint32_t slot, uint32_t first,
                     uint4 *__restrict__ out) {
    qk::pdl_launch();
    qk::pdl_wait();
    const uint4 *src = cache + ((size_t)slot * ring + (first + blockIdx.x) % ring) * pieces;
    for (uint32_t i = threadIdx.x; i < pieces; i += 128) out[(size_t)blockIdx.x * pieces + i] = src[i];
}

// ------------------------------------------------------------------ expanded: band of keys
// Four warps, 16 query rows each, one head; tiles of 64 keys, double-buffered.  Row i (position
// p0 + i) sees keys j with 0 <= p0 + i - j < window.
struct BandArgs {
    const uint16_t *q, *kv;
    uint16_t *out;
    uint32_t q_stride, kv_row, key0, n_keys, p0, tokens, heads, dim_stride, vdim, vdim_stride, window, out_stride;
    float scale_log2;
};
constexpr int kBandQ = 64, kBandK = 64;
template <int DK, int DV> struct BandShape {
    static constexpr int kKPitch = DK + 8, kVPitch = DV + 8;
    static constexpr size_t kQBytes = kBandQ * kKPitch * 2, kKBytes = kBandK * kKPitch * 2, kVBytes = kBandK * kVPitch * 2;
    static constexpr size_t kSmem = kQBytes + 2 * (kKBytes + kVBytes);
};
template <int DK, int DV>
__global__ void __launch_bounds__(128)
window_attention_kernel(BandArgs a) {
    using S = BandShape<DK, DV>;
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) uint8_t band_smem[];
    uint8_t *qs = band_smem, *kvs = band_smem + S::kQBytes;
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane >> 2, c4 = lane & 3;
    const uint32_t h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * kBandQ;  // (late rows see most keys)
    const uint32_t q_last = min(q0 + kBandQ, a.tokens) - 1;
    const uint32_t lo = a.p0 + q0 + 1 > a.window ? a.p0 + q0 + 1 - a.window : 0, hi = a.p0 + q_last;  // positions
    const uint32_t first = lo - a.key0, n = hi - lo + 1, n_tiles = (n + kBandK - 1) / kBandK;
    auto fetch = [&](uint32_t jt, uint32_t buf) {
        uint8_t *kt = kvs + buf * (S::kKBytes + S::kVBytes), *vt = kt + S::kKBytes;
        const uint32_t r0 = first + jt * kBandK;
        for (uint32_t i = threadIdx.x; i < kBandK * (DK / 8); i += 128) {
            const uint32_t key = i / (DK / 8), piece = i % (DK / 8);
            const bool live = r0 + key < a.n_keys && piece * 8 < a.dim_stride;
            copy16(kt + (key * S::kKPitch + piece * 8) * 2,
                      a.kv + (live ? (size_t)(r0 + key) * a.kv_row + h * a.dim_stride + piece * 8 : 0), live ? 16u : 0u);
        }
        for (uint32_t i = threadIdx.x; i < kBandK * (DV / 8); i += 128) {
            const uint32_t key = i / (DV / 8), piece = i % (DV / 8);
            const bool live = r0 + key < a.n_keys && piece * 8 < a.vdim_stride;
            copy16(vt + (key * S::kVPitch + piece * 8) * 2,
                      a.kv + (live ? (size_t)(r0 + key) * a.kv_row + a.heads * a.dim_stride + h * a.vdim_stride + piece * 8
                                   : 0),
                      live ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (uint32_t i = threadIdx.x; i < kBandQ * (DK / 8); i += 128) {
        const uint32_t r = i / (DK / 8), piece = i % (DK / 8);
        const bool live = q0 + r < a.tokens && piece * 8 < a.dim_stride;
        copy16(qs + (r * S::kKPitch + piece * 8) * 2,
                  a.q + (live ? (size_t)(q0 + r) * a.q_stride + h * a.dim_stride + piece * 8 : 0), live ? 16u : 0u);
    }
    fetch(0, 0);
    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const uint32_t row0 = q0 + warp * 16;                      // this warp's rows: positions p0 + row0 ..
    const int pos_g = (int)(a.p0 + row0 + g);
    const int warp_lo = (int)(a.p0 + row0) - (int)a.window + 1, warp_hi = (int)(a.p0 + row0) + 15;
    const uint32_t q_addr = (uint32_t)__cvta_generic_to_shared(qs) +
                            ((warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::kKPitch + (lane >> 4) * 8) * 2;
    uint32_t qf[DK <= 128 ? DK / 16 : 1][4];
    for (uint32_t jt = 0; jt < n_tiles; ++jt) {
        const uint32_t buf = jt & 1;
        if (jt + 1 < n_tiles) {
            fetch(jt + 1, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if constexpr (DK <= 128) {
            if (jt == 0) {
#pragma unroll
                for (int ks = 0; ks < DK / 16; ++ks) ldsm4(qf[ks], q_addr + ks * 32);
            }
        }
        const int j0 = (int)(lo + jt * kBandK);
        if (row0 < a.tokens && j0 <= warp_hi && j0 + kBandK > warp_lo) {
            const uint32_t kt = (uint32_t)__cvta_generic_to_shared(kvs + buf * (S::kKBytes + S::kVBytes));
            const uint32_t vt = kt + (uint32_t)S::kKBytes;
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DK / 16; ++ks) {
                uint32_t qa[4];
                if constexpr (DK > 128) ldsm4(qa, q_addr + ks * 32);
#pragma unroll
                for (int pr = 0; pr < 4; ++pr) {
                    uint32_t b[4];
                    ldsm4(b, kt + (((2 * pr + (lane >> 4)) * 8 + (lane & 7)) * S::kKPitch + ks * 16 +
                                      ((lane >> 3) & 1) * 8) * 2);
                    if constexpr (DK > 128) {
                        mma16(s[2 * pr], qa, b[0], b[1]);
                        mma16(s[2 * pr + 1], qa, b[2], b[3]);
                    } else {
                        mma16(s[2 * pr], qf[ks], b[0], b[1]);
                        mma16(s[2 * pr + 1], qf[ks], b[2], b[3]);
                    }
                }
            }
            // a tile inside every row's band needs no mask
            const bool whole = j0 + kBandK - 1 <= (int)(a.p0 + row0) && j0 >= warp_hi - (int)a.window + 1;
            if (!whole) {
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int back = pos_g + (e >> 1) * 8 - (j0 + 8 * i + 2 * (int)c4 + (e & 1));
                        if (back < 0 || back >= (int)a.window) s[i][e] = -INFINITY;
                    }
            }
            float alpha[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float mx = m[r];
#pragma unroll
                for (int i = 0; i < 8; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * r], s[i][2 * r + 1]));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float ref = mx == -INFINITY ? 0.f : mx;
                alpha[r] = exp2f((m[r] - ref) * a.scale_log2);  // (m = -inf: 0)
                m[r] = mx;
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    s[i][2 * r] = exp2f((s[i][2 * r] - ref) * a.scale_log2);
                    s[i][2 * r + 1] = exp2f((s[i][2 * r + 1] - ref) * a.scale_log2);
                    sum += s[i][2 * r] + s[i][2 * r + 1];
                }
                l[r] = l[r] * alpha[r] + sum;
            }
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) {
                o[i][0] *= alpha[0];
                o[i][1] *= alpha[0];
                o[i][2] *= alpha[1];
                o[i][3] *= alpha[1];
            }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                const uint32_t p[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                       pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]),
                                       pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                for (int i = 0; i < DV / 8; i += 2) {
                    uint32_t b[4];
                    ldsm4_trans(b, vt + ((kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * S::kVPitch +
                                            (i + (lane >> 4)) * 8) * 2);
                    mma16(o[i], p, b[0], b[1]);
                    mma16(o[i + 1], p, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const uint32_t t = row0 + g + 8 * r;
        if (t >= a.tokens) continue;
        const float inv = 1.0f / l[r];
        uint16_t *dst = a.out + (size_t)t * a.out_stride + h * a.vdim;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
            const uint32_t c = i * 8 + 2 * c4;
            if (c < a.vdim) dst[c] = float_to_bf16_bits(o[i][2 * r] * inv);
            if (c + 1 < a.vdim) dst[c + 1] = float_to_bf16_bits(o[i][2 * r + 1] * inv);
        }
    }
}

qk_status enter(qk_ctx *ctx, qk_ctx **c) {
    qk_status st = qk::resolve_ctx(ctx, c);
    if (st != QK_OK) return st;
    QK_CUDA(cudaSetDevice((*c)->device));
    return QK_OK;
}
// With many rows a kernel is launched only when the one before it has finished: blocks that come in
// early crowd on the SMs that have room at that moment, and stay there.
constexpr uint32_t kFewRows = 8, kManyRows = 16;
#define QK_LAUNCH(c, kernel, grid, block, smem, ...)                                                   \
    do {                                                                                               \
        (void)qk::launch_pdl((c)->pdl && a.tokens <= kFewRows, kernel, grid, block, smem, (c)->stream, __VA_ARGS__);           \
        QK_CUDA(cudaGetLastError());                                                                   \
        (c)->launches++;                                                                               \
    } while (0)

template <int KV, int TERMS>
qk_status launch_mma_terms(qk_ctx *c, const LatentArgs &a, const uint16_t *cache, uint32_t cluster) {
    QK_CUDA(cudaFuncSetAttribute((latent_mma_kernel<KV, TERMS>), cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)LatShape<KV>::kSmem));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.n_splits, (a.heads + 15) / 16, a.tokens);
    cfg.blockDim = dim3(128);
    cfg.dynamicSmemBytes = LatShape<KV>::kSmem;
    cfg.stream = c->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = c->pdl && a.tokens <= kFewRows ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    QK_CUDA(cudaLaunchKernelEx(&cfg, (latent_mma_kernel<KV, TERMS>), a, cache, cluster));
    c->launches++;
    return QK_OK;
}

template <int KV>
qk_status launch_mma(qk_ctx *c, const LatentArgs &a, const uint16_t *cache, uint32_t cluster) {
    return a.tokens < kManyRows ? launch_mma_terms<KV, 2>(c, a, cache, cluster) : launch_mma_terms<KV, 1>(c, a, cache, cluster);
}

template <int DK, int DV>
qk_status launch_band(qk_ctx *c, const BandArgs &a) {
    using S = BandShape<DK, DV>;
    QK_CUDA(cudaFuncSetAttribute(window_attention_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)S::kSmem));
    QK_LAUNCH(c, (window_attention_kernel<DK, DV>), dim3((a.tokens + kBandQ - 1) / kBandQ, a.heads), dim3(128), S::kSmem, a);
    return QK_OK;
}

}  // namespace

extern "C" {

size_t qk_latent_scratch(size_t tokens, size_t heads, size_t kv_stride, size_t n_splits) {
    return tokens * heads * (kv_stride + n_splits * (kv_stride + 8)) * sizeof(float);
}

qk_status qk_latent_attention(qk_ctx *ctx, const qk_latent_call *d) {
    qk_ctx *c;
    qk_status st = enter(ctx, &c);
    if (st != QK_OK) return st;
    if (!d || !d->q || !d->uk || !d->uv || !d->cache || !d->scratch || !d->out || !d->positions || !d->slots)
        return qk::fail(QK_ERR_VALUE, "qk_latent_attention: null argument");
    if (d->heads == 0 || d->window == 0 || d->ring < d->window || d->n_splits == 0 || d->kv_stride % 8 ||
        d->kv_rank > d->kv_stride || d->dim > d->dim_stride || d->vdim > d->vdim_stride)
        return qk::fail(QK_ERR_VALUE, "qk_latent_attention: heads %zu, window %zu in a ring of %zu, latent %zu (stride %zu)",
                        d->heads, d->window, d->ring, d->kv_rank, d->kv_stride);
    if (d->q_dtype != QK_F32) return qk::fail(QK_ERR_VALUE, "qk_latent_attention: the queries must be float32");
    if (d->w_dtype != QK_F32 && d->w_dtype != QK_BF16)
        return qk::fail(QK_ERR_VALUE, "qk_latent_attention: weight dtype must be float32 or bfloat16, got tag %d", d->w_dtype);
    if (d->kv_stride * 8 > 200 * 1024 || d->n_splits > 1024)
        return qk::fail(QK_ERR_VALUE, "qk_latent_attention: a latent of %zu entries does not fit shared memory", d->kv_stride);
    if (d->tokens == 0) return QK_OK;
    if (d->tokens > 65535) return qk::fail(QK_ERR_VALUE, "qk_latent_attention: at most 65535 rows, got %zu", d->tokens);
    LatentArgs a{};
    a.positions = d->positions;
    a.slots = d->slots;
    a.q = (const float *)d->q;
    a.absorbed = d->scratch;
    a.partial = d->scratch + d->tokens * d->heads * d->kv_stride;
    a.out = d->out;
    a.tokens = (uint32_t)d->tokens;
    a.heads = (uint32_t)d->heads;
    a.dim = (uint32_t)d->dim;
    a.dim_stride = (uint32_t)d->dim_stride;
    a.vdim = (uint32_t)d->vdim;
    a.vdim_stride = (uint32_t)d->vdim_stride;
    a.kv_stride = (uint32_t)d->kv_stride;
    a.window = (uint32_t)d->window;
    a.ring = (uint32_t)d->ring;
    a.n_splits = (uint32_t)d->n_splits;
    a.q_stride = (uint32_t)d->q_stride;
    a.out_stride = (uint32_t)d->out_stride;
    a.scale = d->scale;
    a.out_bf16 = d->out_dtype == QK_BF16;
    const bool bf16 = d->w_dtype == QK_BF16;
    const dim3 ag((unsigned)qk::ceil_div(d->kv_stride, 256), (unsigned)d->heads, (unsigned)qk::ceil_div(d->tokens, kAbsRows));
    const size_t ab_smem = (kAbsRows * d->dim + kAbsWarps * 256) * 4;
    if (ab_smem > 48 * 1024) return qk::fail(QK_ERR_VALUE, "qk_latent_attention: dim %zu does not fit shared memory", d->dim);
    if (bf16) QK_LAUNCH(c, absorb_query_kernel<uint16_t>, ag, dim3(kAbsWarps * 32), ab_smem, a, (const uint16_t *)d->uk);
    else QK_LAUNCH(c, absorb_query_kernel<float>, ag, dim3(kAbsWarps * 32), ab_smem, a, (const float *)d->uk);
    if (bf16 && d->kv_stride <= 512 && c->decode_attention_kernel != 0) {
        const uint16_t *cache = (const uint16_t *)d->cache;
        const uint32_t cluster = a.n_splits % 8 == 0 ? 8 : a.n_splits % 4 == 0 ? 4 : a.n_splits % 2 == 0 ? 2 : 1;
        if (d->kv_stride <= 64) st = launch_mma<64>(c, a, cache, cluster);
        else if (d->kv_stride <= 128) st = launch_mma<128>(c, a, cache, cluster);
        else if (d->kv_stride <= 256) st = launch_mma<256>(c, a, cache, cluster);
        else st = launch_mma<512>(c, a, cache, cluster);
        if (st != QK_OK) return st;
        a.n_splits /= cluster;  // (what is left for the last launch to combine)
    } else {
        const dim3 pg(a.n_splits, a.heads, a.tokens);
        const size_t smem = d->kv_stride * 8;
        if (bf16) {
            QK_CUDA(cudaFuncSetAttribute(latent_plain_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
            QK_LAUNCH(c, latent_plain_kernel<uint16_t>, pg, dim3(kPlainThreads), smem, a, (const uint16_t *)d->cache);
        } else {
            QK_CUDA(cudaFuncSetAttribute(latent_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
            QK_LAUNCH(c, latent_plain_kernel<float>, pg, dim3(kPlainThreads), smem, a, (const float *)d->cache);
        }
    }
    // few rows: several blocks share the value channels of a head; many: a block takes eight rows
    const bool tiled = d->tokens >= 16;
    const uint32_t parts = d->tokens * d->heads >= 256 ? 1u : (uint32_t)std::min<size_t>(4, qk::ceil_div(d->vdim, 16));
    const uint32_t per = (uint32_t)qk::ceil_div(d->vdim, parts), rows = tiled ? 8 : 1;
    const dim3 og(a.heads, parts, (a.tokens + rows - 1) / rows);
    const size_t smem = rows * (d->kv_stride + a.n_splits) * 4;
    if (smem > 200 * 1024)
        return qk::fail(QK_ERR_VALUE, "qk_latent_attention: a latent of %zu entries does not fit shared memory", d->kv_stride);
#define QK_LATENT_OUT(W, R)                                                                                                 \
    do {                                                                                                                    \
        QK_CUDA(cudaFuncSetAttribute(latent_output_kernel<W, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); \
        QK_LAUNCH(c, (latent_output_kernel<W, R>), og, dim3(kOutThreads), smem, a, (const W *)d->uv, per);                  \
    } while (0)
    const size_t mma_smem = 2 * 16 * (d->kv_stride + 8) * 2;
    if (bf16 && tiled && d->kv_stride % 16 == 0 && mma_smem <= 200 * 1024 && c->decode_attention_kernel != 0) {
        QK_CUDA(cudaFuncSetAttribute(latent_output_mma_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        QK_LAUNCH(c, latent_output_mma_kernel<2>, dim3(a.heads, (a.tokens + 15) / 16), dim3(kOutThreads), mma_smem, a,
                  (const uint16_t *)d->uv);
    } else if (bf16 && tiled) QK_LATENT_OUT(uint16_t, 8);
    else if (bf16) QK_LATENT_OUT(uint16_t, 1);
    else if (tiled) QK_LATENT_OUT(float, 8);
    else QK_LATENT_OUT(float, 1);
#undef QK_LATENT_OUT
    return QK_OK;
}

qk_status qk_latent_gather(qk_ctx *ctx, const void *cache, int32_t dtype, size_t ring, size_t stride, size_t slot,
                           size_t first, size_t count, void *out) {
    qk_ctx *c;
    qk_status st = enter(ctx, &c);
    if (st != QK_OK) return st;
    const size_t bytes = stride * (dtype == QK_BF16 ? 2 : 4);
    if (!cache || !out || bytes % 16 || count > ring)
        return qk::fail(QK_ERR_VALUE, "qk_latent_gather: %zu rows of %zu bytes from a ring of %zu", count, bytes, ring);
    if (count == 0) return QK_OK;
    const struct { uint32_t tokens; } a{(uint32_t)count};
    QK_LAUNCH(c, latent_gather_kernel, dim3((unsigned)count), dim3(128), 0, (const uint4 *)cache, (uint32_t)ring,
              (uint32_t)(bytes / 16), (uint32_t)slot, (uint32_t)first, (uint4 *)out);
    return QK_OK;
}

qk_status qk_window_attention(qk_ctx *ctx, const void *q, size_t q_stride, const void *kv, size_t kv_row, size_t key0,
                              size_t n_keys, size_t first_position, size_t tokens, size_t heads, size_t dim_stride,
                              size_t vdim, size_t vdim_stride, size_t window, float scale, void *out, size_t out_stride) {
    qk_ctx *c;
    qk_status st = enter(ctx, &c);
    if (st != QK_OK) return st;
    if (!q || !kv || !out || heads == 0 || window == 0 || vdim > vdim_stride || dim_stride % 8 || vdim_stride % 8 ||
        q_stride % 8 || kv_row % 8)
        return qk::fail(QK_ERR_VALUE, "qk_window_attention: bad arguments");
    if (dim_stride > 256 || vdim_stride > 256)
        return qk::fail(QK_ERR_VALUE, "qk_window_attention: head sizes above 256 are not supported, got %zu and %zu",
                        dim_stride, vdim_stride);
    if (tokens == 0) return QK_OK;
    const size_t lo = first_position + 1 > window ? first_position + 1 - window : 0;
    if (key0 > lo || key0 + n_keys < first_position + tokens)
        return qk::fail(QK_ERR_VALUE, "qk_window_attention: keys %zu..%zu do not cover the windows of positions %zu..%zu",
                        key0, key0 + n_keys - 1, first_position, first_position + tokens - 1);
    BandArgs a{};
    a.q = (const uint16_t *)q;
    a.kv = (const uint16_t *)kv;
    a.out = (uint16_t *)out;
    a.q_stride = (uint32_t)q_stride;
    a.kv_row = (uint32_t)kv_row;
    a.key0 = (uint32_t)key0;
    a.n_keys = (uint32_t)n_keys;
    a.p0 = (uint32_t)first_position;
    a.tokens = (uint32_t)tokens;
    a.heads = (uint32_t)heads;
    a.dim_stride = (uint32_t)dim_stride;
    a.vdim = (uint32_t)vdim;
    a.vdim_stride = (uint32_t)vdim_stride;
    a.window = (uint32_t)std::min<size_t>(window, 1u << 30);
    a.out_stride = (uint32_t)out_stride;
    a.scale_log2 = scale * 1.4426950408889634f;
#define QK_BAND_V(DK)                                        \
    (vdim_stride <= 32 ? launch_band<DK, 32>(c, a)           \
     : vdim_stride <= 64 ? launch_band<DK, 64>(c, a)         \
     : vdim_stride <= 128 ? launch_band<DK, 128>(c, a)       \
                          : launch_band<DK, 256>(c, a))
    if (dim_stride <= 32) return QK_BAND_V(32);
    if (dim_stride <= 64) return QK_BAND_V(64);
    if (dim_stride <= 128) return QK_BAND_V(128);
    return QK_BAND_V(256);
#undef QK_BAND_V
}

}  // extern "C"
