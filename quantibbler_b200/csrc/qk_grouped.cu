// Causal attention with grouped heads over a full key/value cache: a query temperature that grows
// with the position and a learned bias per head and distance.
//   * append: a row's keys and values into its slot's cache;
//   * rows (bfloat16): any mix of rows, a few each of many sequences; the keys of a row are split over
//     blocks, whose results the last one to finish combines.  mma.sync with up to eight query heads of
//     one key/value head as rows 0-7 and their second bfloat16 terms as rows 8-15, so that the
//     queries and the softmax weights keep 16 bits of mantissa at no extra product.  A decode step's
//     rows append their own key and value here;
//   * portion (bfloat16): consecutive rows of one sequence.  Head sizes of 64 to 128 on tcgen05, two
//     tiles of 128 rows per CTA that share their keys and values; others on mma.sync, 64 rows per block;
//   * plain: float32, and head sizes the others do not take.
// The bias of a distance is looked up in a table per head that ends where the bias stops changing;
// key tiles that lie wholly beyond it need no lookup.
#include <cuda.h>  // CUtensorMap types only; the encoder is fetched through the runtime

#include <algorithm>

#include "qk_dense_dev.cuh"
#include "qk_mma.cuh"
#include "qk_tma.cuh"
#include "qk_umma.cuh"

namespace {

constexpr float kLog2E = 1.4426950408889634f;

struct GroupedArgs {
    const int32_t *positions, *slots;
    const void *proj;
    const float *bias;
    void *cache_k, *cache_v, *out;
    float *partial;      // [tokens][heads][n_splits][vdim_stride + 8]: sums, then maximum and weight
    uint32_t *tickets;   // [tokens][heads], zero between calls
    int *error;
    uint32_t tokens, heads, kv_heads, dim, vdim, s_max, n_slots, proj_stride, out_stride, n_splits, bias_len, slot, p0;
    float scale, temp_coef;
    double temp_every;
    int append, out_bf16;
};
// dim and vdim are strides: multiples of 16 with zeros behind the entries.

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float query_scale(const GroupedArgs &a, int pos) {
    if (a.temp_every == 0.0) return a.scale;
    const float steps = (float)floor((double)(pos + 1) / a.temp_every);
    return a.scale * (1.0f + a.temp_coef * logf(steps + 1.0f));
}
// The row's position if it is a live row of a cached sequence, else -1.
__device__ __forceinline__ int live_position(const GroupedArgs &a, uint32_t t) {
    const int pos = a.positions[t];
    if (pos < 0) return -1;
    if ((uint32_t)pos >= a.s_max || (uint32_t)a.slots[t] >= a.n_slots) {
        if (threadIdx.x == 0) atomicOr(a.error, 4);
        return -1;
    }
    return pos;
}

__device__ __forceinline__ void load_piece(const float *p, float (&v)[4]) {
    const float4 x = *reinterpret_cast<const float4 *>(p);
    v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
__device__ __forceinline__ void load_piece(const uint16_t *p, float (&v)[4]) {
    const uint2 x = *reinterpret_cast<const uint2 *>(p);
    v[0] = __uint_as_float(x.x << 16), v[1] = __uint_as_float(x.x & 0xffff0000u);
    v[2] = __uint_as_float(x.y << 16), v[3] = __uint_as_float(x.y & 0xffff0000u);
}
__device__ __forceinline__ void store_piece(float *p, const float (&v)[4]) {
    *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_piece(uint16_t *p, const float (&v)[4]) {
    *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
}

// ------------------------------------------------------------------ append
template <typename P, typename C>
__global__ void __launch_bounds__(256)
grouped_append_kernel(GroupedArgs a) {
    qk::pdl_launch();
    qk::pdl_wait();
    const uint32_t t = blockIdx.x;
    const int pos = live_position(a, t);
    if (pos < 0) return;
    const P *k = (const P *)a.proj + (size_t)t * a.proj_stride + a.heads * a.dim, *v = k + a.kv_heads * a.dim;
    const size_t first = (size_t)a.slots[t] * a.kv_heads;
    const uint32_t nk = a.kv_heads * a.dim / 4, nv = a.kv_heads * a.vdim / 4;
    for (uint32_t i = threadIdx.x; i < nk + nv; i += 256) {
        const bool is_k = i < nk;
        const uint32_t at = (is_k ? i : i - nk) * 4, size = is_k ? a.dim : a.vdim;
        float x[4];
        load_piece((is_k ? k : v) + at, x);
        store_piece((C *)(is_k ? a.cache_k : a.cache_v) + ((first + at / size) * a.s_max + pos) * size + at % size, x);
    }
}

// ------------------------------------------------------------------ combining splits
// The last block of a row's heads to finish adds up the splits; `n_heads` heads from h0 on, maxima in
// units where the weight of a split is BASE ** (its maximum - the largest).
template <bool kBase2>
__device__ __forceinline__ float weight_of(float d) { return kBase2 ? exp2f(d) : expf(d); }
template <bool kBase2>
__device__ __forceinline__ void combine_splits(const GroupedArgs &a, uint32_t t, uint32_t h0, uint32_t n_heads,
                                               uint32_t n_active) {
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, pitch = a.vdim + 8;
    for (uint32_t h = h0 + warp; h < h0 + n_heads; h += blockDim.x / 32) {
        const float *src = a.partial + ((size_t)t * a.heads + h) * a.n_splits * pitch;
        float m = -INFINITY;
        for (uint32_t s = lane; s < n_active; s += 32) m = fmaxf(m, __ldcg(src + (size_t)s * pitch + a.vdim));
        for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
        float l = 0.f;
        for (uint32_t s = lane; s < n_active; s += 32)
            l += weight_of<kBase2>(__ldcg(src + (size_t)s * pitch + a.vdim) - m) * __ldcg(src + (size_t)s * pitch + a.vdim + 1);
        for (int off = 16; off > 0; off >>= 1) l += __shfl_xor_sync(0xffffffffu, l, off);
        const float inv = 1.0f / l;
        for (uint32_t c = lane * 4; c < a.vdim; c += 128) {
            float o[4] = {};
#pragma unroll 4
            for (uint32_t s = 0; s < n_active; ++s) {
                const float e = weight_of<kBase2>(__ldcg(src + (size_t)s * pitch + a.vdim) - m);
                const float4 x = __ldcg(reinterpret_cast<const float4 *>(src + (size_t)s * pitch + c));
                o[0] = fmaf(e, x.x, o[0]);
                o[1] = fmaf(e, x.y, o[1]);
                o[2] = fmaf(e, x.z, o[2]);
                o[3] = fmaf(e, x.w, o[3]);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) o[i] *= inv;
            const size_t at = (size_t)t * a.out_stride + h * a.vdim + c;
            if (a.out_bf16) store_piece((uint16_t *)a.out + at, o);
            else store_piece((float *)a.out + at, o);
        }
    }
}
// True in every thread of the block that finishes last of n_active; the counter is zero again then.
__device__ __forceinline__ bool last_to_finish(uint32_t *ticket, uint32_t n_active) {
    __shared__ bool is_last;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        is_last = atomicAdd(ticket, 1u) == n_active - 1;
        if (is_last) *ticket = 0;
    }
    __syncthreads();
    if (is_last) __threadfence();
    return is_last;
}

// ------------------------------------------------------------------ rows, bfloat16
template <int DM> struct RowShape {
    static constexpr int kKeys = DM <= 64 ? 32 : 16, kBufs = DM <= 128 ? 3 : 2, kPitch = DM + 8;
    static constexpr size_t kTile = 2 * kKeys * kPitch * 2;  // keys, then values
    static constexpr size_t kRing = 4 * kBufs * kTile;
    static constexpr size_t kSums = 4 * (8 * (DM + 4) + 16) * 4;
    static constexpr size_t kSmem = kRing > kSums ? kRing : kSums;
};
// Grid (splits, key/value heads x groups of eight query heads, rows); four warps, each with key tiles of
// its own.  FULL: both head strides are DM.
template <int DM, bool FULL>
__global__ void __launch_bounds__(128)
grouped_rows_kernel(const __grid_constant__ GroupedArgs a) {
    using S = RowShape<DM>;
    constexpr int kSteps = DM / 16, kKeyTiles = S::kKeys / 8;
    const uint32_t dim = FULL ? (uint32_t)DM : a.dim, vdim = FULL ? (uint32_t)DM : a.vdim;
    qk::pdl_launch();
    extern __shared__ __align__(16) uint8_t row_smem[];
    const uint32_t t = blockIdx.z, warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane >> 2, c4 = lane & 3;
    const uint32_t group = a.heads / a.kv_heads, subs = (group + 7) / 8, kvh = blockIdx.y / subs, sub = blockIdx.y % subs;
    const uint32_t h0 = kvh * group + sub * 8, n_heads = min(8u, group - sub * 8);
    // Positions and slots are written by copies and ordinary launches in front of the step, none of
    // which lets a kernel start early; so are the cached rows of earlier steps.
    if (!a.append) qk::pdl_wait();
    const int pos = live_position(a, t);
    const uint32_t n_keys = (uint32_t)(pos + 1);
    const uint32_t per = max(4u * S::kKeys, ((n_keys + a.n_splits - 1) / a.n_splits + S::kKeys - 1) / S::kKeys * S::kKeys);
    const uint32_t first = blockIdx.x * per;
    if (pos < 0 || first >= n_keys) {
        if (a.append) qk::pdl_wait();
        return;
    }
    const uint32_t n_active = (n_keys + per - 1) / per, count = min(per, n_keys - first);
    const uint32_t cached = a.append ? n_keys - 1 - first : count;  // (the newest key is not in the cache yet)
    const uint32_t n_tiles = (count + S::kKeys - 1) / S::kKeys;
    const size_t head_row = ((size_t)a.slots[t] * a.kv_heads + kvh) * a.s_max;
    const uint16_t *kb = (const uint16_t *)a.cache_k + (head_row + first) * dim;
    const uint16_t *vb = (const uint16_t *)a.cache_v + (head_row + first) * vdim;
    uint8_t *ring = row_smem + warp * S::kBufs * S::kTile;
    // a lane copies one column piece of every kStride-th key
    constexpr uint32_t kPieces = DM / 8, kStride = 32 / kPieces ? 32 / kPieces : 1;
    const uint32_t piece = lane % kPieces * 8, key0 = lane / kPieces, end = min(cached, count);
    const bool in_k = FULL || piece < dim, in_v = FULL || piece < vdim;
    auto fetch = [&](uint32_t i) {  // this warp's i-th tile
        const uint32_t k0 = (warp + 4 * i) * S::kKeys;
        if (k0 < count) {
            uint8_t *kt = ring + (i % S::kBufs) * S::kTile + (key0 * S::kPitch + piece) * 2;
            const uint16_t *ks = kb + (size_t)(k0 + key0) * dim + piece, *vs = vb + (size_t)(k0 + key0) * vdim + piece;
            if (k0 + S::kKeys <= end) {
#pragma unroll
                for (int x = 0; x < S::kKeys; x += kStride) {
                    if (in_k) copy16(kt + x * S::kPitch * 2, ks + x * dim, 16u);
                    if (in_v) copy16(kt + S::kTile / 2 + x * S::kPitch * 2, vs + x * vdim, 16u);
                }
            } else {
#pragma unroll 1
                for (int x = 0; x < S::kKeys; x += kStride) {
                    const bool live = k0 + key0 + x < end;
                    if (in_k) copy16(kt + x * S::kPitch * 2, live ? ks + x * dim : kb, live ? 16u : 0u);
                    if (in_v) copy16(kt + S::kTile / 2 + x * S::kPitch * 2, live ? vs + x * vdim : vb, live ? 16u : 0u);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i + 1 < S::kBufs; ++i) fetch(i);
    if (a.append) qk::pdl_wait();

    // queries: rows g the high terms, rows g + 8 the low terms of the same head
    const float *proj = (const float *)a.proj + (size_t)t * a.proj_stride;
    uint32_t q[kSteps][4];
#pragma unroll
    for (int ks = 0; ks < kSteps; ++ks)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t c = ks * 16 + 2 * c4 + half * 8;
            float2 v = make_float2(0.f, 0.f);
            if (g < n_heads && c < a.dim) v = *reinterpret_cast<const float2 *>(proj + (h0 + g) * a.dim + c);
            split_bf16(v.x, v.y, q[ks][2 * half], q[ks][2 * half + 1]);
        }
    const float factor = query_scale(a, pos) * kLog2E;
    const float *bias = a.bias ? a.bias + (size_t)min(h0 + g, a.heads - 1) * a.bias_len : nullptr;
    const uint32_t last = a.bias_len - 1;
    const float far = bias ? bias[last] * kLog2E : 0.f;

    float o[DM / 8][4];
#pragma unroll
    for (int n = 0; n < DM / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m = -INFINITY, l = 0.f;
#pragma unroll 1
    for (uint32_t i = 0; warp + 4 * i < n_tiles; ++i) {
        const uint32_t k0 = (warp + 4 * i) * S::kKeys;
        asm volatile("cp.async.wait_group %0;" ::"n"(S::kBufs - 2) : "memory");
        __syncwarp();  // the tile is in place, and the warp is done with the one before
        fetch(i + S::kBufs - 1);
        uint8_t *kt_ptr = ring + (i % S::kBufs) * S::kTile;
        if (a.append && first + count == n_keys && k0 + S::kKeys >= count) {
            // the newest key and value, from the projections, also into the cache
            const float *nk = proj + (a.heads + kvh) * a.dim, *nv = proj + (a.heads + a.kv_heads) * a.dim + kvh * a.vdim;
            uint16_t *ks = reinterpret_cast<uint16_t *>(kt_ptr) + (count - 1 - k0) * S::kPitch;
            uint16_t *vs = reinterpret_cast<uint16_t *>(kt_ptr + S::kTile / 2) + (count - 1 - k0) * S::kPitch;
            for (uint32_t c = lane * 4; c < a.dim; c += 128) {
                float x[4];
                load_piece(nk + c, x);
                store_piece(ks + c, x);
                if (sub == 0) store_piece((uint16_t *)a.cache_k + (head_row + pos) * a.dim + c, x);
            }
            for (uint32_t c = lane * 4; c < a.vdim; c += 128) {
                float x[4];
                load_piece(nv + c, x);
                store_piece(vs + c, x);
                if (sub == 0) store_piece((uint16_t *)a.cache_v + (head_row + pos) * a.vdim + c, x);
            }
            __syncwarp();
        }
        const uint32_t kt = (uint32_t)__cvta_generic_to_shared(kt_ptr), vt = kt + (uint32_t)(S::kTile / 2);
        float s[kKeyTiles][4];
#pragma unroll
        for (int n = 0; n < kKeyTiles; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < kSteps; ++ks) {
            if (ks * 16 >= (int)dim) break;
#pragma unroll
            for (int pr = 0; pr < kKeyTiles / 2; ++pr) {
                uint32_t b[4];
                ldsm4(b, kt + (((2 * pr + (lane >> 4)) * 8 + (lane & 7)) * S::kPitch + ks * 16 + ((lane >> 3) & 1) * 8) * 2);
                mma16(s[2 * pr], q[ks], b[0], b[1]);
                mma16(s[2 * pr + 1], q[ks], b[2], b[3]);
            }
        }
        // scores of head g, keys k0 + 8 n + 2 c4 + e
        const uint32_t back0 = n_keys - 1 - first - k0;  // distance of the tile's first key
        const bool near = bias && back0 + 1 < S::kKeys + last, ragged = k0 + S::kKeys > count;
        float x[kKeyTiles][2], mx = m;
#pragma unroll
        for (int n = 0; n < kKeyTiles; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const uint32_t key = 8 * n + 2 * c4 + e;
                float b = far;
                if (near) b = __ldg(bias + max(min((int)back0 - (int)key, (int)last), 0)) * kLog2E;
                x[n][e] = fmaf(s[n][e] + s[n][e + 2], factor, b);
                if (ragged && k0 + key >= count) x[n][e] = -INFINITY;
                mx = fmaxf(mx, x[n][e]);
            }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));  // (a tile's first key is live: mx is finite)
        if (__any_sync(0xffffffffu, mx > m)) {
            const float alpha = ex2(m - mx);
            m = mx;
            l *= alpha;
#pragma unroll
            for (int n = 0; n < DM / 8; ++n) {
                o[n][0] *= alpha;
                o[n][1] *= alpha;
                o[n][2] *= alpha;
                o[n][3] *= alpha;
            }
        }
#pragma unroll
        for (int n = 0; n < kKeyTiles; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                x[n][e] = ex2(x[n][e] - mx);
                l += x[n][e];
            }
#pragma unroll
        for (int kk = 0; kk < kKeyTiles / 2; ++kk) {
            uint32_t p[4];
            split_bf16(x[2 * kk][0], x[2 * kk][1], p[0], p[1]);
            split_bf16(x[2 * kk + 1][0], x[2 * kk + 1][1], p[2], p[3]);
#pragma unroll
            for (int n = 0; n < DM / 8; n += 2) {
                if (n * 8 >= (int)vdim) break;
                uint32_t b[4];
                ldsm4_trans(b, vt + ((kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * S::kPitch + (n + (lane >> 4)) * 8) * 2);
                mma16(o[n], p, b[0], b[1]);
                mma16(o[n + 1], p, b[2], b[3]);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // the warps' sums together
    constexpr int kSumPitch = DM + 4;
    float *sums = reinterpret_cast<float *>(row_smem), *stat = sums + 4 * 8 * kSumPitch;  // [warp][8]; [warp][2][8]
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
#pragma unroll
    for (int n = 0; n < DM / 8; ++n)
        *reinterpret_cast<float2 *>(sums + (warp * 8 + g) * kSumPitch + n * 8 + 2 * c4) =
            make_float2(o[n][0] + o[n][2], o[n][1] + o[n][3]);
    if (c4 == 0) {
        stat[warp * 16 + g] = m;
        stat[warp * 16 + 8 + g] = l;
    }
    __syncthreads();
    const uint32_t pieces = a.vdim / 4, pitch = a.vdim + 8;
    for (uint32_t i = threadIdx.x; i < n_heads * pieces; i += 128) {
        const uint32_t r = i / pieces, c = i % pieces * 4;
        float mx = -INFINITY, w = 0.f, v[4] = {};
#pragma unroll
        for (int p = 0; p < 4; ++p) mx = fmaxf(mx, stat[p * 16 + r]);
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const float e = exp2f(stat[p * 16 + r] - mx);
            const float4 y = *reinterpret_cast<const float4 *>(sums + (p * 8 + r) * kSumPitch + c);
            w = fmaf(e, stat[p * 16 + 8 + r], w);
            v[0] = fmaf(e, y.x, v[0]);
            v[1] = fmaf(e, y.y, v[1]);
            v[2] = fmaf(e, y.z, v[2]);
            v[3] = fmaf(e, y.w, v[3]);
        }
        if (n_active == 1) {
            const float inv = 1.0f / w;
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] *= inv;
            const size_t at = (size_t)t * a.out_stride + (h0 + r) * a.vdim + c;
            if (a.out_bf16) store_piece((uint16_t *)a.out + at, v);
            else store_piece((float *)a.out + at, v);
        } else {
            float *dst = a.partial + (((size_t)t * a.heads + h0 + r) * a.n_splits + blockIdx.x) * pitch;
            store_piece(dst + c, v);
            if (c == 0) *reinterpret_cast<float2 *>(dst + a.vdim) = make_float2(mx, w);
        }
    }
    if (n_active > 1 && last_to_finish(a.tickets + (size_t)t * a.heads + h0, n_active))
        combine_splits<true>(a, t, h0, n_heads, n_active);
}

// ------------------------------------------------------------------ portion, bfloat16
// Four warps, 16 rows each, one query head; tiles of 64 keys, double-buffered.  Row i is position
// p0 + i of the sequence and sees keys 0 .. p0 + i.
constexpr int kPortQ = 64, kPortK = 64;
template <int DM> struct PortShape {
    static constexpr int kPitch = DM + 8;
    static constexpr size_t kRows = 64 * kPitch * 2, kSmem = 5 * kRows;
};
template <int DM>
__global__ void __launch_bounds__(128)
grouped_portion_kernel(GroupedArgs a) {
    using S = PortShape<DM>;
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) uint8_t port_smem[];
    uint8_t *qs = port_smem, *kvs = port_smem + S::kRows;
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane >> 2, c4 = lane & 3;
    const uint32_t h = blockIdx.y, kvh = h / (a.heads / a.kv_heads);
    const uint32_t q0 = (gridDim.x - 1 - blockIdx.x) * kPortQ;  // (late rows see most keys)
    const uint32_t n_keys = a.p0 + min(q0 + kPortQ, a.tokens), n_tiles = (n_keys + kPortK - 1) / kPortK;
    const size_t head_row = ((size_t)a.slot * a.kv_heads + kvh) * a.s_max;
    const uint16_t *kb = (const uint16_t *)a.cache_k + head_row * a.dim, *vb = (const uint16_t *)a.cache_v + head_row * a.vdim;
    auto fetch = [&](uint32_t jt, uint32_t buf) {
        uint8_t *kt = kvs + buf * 2 * S::kRows, *vt = kt + S::kRows;
        for (uint32_t i = threadIdx.x; i < kPortK * (DM / 8); i += 128) {
            const uint32_t key = i / (DM / 8), c = i % (DM / 8) * 8, j = jt * kPortK + key;
            const bool live = j < n_keys;
            if (c < a.dim) copy16(kt + (key * S::kPitch + c) * 2, live ? kb + (size_t)j * a.dim + c : kb, live ? 16u : 0u);
            if (c < a.vdim) copy16(vt + (key * S::kPitch + c) * 2, live ? vb + (size_t)j * a.vdim + c : vb, live ? 16u : 0u);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const uint16_t *q = (const uint16_t *)a.proj + h * a.dim;
    for (uint32_t i = threadIdx.x; i < kPortQ * (DM / 8); i += 128) {
        const uint32_t r = i / (DM / 8), c = i % (DM / 8) * 8;
        const bool live = q0 + r < a.tokens;
        if (c < a.dim) copy16(qs + (r * S::kPitch + c) * 2, live ? q + (size_t)(q0 + r) * a.proj_stride + c : q, live ? 16u : 0u);
    }
    fetch(0, 0);
    float o[DM / 8][4];
#pragma unroll
    for (int i = 0; i < DM / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const uint32_t row0 = q0 + warp * 16, last = a.bias_len - 1;
    const int pos_g = (int)(a.p0 + row0 + g), warp_first = (int)(a.p0 + row0);
    const float factor[2] = {query_scale(a, pos_g) * kLog2E, query_scale(a, pos_g + 8) * kLog2E};
    const float *bias = a.bias ? a.bias + (size_t)h * a.bias_len : nullptr;
    const float far = bias ? bias[last] * kLog2E : 0.f;
    const uint32_t q_addr = (uint32_t)__cvta_generic_to_shared(qs) +
                            ((warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::kPitch + (lane >> 4) * 8) * 2;
    uint32_t qf[DM <= 128 ? DM / 16 : 1][4];
    for (uint32_t jt = 0; jt < n_tiles; ++jt) {
        const uint32_t buf = jt & 1;
        if (jt + 1 < n_tiles) {
            fetch(jt + 1, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        if constexpr (DM <= 128) {
            if (jt == 0) {
#pragma unroll
                for (int ks = 0; ks < DM / 16; ++ks)
                    if (ks * 16 < (int)a.dim) ldsm4(qf[ks], q_addr + ks * 32);
            }
        }
        const int j0 = (int)(jt * kPortK);
        if (row0 < a.tokens && j0 <= warp_first + 15) {
            const uint32_t kt = (uint32_t)__cvta_generic_to_shared(kvs + buf * 2 * S::kRows), vt = kt + (uint32_t)S::kRows;
            float s[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DM / 16; ++ks) {
                if (ks * 16 >= (int)a.dim) break;
                uint32_t qa[4];
                if constexpr (DM > 128) ldsm4(qa, q_addr + ks * 32);
#pragma unroll
                for (int pr = 0; pr < 4; ++pr) {
                    uint32_t b[4];
                    ldsm4(b, kt + (((2 * pr + (lane >> 4)) * 8 + (lane & 7)) * S::kPitch + ks * 16 + ((lane >> 3) & 1) * 8) * 2);
                    if constexpr (DM > 128) {
                        mma16(s[2 * pr], qa, b[0], b[1]);
                        mma16(s[2 * pr + 1], qa, b[2], b[3]);
                    } else {
                        mma16(s[2 * pr], qf[ks], b[0], b[1]);
                        mma16(s[2 * pr + 1], qf[ks], b[2], b[3]);
                    }
                }
            }
            if (j0 + kPortK - 1 + (int)last <= warp_first) {  // every distance is beyond the table
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[i][e] = fmaf(s[i][e], factor[e >> 1], far);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int back = pos_g + (e >> 1) * 8 - (j0 + 8 * i + 2 * (int)c4 + (e & 1));
                        const float b = bias ? __ldg(bias + min((uint32_t)max(back, 0), last)) * kLog2E : 0.f;
                        s[i][e] = back < 0 ? -INFINITY : fmaf(s[i][e], factor[e >> 1], b);
                    }
            }
            float alpha[2];
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float mx = m[r];
#pragma unroll
                for (int i = 0; i < 8; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * r], s[i][2 * r + 1]));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));  // (finite: key 0 is visible to every row)
                alpha[r] = exp2f(m[r] - mx);
                m[r] = mx;
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    s[i][2 * r] = exp2f(s[i][2 * r] - mx);
                    s[i][2 * r + 1] = exp2f(s[i][2 * r + 1] - mx);
                    sum += s[i][2 * r] + s[i][2 * r + 1];
                }
                l[r] = l[r] * alpha[r] + sum;
            }
#pragma unroll
            for (int i = 0; i < DM / 8; ++i) {
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
                for (int i = 0; i < DM / 8; i += 2) {
                    if (i * 8 >= (int)a.vdim) break;
                    uint32_t b[4];
                    ldsm4_trans(b, vt + ((kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * S::kPitch + (i + (lane >> 4)) * 8) * 2);
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
        uint16_t *dst = (uint16_t *)a.out + (size_t)t * a.out_stride + h * a.vdim;
#pragma unroll
        for (int i = 0; i < DM / 8; ++i) {
            const uint32_t c = i * 8 + 2 * c4;
            if (c < a.vdim) *reinterpret_cast<uint32_t *>(dst + c) = pack_bf16(o[i][2 * r] * inv, o[i][2 * r + 1] * inv);
        }
    }
}

// ------------------------------------------------------------------ portion, bfloat16, tcgen05
// A CTA works on two units, each 128 rows of one query head; both read the same key/value head (two
// heads of a group at the same rows, or neighbouring row tiles).  Per block of 128 keys: S = Q K^T into
// tensor memory; four warps per unit turn their rows' scores into weights, which go back to tensor
// memory over S as the A operand of O += P V; O stays in tensor memory.  While one unit's warps
// exponentiate, the other unit's products run.  V is read as it lies in the cache (rows are keys), as an
// MN-major B operand.  A row's accumulator is rescaled only when its maximum has grown by more than
// 2^kUmLazy since its reference was set.  The bias of a block is a band of 255 distances: staged in
// shared memory with the mask (-inf) built in, in four copies shifted by one so that every row reads
// it in aligned pieces of four; blocks beyond the end of the bias table need no band.
// Warps 0-3 and 4-7: the units' rows; warp 8: TMA; warp 9: MMA issue.  All waits are bounded.
constexpr int kUmRows = 128, kUmKeys = 128, kUmThreads = 320, kUmStages = 2;
constexpr uint32_t kUmChunk = 128 * 128;                       // 128 rows of 64 bfloat16
constexpr uint32_t kUmTile = 2 * kUmChunk;                     // up to 128 channels
constexpr int kUmBandPitch = 264;                              // floats per copy of the band
constexpr uint32_t kUmBand = 4 * kUmBandPitch * 4;
constexpr size_t kUmSmem = 1024 + (2 + 2 * kUmStages) * kUmTile + 4 * kUmBand + 256;
constexpr uint32_t kUmOCol = 256, kUmTmemCols = 512;           // S of unit u at 128 u, O at 256 + 128 u
constexpr float kUmLazy = 8.0f;
constexpr uint32_t kUmWaitDefault = 1u << 22;
static_assert(kUmSmem <= 227 * 1024, "the tiles must fit the shared memory of a CTA");

__device__ __forceinline__ void tmem_store32(uint32_t taddr, const uint32_t *v) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, %21, %22, "
        "%23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
        "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
        "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]),
        "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]),
        "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
        : "memory");
}
// bf16 x bf16 -> f32, M = 128, N = n; b_mn: B is MN-major
__device__ __forceinline__ uint32_t portion_idesc(uint32_t n, uint32_t b_mn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn << 16) | ((n >> 3) << 17) | ((uint32_t)(kUmRows >> 4) << 24);
}
// MN-major tile in chunks of 64 columns (128-byte rows, swizzled): 8-row groups 1024 bytes apart,
// chunks kUmChunk apart.
__device__ __forceinline__ uint64_t umma_desc_mn(uint32_t smem_addr) {
    return umma_desc(smem_addr) | ((uint64_t)(kUmChunk >> 4) << 16);
}
// Barrier of the 128 threads of a unit; true when all of them say so.
__device__ __forceinline__ bool unit_vote(uint32_t u, bool ok) {
    uint32_t all;
#define QK_UNIT_VOTE(id)                                                 \
    asm volatile(                                                        \
        "{\n .reg .pred p, q;\n setp.ne.b32 p, %1, 0;\n"                 \
        " barrier.cta.red.and.pred q, " id ", 128, p;\n selp.u32 %0, 1, 0, q;\n}" \
        : "=r"(all)                                                      \
        : "r"((uint32_t)ok)                                              \
        : "memory")
    if (u == 0) QK_UNIT_VOTE("1");
    else QK_UNIT_VOTE("2");
#undef QK_UNIT_VOTE
    return all != 0;
}
// The unit `index` of a key/value head: heads of the group fastest, then row tiles.
struct PortionUnit {
    uint32_t h, row0, n_blocks;
};
__device__ __forceinline__ PortionUnit portion_unit(const GroupedArgs &a, uint32_t kvh, uint32_t index) {
    const uint32_t group = a.heads / a.kv_heads, row0 = index / group * kUmRows;
    if (row0 >= a.tokens) return {0, 0, 0};
    return {kvh * group + index % group, row0, (a.p0 + min(row0 + kUmRows, a.tokens) + kUmKeys - 1) / kUmKeys};
}

__global__ void __launch_bounds__(kUmThreads, 1)
grouped_portion_umma_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                            const __grid_constant__ CUtensorMap v_map, GroupedArgs a, uint32_t wait_limit) {
    qk::pdl_launch();
    extern __shared__ __align__(1024) uint8_t um_smem[];
    uint8_t *qs = reinterpret_cast<uint8_t *>(((uintptr_t)um_smem + 1023) & ~(uintptr_t)1023);
    uint8_t *ks = qs + 2 * kUmTile, *vs = ks + kUmStages * kUmTile;
    float *bands = reinterpret_cast<float *>(vs + kUmStages * kUmTile);  // [unit][2][4][kUmBandPitch]
    uint64_t *q_full = reinterpret_cast<uint64_t *>(bands + 4 * 4 * kUmBandPitch);
    uint64_t *k_full = q_full + 1, *k_empty = k_full + kUmStages, *v_full = k_empty + kUmStages, *v_empty = v_full + kUmStages;
    uint64_t *s_full = v_empty + kUmStages, *p_full = s_full + 2, *o_full = p_full + 2, *drain = o_full + 2;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(drain + 1);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    volatile int *never = reinterpret_cast<volatile int *>(tmem_slot + 2);
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const uint32_t kvh = blockIdx.x, pair = gridDim.y - 1 - blockIdx.y;  // (late rows see most keys)
    const PortionUnit unit[2] = {portion_unit(a, kvh, 2 * pair), portion_unit(a, kvh, 2 * pair + 1)};
    const uint32_t n_blocks = max(unit[0].n_blocks, unit[1].n_blocks);
    const uint32_t d_chunks = (a.dim + 63) / 64, v_chunks = (a.vdim + 63) / 64;
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < kUmStages; ++s) {
            mbar_init(k_full + s, 1);
            mbar_init(k_empty + s, 1);
            mbar_init(v_full + s, 1);
            mbar_init(v_empty + s, 1);
        }
        for (int u = 0; u < 2; ++u) {
            mbar_init(s_full + u, 1);
            mbar_init(p_full + u, 4);
            mbar_init(o_full + u, 1);
        }
        mbar_init(drain, 1);
        *abort_flag = 0;
        *never = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&q_map) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&k_map) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&v_map) : "memory");
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)),
                     "r"(kUmTmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    qk::pdl_wait();
    const uint32_t tmem = *tmem_slot;
    uint32_t fetched = 0;  // (warp 8) blocks whose copies have been issued

    if (warp == 8) {
        if (lane == 0) {
            const uint32_t live = (unit[0].n_blocks ? 1 : 0) + (unit[1].n_blocks ? 1 : 0);
            mbar_expect(q_full, live * d_chunks * kUmChunk);
#pragma unroll
            for (uint32_t u = 0; u < 2; ++u)
                for (uint32_t c = 0; c < d_chunks && unit[u].n_blocks; ++c)
                    tma_load_2d(smem_u32(qs + u * kUmTile + c * kUmChunk), &q_map, unit[u].h * a.dim + c * 64, unit[u].row0, q_full);
        }
        __syncwarp();
        for (uint32_t j = 0; j < n_blocks; ++j) {
            const uint32_t s = j % kUmStages, parity = ((j / kUmStages) & 1) ^ 1;
            if (!mbar_wait(k_empty + s, parity, abort_flag, wait_limit) || !mbar_wait(v_empty + s, parity, abort_flag, wait_limit)) {
                *abort_flag = 1;
                break;
            }
            if (lane == 0) {
                mbar_expect(k_full + s, d_chunks * kUmChunk);
                for (uint32_t c = 0; c < d_chunks; ++c)
                    tma_load_3d(smem_u32(ks + s * kUmTile + c * kUmChunk), &k_map, c * 64, j * kUmKeys, kvh, k_full + s);
                mbar_expect(v_full + s, v_chunks * kUmChunk);
                for (uint32_t c = 0; c < v_chunks; ++c)
                    tma_load_3d(smem_u32(vs + s * kUmTile + c * kUmChunk), &v_map, c * 64, j * kUmKeys, kvh, v_full + s);
            }
            fetched = j + 1;
            __syncwarp();
        }
    } else if (warp == 9) {
        const uint32_t idesc_s = portion_idesc(kUmKeys, 0), idesc_o = portion_idesc(a.vdim, 1);
        auto scores = [&](uint32_t u, uint32_t j) {  // (lane 0)
            const uint32_t q0 = smem_u32(qs + u * kUmTile), k0 = smem_u32(ks + (j % kUmStages) * kUmTile);
            for (uint32_t k = 0; k < a.dim / 16; ++k) {
                const uint32_t at = k / 4 * kUmChunk + k % 4 * 32;
                const uint64_t ad = umma_desc(q0 + at), bd = umma_desc(k0 + at);
                asm volatile(
                    "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
                    " tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}" ::"r"(tmem + 128 * u),
                    "l"(ad), "l"(bd), "r"(idesc_s), "r"(k)
                    : "memory");
            }
            umma_commit(s_full + u);
        };
        auto values = [&](uint32_t u, uint32_t j) {  // (lane 0)
            const uint32_t v0 = smem_u32(vs + (j % kUmStages) * kUmTile);
#pragma unroll
            for (uint32_t k = 0; k < kUmKeys / 16; ++k) {
                const uint64_t bd = umma_desc_mn(v0 + k * 2048);
                asm volatile(
                    "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
                    " tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}" ::"r"(tmem + kUmOCol + 128 * u),
                    "r"(tmem + 128 * u + k * 8), "l"(bd), "r"(idesc_o), "r"(j + k)
                    : "memory");
            }
        };
        bool ok = mbar_wait(q_full, 0, abort_flag, wait_limit) && mbar_wait(k_full, 0, abort_flag, wait_limit);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (ok && lane == 0) {
#pragma unroll
            for (uint32_t u = 0; u < 2; ++u)
                if (unit[u].n_blocks) scores(u, 0);
            umma_commit(k_empty);
        }
        __syncwarp();
        for (uint32_t j = 0; j < n_blocks && ok; ++j) {
            const uint32_t s = j % kUmStages, s1 = (j + 1) % kUmStages;
            ok = mbar_wait(v_full + s, (j / kUmStages) & 1, abort_flag, wait_limit);
            if (ok && j + 1 < n_blocks) ok = mbar_wait(k_full + s1, ((j + 1) / kUmStages) & 1, abort_flag, wait_limit);
#pragma unroll
            for (uint32_t u = 0; u < 2; ++u) {
                if (!ok || j >= unit[u].n_blocks) continue;
                ok = mbar_wait(p_full + u, j & 1, abort_flag, wait_limit);
                if (!ok) continue;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lane == 0) {
                    values(u, j);
                    if (j + 1 < unit[u].n_blocks) scores(u, j + 1);
                    else umma_commit(o_full + u);
                }
                __syncwarp();
            }
            if (ok && lane == 0) {
                umma_commit(v_empty + s);
                if (j + 1 < n_blocks) umma_commit(k_empty + s1);
            }
            __syncwarp();
        }
        if (!ok) {
            *abort_flag = 1;
            if (lane == 0) umma_commit(drain);  // the products still in flight
            __syncwarp();
            (void)mbar_wait(drain, 0, never, kUmWaitDefault);
        }
    } else {
        const uint32_t u = warp / 4, r = threadIdx.x % 128;
        const PortionUnit me = u ? unit[1] : unit[0];
        const uint32_t s_tmem = tmem + 128 * u + (((warp % 4) * 32) << 16), o_tmem = s_tmem - 128 * u + kUmOCol + 128 * u;
        const int pos = (int)(a.p0 + me.row0 + r);
        const uint32_t last = a.bias_len - 1;
        const float factor = query_scale(a, pos) * kLog2E;
        const float *bias = a.bias ? a.bias + (size_t)me.h * a.bias_len : nullptr;
        const float far = bias ? bias[last] * kLog2E : 0.f;
        float m = -INFINITY, l = 0.f;   // the accumulator's reference, the sum of the weights
        bool ok = true;
        float2 s[kUmKeys / 2];
        for (uint32_t j = 0; j < me.n_blocks; ++j) {
            // distance of the tile's first row to the block's last key; what lies before is masked
            const int nearest = (int)(a.p0 + me.row0) - (int)(j * kUmKeys + kUmKeys - 1);
            const bool near = nearest < (int)last || nearest < 0;
            float *band = bands + (u * 2 + (j & 1)) * 4 * kUmBandPitch;
            if (near) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int at = (int)r + 128 * half, distance = nearest + 2 * kUmKeys - 2 - at;
                    float b = -INFINITY;
                    if (distance >= 0) b = bias ? __ldg(bias + min((uint32_t)distance, last)) * kLog2E : 0.f;
#pragma unroll
                    for (int c = 0; c < 4; ++c)
                        if (at >= c) band[c * kUmBandPitch + at - c] = b;
                }
            }
            // (the unit's four warps go on together, or leave together; the band is complete then)
            ok = unit_vote(u, mbar_wait(s_full + u, j & 1, abort_flag, wait_limit));
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            uint32_t raw[4][32];
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_ld32(s_tmem + 32 * c, raw[c]);
            tmem_ld_wait();
            const float2 f2 = make_float2(factor, factor);
            float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (near) {
                const uint32_t shift = 127 - r;
                const float4 *bp = reinterpret_cast<const float4 *>(band + (shift & 3) * kUmBandPitch + (shift & ~3u));
#pragma unroll
                for (int e = 0; e < kUmKeys / 4; ++e) {
                    const float4 b = bp[e];
                    s[2 * e] = __ffma2_rn(make_float2(__uint_as_float(raw[e / 8][e % 8 * 4]), __uint_as_float(raw[e / 8][e % 8 * 4 + 1])),
                                          f2, make_float2(b.x, b.y));
                    s[2 * e + 1] = __ffma2_rn(
                        make_float2(__uint_as_float(raw[e / 8][e % 8 * 4 + 2]), __uint_as_float(raw[e / 8][e % 8 * 4 + 3])), f2,
                        make_float2(b.z, b.w));
                }
            } else {
                const float2 b2 = make_float2(far, far);
#pragma unroll
                for (int e = 0; e < kUmKeys / 2; ++e)
                    s[e] = __ffma2_rn(make_float2(__uint_as_float(raw[e / 16][e % 16 * 2]), __uint_as_float(raw[e / 16][e % 16 * 2 + 1])),
                                      f2, b2);
            }
#pragma unroll
            for (int e = 0; e < kUmKeys / 2; ++e) mx[e % 4] = fmaxf(mx[e % 4], fmaxf(s[e].x, s[e].y));
            const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
            float alpha = 1.f;
            if (top > m + kUmLazy) {  // (in the first block always: key 0 is visible to every row)
                alpha = ex2(m - top);
                m = top;
            }
            if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
                // (the scores' barrier also says that the product before them is complete)
#pragma unroll 1
                for (uint32_t c = 0; c < a.vdim; c += 32) {
                    uint32_t o[32];
                    tmem_ld32(o_tmem + c, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
                    tmem_store32(o_tmem + c, o);
                }
            }
            float2 sum[2] = {make_float2(l * alpha, 0.f), make_float2(0.f, 0.f)};
            const float2 m2 = make_float2(-m, -m);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t p[32];
#pragma unroll
                for (int e = 0; e < 32; ++e) {
                    const float2 x = __fadd2_rn(s[32 * half + e], m2);
                    const float2 w = make_float2(ex2(x.x), ex2(x.y));
                    sum[e % 2] = __fadd2_rn(sum[e % 2], w);
                    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(p[e]) : "f"(w.y), "f"(w.x));
                }
                tmem_store32(s_tmem + 32 * half, p);
            }
            l = (sum[0].x + sum[0].y) + (sum[1].x + sum[1].y);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + u);
        }
        if (me.n_blocks && ok) ok = mbar_wait(o_full + u, 0, abort_flag, wait_limit);
        if (!ok) *abort_flag = 1;
        if (me.n_blocks && ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float inv = 1.0f / l;
            const uint32_t t = me.row0 + r;
            uint16_t *dst = (uint16_t *)a.out + (size_t)t * a.out_stride + me.h * a.vdim;
#pragma unroll 1
            for (uint32_t c = 0; c < a.vdim; c += 32) {
                uint32_t o[32];
                tmem_ld32(o_tmem + c, o);
                tmem_ld_wait();
                if (t >= a.tokens) continue;
#pragma unroll
                for (int e = 0; e < 32; e += 8) {
                    if (c + e >= a.vdim) break;
                    uint32_t w[4];
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        w[i] = pack_bf16(__uint_as_float(o[e + 2 * i]) * inv, __uint_as_float(o[e + 2 * i + 1]) * inv);
                    *reinterpret_cast<uint4 *>(dst + c + e) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        }
    }
    __syncwarp();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 8 && *abort_flag) {  // the copies still in flight
        (void)mbar_wait(q_full, 0, never, kUmWaitDefault);
        for (uint32_t j = fetched > kUmStages ? fetched - kUmStages : 0; j < fetched; ++j) {
            (void)mbar_wait(k_full + j % kUmStages, (j / kUmStages) & 1, never, kUmWaitDefault);
            (void)mbar_wait(v_full + j % kUmStages, (j / kUmStages) & 1, never, kUmWaitDefault);
        }
    }
    if (warp == 9)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kUmTmemCols) : "memory");
    if (threadIdx.x == 0 && *abort_flag) atomicOr(a.error, 1);
}

// ------------------------------------------------------------------ plain, float32 arithmetic
// Grid (splits, query heads, rows).  Tiles of 128 keys: a thread scores one key, then owns value
// channels threadIdx.x, + 128, ...
constexpr int kPlainKeys = 128, kPlainChannels = 8;
template <typename C>
__device__ __forceinline__ float dot_row(const C *__restrict__ k, const float *q, uint32_t n) {
    float s = 0.f;
    for (uint32_t c = 0; c < n; c += 4) {
        float x[4];
        load_piece(k + c, x);
        s = fmaf(q[c], x[0], fmaf(q[c + 1], x[1], fmaf(q[c + 2], x[2], fmaf(q[c + 3], x[3], s))));
    }
    return s;
}
template <typename C>
__global__ void __launch_bounds__(kPlainKeys)
grouped_plain_kernel(GroupedArgs a) {
    qk::pdl_launch();
    qk::pdl_wait();
    extern __shared__ __align__(16) float plain_smem[];  // [dim] query, [128] weights
    __shared__ float red[4];
    float *q = plain_smem, *p = plain_smem + a.dim;
    const uint32_t t = blockIdx.z, h = blockIdx.y, kvh = h / (a.heads / a.kv_heads);
    const int pos = live_position(a, t);
    if (pos < 0) return;
    const uint32_t n_keys = (uint32_t)pos + 1;
    const uint32_t per = max((uint32_t)kPlainKeys, (n_keys + a.n_splits - 1) / a.n_splits), first = blockIdx.x * per;
    if (first >= n_keys) return;
    const uint32_t n_active = (n_keys + per - 1) / per, end = min(first + per, n_keys);
    for (uint32_t c = threadIdx.x; c < a.dim; c += kPlainKeys) q[c] = ((const float *)a.proj)[(size_t)t * a.proj_stride + h * a.dim + c];
    const size_t head_row = ((size_t)a.slots[t] * a.kv_heads + kvh) * a.s_max;
    const C *kb = (const C *)a.cache_k + head_row * a.dim, *vb = (const C *)a.cache_v + head_row * a.vdim;
    const float *bias = a.bias ? a.bias + (size_t)h * a.bias_len : nullptr;
    const float factor = query_scale(a, pos);
    float o[kPlainChannels] = {}, m = -INFINITY, l = 0.f;
    __syncthreads();
    for (uint32_t k0 = first; k0 < end; k0 += kPlainKeys) {
        const uint32_t j = k0 + threadIdx.x;
        float s = -INFINITY;
        if (j < end) {
            s = dot_row(kb + (size_t)j * a.dim, q, a.dim) * factor;
            if (bias) s += bias[min((uint32_t)pos - j, a.bias_len - 1)];
        }
        float mx = s;
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        if (threadIdx.x % 32 == 0) red[threadIdx.x / 32] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);  // (finite: key k0 is live)
        const float alpha = expf(m - mx), w = expf(s - mx);
        m = mx;
        p[threadIdx.x] = w;
        __syncthreads();
        l *= alpha;
        const uint32_t n = min((uint32_t)kPlainKeys, end - k0);
        for (uint32_t i = 0; i < n; ++i) l += p[i];  // (the same sum in every thread)
#pragma unroll
        for (int e = 0; e < kPlainChannels; ++e) {
            const uint32_t c = threadIdx.x + kPlainKeys * e;
            if (c >= a.vdim) break;
            float v = o[e] * alpha;
            for (uint32_t i = 0; i < n; ++i) v = fmaf(p[i], load_as_float<C>(vb, (size_t)(k0 + i) * a.vdim + c), v);
            o[e] = v;
        }
        __syncthreads();
    }
    const float inv = 1.0f / l;
#pragma unroll
    for (int e = 0; e < kPlainChannels; ++e) {
        const uint32_t c = threadIdx.x + kPlainKeys * e;
        if (c >= a.vdim) break;
        if (n_active == 1) put(a.out, a.out_bf16, (size_t)t * a.out_stride + h * a.vdim + c, o[e] * inv);
        else a.partial[(((size_t)t * a.heads + h) * a.n_splits + blockIdx.x) * (a.vdim + 8) + c] = o[e];
    }
    if (n_active > 1) {
        if (threadIdx.x == 0) {
            float *dst = a.partial + (((size_t)t * a.heads + h) * a.n_splits + blockIdx.x) * (a.vdim + 8) + a.vdim;
            dst[0] = m;
            dst[1] = l;
        }
        if (last_to_finish(a.tickets + (size_t)t * a.heads + h, n_active)) combine_splits<false>(a, t, h, 1, n_active);
    }
}

qk_status enter(qk_ctx *ctx, const qk_grouped_call *d, qk_ctx **out, GroupedArgs *args) {
    qk_status st = qk::resolve_ctx(ctx, out);
    if (st != QK_OK) return st;
    qk_ctx *c = *out;
    QK_CUDA(cudaSetDevice(c->device));
    if (!d || !d->proj || !d->cache_k || !d->cache_v) return qk::fail(QK_ERR_VALUE, "grouped attention: null argument");
    if (d->heads == 0 || d->kv_heads == 0 || d->heads % d->kv_heads)
        return qk::fail(QK_ERR_VALUE, "grouped attention: %zu heads over %zu key/value heads", d->heads, d->kv_heads);
    if (d->dim_stride == 0 || d->vdim_stride == 0 || d->dim_stride % 16 || d->vdim_stride % 16 || d->proj_stride % 8 ||
        d->proj_stride < d->heads * d->dim_stride + d->kv_heads * (d->dim_stride + d->vdim_stride))
        return qk::fail(QK_ERR_VALUE, "grouped attention: head strides %zu and %zu in rows of %zu", d->dim_stride, d->vdim_stride,
                        d->proj_stride);
    if ((d->proj_dtype != QK_F32 && d->proj_dtype != QK_BF16) || (d->cache_dtype != QK_F32 && d->cache_dtype != QK_BF16))
        return qk::fail(QK_ERR_VALUE, "grouped attention: dtypes must be float32 or bfloat16, got tags %d and %d", d->proj_dtype,
                        d->cache_dtype);
    if (d->s_max == 0 || d->n_slots == 0 || d->s_max > (1u << 30) || (d->bias && d->bias_len == 0) || d->temp_every < 0.0)
        return qk::fail(QK_ERR_VALUE, "grouped attention: %zu slots of %zu positions, %zu biases", d->n_slots, d->s_max, d->bias_len);
    if ((st = qk::error_word(c)) != QK_OK) return st;
    c->err_armed = true;
    GroupedArgs a{};
    a.positions = d->positions;
    a.slots = d->slots;
    a.proj = d->proj;
    a.bias = d->bias;
    a.cache_k = d->cache_k;
    a.cache_v = d->cache_v;
    a.out = d->out;
    a.error = (int *)c->d_err.ptr;
    a.tokens = (uint32_t)d->tokens;
    a.heads = (uint32_t)d->heads;
    a.kv_heads = (uint32_t)d->kv_heads;
    a.dim = (uint32_t)d->dim_stride;
    a.vdim = (uint32_t)d->vdim_stride;
    a.s_max = (uint32_t)d->s_max;
    a.n_slots = (uint32_t)d->n_slots;
    a.proj_stride = (uint32_t)d->proj_stride;
    a.out_stride = (uint32_t)d->out_stride;
    a.n_splits = (uint32_t)d->n_splits;
    a.bias_len = d->bias ? (uint32_t)d->bias_len : 1;
    a.slot = (uint32_t)d->slot;
    a.p0 = (uint32_t)d->first_position;
    a.scale = d->scale;
    a.temp_coef = d->temp_coef;
    a.temp_every = d->temp_every;
    a.append = d->append;
    a.out_bf16 = d->out_dtype == QK_BF16;
    *args = a;
    return QK_OK;
}
#define QK_GROUPED(c, kernel, grid, block, smem, ...)                                                                  \
    do {                                                                                                               \
        if ((smem) > 48 * 1024)                                                                                        \
            QK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(smem)));           \
        (void)qk::launch_pdl((c)->pdl, kernel, grid, block, smem, (c)->stream, __VA_ARGS__);                           \
        QK_CUDA(cudaGetLastError());                                                                                   \
        (c)->launches++;                                                                                               \
    } while (0)

qk_status launch_portion_umma(qk_ctx *c, const qk_grouped_call *d, const GroupedArgs &a) {
    CUtensorMap qm, km, vm;
    qk_status st;
    const size_t n_keys = d->first_position + d->tokens;  // (rows behind them are filled with zeros)
    const uint16_t *k = (const uint16_t *)d->cache_k + d->slot * d->kv_heads * d->s_max * d->dim_stride;
    const uint16_t *v = (const uint16_t *)d->cache_v + d->slot * d->kv_heads * d->s_max * d->vdim_stride;
    const cuuint64_t q_dims[2] = {d->proj_stride, d->tokens}, q_strides[1] = {d->proj_stride * 2};
    const cuuint64_t k_dims[3] = {d->dim_stride, n_keys, d->kv_heads}, k_strides[2] = {d->dim_stride * 2, d->s_max * d->dim_stride * 2};
    const cuuint64_t v_dims[3] = {d->vdim_stride, n_keys, d->kv_heads}, v_strides[2] = {d->vdim_stride * 2, d->s_max * d->vdim_stride * 2};
    const cuuint32_t box[3] = {64, 128, 1};
    if ((st = encode_bf16_map(d->proj, 2, q_dims, q_strides, box, &qm)) != QK_OK) return st;
    if ((st = encode_bf16_map(k, 3, k_dims, k_strides, box, &km)) != QK_OK) return st;
    if ((st = encode_bf16_map(v, 3, v_dims, v_strides, box, &vm)) != QK_OK) return st;
    const uint32_t units = (a.heads / a.kv_heads) * (uint32_t)qk::ceil_div(d->tokens, kUmRows);
    const dim3 grid(a.kv_heads, (units + 1) / 2), block(kUmThreads);
    QK_GROUPED(c, grouped_portion_umma_kernel, grid, block, kUmSmem, qm, km, vm, a, c->wait_limit ? c->wait_limit : kUmWaitDefault);
    return QK_OK;
}

qk_status launch_append(qk_ctx *c, const qk_grouped_call *d, const GroupedArgs &a) {
    const dim3 grid(a.tokens), block(256);
    if (d->proj_dtype == QK_F32 && d->cache_dtype == QK_F32) QK_GROUPED(c, (grouped_append_kernel<float, float>), grid, block, 0, a);
    else if (d->proj_dtype == QK_F32) QK_GROUPED(c, (grouped_append_kernel<float, uint16_t>), grid, block, 0, a);
    else if (d->cache_dtype == QK_BF16) QK_GROUPED(c, (grouped_append_kernel<uint16_t, uint16_t>), grid, block, 0, a);
    else return qk::fail(QK_ERR_VALUE, "grouped attention: bfloat16 projections need a bfloat16 cache");
    return QK_OK;
}

}  // namespace

extern "C" {

size_t qk_grouped_scratch(size_t tokens, size_t heads, size_t kv_heads, size_t vdim_stride, size_t n_splits) {
    (void)kv_heads;
    return tokens * heads * (n_splits * (vdim_stride + 8) + 1) * 4;
}

qk_status qk_grouped_append(qk_ctx *ctx, const qk_grouped_call *d) {
    qk_ctx *c;
    GroupedArgs a;
    qk_status st = enter(ctx, d, &c, &a);
    if (st != QK_OK) return st;
    if (!d->positions || !d->slots) return qk::fail(QK_ERR_VALUE, "qk_grouped_append: null argument");
    return d->tokens == 0 ? QK_OK : launch_append(c, d, a);
}

qk_status qk_grouped_attention(qk_ctx *ctx, const qk_grouped_call *d) {
    qk_ctx *c;
    GroupedArgs a;
    qk_status st = enter(ctx, d, &c, &a);
    if (st != QK_OK) return st;
    if (!d->positions || !d->slots || !d->scratch || !d->out || d->n_splits == 0)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_attention: null argument");
    if (d->proj_dtype != QK_F32) return qk::fail(QK_ERR_VALUE, "qk_grouped_attention: the projections must be float32");
    if (d->out_stride % 4 || d->out_stride < d->heads * d->vdim_stride)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_attention: output rows of %zu", d->out_stride);
    if (d->tokens == 0) return QK_OK;
    if (d->tokens > 65535 || d->heads > 65535) return qk::fail(QK_ERR_VALUE, "qk_grouped_attention: at most 65535 rows and heads");
    a.partial = d->scratch;
    a.tickets = reinterpret_cast<uint32_t *>(d->scratch + d->tokens * d->heads * d->n_splits * (d->vdim_stride + 8));
    const uint32_t widest = std::max(a.dim, a.vdim), group = a.heads / a.kv_heads;
    if (d->cache_dtype == QK_BF16 && widest <= 256 && c->decode_attention_kernel != 0) {
        const dim3 grid(a.n_splits, a.kv_heads * ((group + 7) / 8), a.tokens), block(128);
        const bool full = a.dim == a.vdim;
        if (widest == 64 && full) QK_GROUPED(c, (grouped_rows_kernel<64, true>), grid, block, RowShape<64>::kSmem, a);
        else if (widest <= 64) QK_GROUPED(c, (grouped_rows_kernel<64, false>), grid, block, RowShape<64>::kSmem, a);
        else if (widest == 128 && full) QK_GROUPED(c, (grouped_rows_kernel<128, true>), grid, block, RowShape<128>::kSmem, a);
        else if (widest <= 128) QK_GROUPED(c, (grouped_rows_kernel<128, false>), grid, block, RowShape<128>::kSmem, a);
        else QK_GROUPED(c, (grouped_rows_kernel<256, false>), grid, block, RowShape<256>::kSmem, a);
        return QK_OK;
    }
    if (d->vdim_stride > kPlainKeys * kPlainChannels || d->dim_stride > 8192)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_attention: head sizes %zu and %zu are not supported", d->dim_stride, d->vdim_stride);
    if (d->append && (st = launch_append(c, d, a)) != QK_OK) return st;
    const dim3 grid(a.n_splits, a.heads, a.tokens), block(kPlainKeys);
    const size_t smem = (d->dim_stride + kPlainKeys) * 4;
    if (d->cache_dtype == QK_F32) QK_GROUPED(c, grouped_plain_kernel<float>, grid, block, smem, a);
    else QK_GROUPED(c, grouped_plain_kernel<uint16_t>, grid, block, smem, a);
    return QK_OK;
}

qk_status qk_grouped_portion(qk_ctx *ctx, const qk_grouped_call *d) {
    qk_ctx *c;
    GroupedArgs a;
    qk_status st = enter(ctx, d, &c, &a);
    if (st != QK_OK) return st;
    if (!d->out || d->proj_dtype != QK_BF16 || d->cache_dtype != QK_BF16 || d->out_dtype != QK_BF16)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_portion: bfloat16 projections, caches and output are needed");
    const uint32_t widest = std::max(a.dim, a.vdim);
    if (widest > 256) return qk::fail(QK_ERR_VALUE, "qk_grouped_portion: head sizes above 256 are not supported, got %u", widest);
    if (d->first_position + d->tokens > d->s_max || d->slot >= d->n_slots)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_portion: positions %zu..%zu of slot %zu do not fit the cache", d->first_position,
                        d->first_position + d->tokens - 1, d->slot);
    if (d->out_stride % 2 || d->out_stride < d->heads * d->vdim_stride)
        return qk::fail(QK_ERR_VALUE, "qk_grouped_portion: output rows of %zu", d->out_stride);
    if (d->tokens == 0) return QK_OK;
    auto aligned = [](const void *p) { return ((uintptr_t)p & 15) == 0; };
    if (a.dim >= 64 && a.vdim >= 64 && widest <= 128 && a.out_stride % 8 == 0 && aligned(d->proj) && aligned(d->out) &&
        aligned(d->cache_k) && aligned(d->cache_v) && c->decode_attention_kernel != 0)
        return launch_portion_umma(c, d, a);
    const dim3 grid((unsigned)qk::ceil_div(d->tokens, kPortQ), a.heads), block(128);
    if (widest <= 64) QK_GROUPED(c, grouped_portion_kernel<64>, grid, block, PortShape<64>::kSmem, a);
    else if (widest <= 128) QK_GROUPED(c, grouped_portion_kernel<128>, grid, block, PortShape<128>::kSmem, a);
    else QK_GROUPED(c, grouped_portion_kernel<256>, grid, block, PortShape<256>::kSmem, a);
    return QK_OK;
}

}  // extern "C"
