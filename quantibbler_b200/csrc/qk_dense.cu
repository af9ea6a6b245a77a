// Dense linears y = W x with bfloat16 or float32 weights, in four forms:
//   * vector (up to kVectorTokens rows): one launch; every block forms the input vectors itself
//     (norm, pending residual, gate - see qk_dense_dev.cuh) and its warps stream weight rows;
//   * narrow (bfloat16, up to kNarrowTokens rows): tcgen05.mma with the weights on the M side, each
//     byte of them read once, the k range shared out over a cluster;
//   * tcgen05 (bfloat16, more rows): persistent TMA-fed tcgen05.mma with two accumulators in
//     tensor memory;
//   * float32 (more rows, float32 weights): plain float32 multiply-adds, no reduced-precision
//     matrix mode.
// The matrix forms take their input rows from a kernel that runs the same device function as
// the vector form.  All forms share the epilogues.
#include <cuda.h>  // CUtensorMap types only; the encoder is fetched through the runtime

#include <algorithm>

#include "qk_dense_dev.cuh"
#include "qk_tma.cuh"
#include "qk_umma.cuh"

namespace {

constexpr int kVecThreads = 256, kVecWarps = kVecThreads / 32;
constexpr int kRouteTile = 5;  // a tile of qk_route: expert, first and last + 1 place, the expert's first tile, its tiles
constexpr int kVectorTokens = 4;
constexpr int kNarrowTokens = 128;
enum { kRowAny = 0, kRowNorm = 1, kRowPlain = 2 };  // how input rows may be read
constexpr size_t kVecSmemMax = 200 * 1024, kVecSmemSm = 226 * 1024;  // of a block, of an SM

// ------------------------------------------------------------------ vector form
template <typename W> struct VecTraits;
template <> struct VecTraits<uint16_t> {
    static constexpr uint32_t kPer = 8, kStep = 32 * 8;  // entries per lane and per warp step
    // A lane reads entries 8l .. 8l+7 of a 256-entry step as two 16-byte pieces: the first
    // halves of all lanes lie side by side, then the second halves, so that a warp's reads hit
    // every bank once.
    __device__ static uint32_t place(uint32_t i) {
        return (i & ~255u) | ((i & 4u) << 5) | ((i & 248u) >> 1) | (i & 3u);
    }
};
template <> struct VecTraits<float> {
    static constexpr uint32_t kPer = 4, kStep = 32 * 4;
    __device__ static uint32_t place(uint32_t i) { return i; }
};

__device__ __forceinline__ uint4 load_weights16(const void *p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(p));
    return v;
}

template <typename W, int NT>
__device__ __forceinline__ void vec_fma(float (&acc)[NT], const uint4 &w, const float *xs, uint32_t pitch,
                                        uint32_t at, uint32_t lane) {
    if constexpr (sizeof(W) == 2) {
        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            const float *p = xs + t * pitch + at + lane * 4;
            const float4 a = *reinterpret_cast<const float4 *>(p);
            const float4 b = *reinterpret_cast<const float4 *>(p + 128);
            const float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                acc[t] = fmaf(__uint_as_float(u[e] << 16), v[2 * e], acc[t]);
                acc[t] = fmaf(__uint_as_float(u[e] & 0xffff0000u), v[2 * e + 1], acc[t]);
            }
        }
    } else {
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            const float4 a = *reinterpret_cast<const float4 *>(xs + t * pitch + at + lane * 4);
            acc[t] = fmaf(__uint_as_float(w.x), a.x, acc[t]);
            acc[t] = fmaf(__uint_as_float(w.y), a.y, acc[t]);
            acc[t] = fmaf(__uint_as_float(w.z), a.z, acc[t]);
            acc[t] = fmaf(__uint_as_float(w.w), a.w, acc[t]);
        }
    }
}

// A warp (or `ksplit` warps that share out the k range) owns R weight rows at a time (with a gated
// pair, R / 2 gate rows and their up rows).  As many blocks as stay resident walk over the rows, so
// that each forms the input once; the next rows' first weights are requested while the last ones
// of the present rows are multiplied.  The rows are dealt out block by block before warp by warp:
// every SM gets its share, wherever blocks that come in early (before the kernel in front has
// left) find room.
// (The blocks per SM matter more than a spilled register: they hide each other's prologues.)
__host__ __device__ constexpr int vec_blocks(int nt, int r) { return nt == 4 && r == 4 ? 2 : r == 1 && nt <= 2 ? 4 : 3; }
template <typename W, int NT, int R>
__global__ void __launch_bounds__(kVecThreads, vec_blocks(NT, R))
dense_vector_kernel(InputArgs in, OutputArgs out, const W *__restrict__ w, uint32_t rows, uint32_t w_stride,
                    uint32_t n_tokens, uint32_t ksplit, ChoiceArgs ch, int row_kind) {
    using T = VecTraits<W>;
    constexpr int U = R >= 4 ? 2 : 4;  // steps in flight
    constexpr int HR = R >= 2 ? R / 2 : 1;
    qk::pdl_launch();
    extern __shared__ __align__(16) float xs[];  // [NT][pitch], staged norm weights [2][width]
    __shared__ float red[kVecWarps];
    __shared__ float part_sum[2][kVecWarps][R * NT];
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    const uint32_t k = in.k, pitch = (k + T::kStep - 1) / T::kStep * T::kStep, steps = pitch / T::kStep;
    const uint32_t part = warp % ksplit, batches = (steps + U * ksplit - 1) / (U * ksplit);
    const bool pair = out.kind == QK_OUTPUT_GLU;
    const uint32_t per_block = kVecWarps / ksplit, per_group = pair ? HR : R;
    const uint32_t groups = ((pair ? rows / 2 : rows) + per_group - 1) / per_group;
    uint32_t t_in = 0, t_out = 0;  // first input and output row
    bool writer = blockIdx.x == 0;
    if (ch.table) {
        // one choice of one token per block row (NT is 1).  The token ids are written by copies and
        // ordinary launches in front of the step, none of which lets a kernel start early.
        const uint32_t t = blockIdx.y / ch.top, id = (uint32_t)min(max(ch.ids[t], 0), (int)ch.vocab - 1);
        w += (size_t)ch.table[(size_t)id * ch.top + blockIdx.y % ch.top] * rows * w_stride;
        t_out = blockIdx.y;
        t_in = ch.by_choice ? t_out : t;
        writer = writer && blockIdx.y % ch.top == 0;
    }
    const W *row[R];   // the rows whose weights are requested next
    bool any = false;
    auto turn_to = [&](uint32_t group) {
        any = group < groups;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const uint32_t n = pair ? pair_row(group * HR + r % HR) + (r >= HR ? 32 : 0) : group * R + r;
            row[r] = w + (size_t)min(n, rows - 1) * w_stride + lane * T::kPer;
        }
    };
    uint4 cur[U][R];
    auto fetch = [&](uint32_t s, uint4 (&dst)[R]) {
        const bool live = any && s < steps && s * T::kStep + lane * T::kPer < k;
#pragma unroll
        for (int r = 0; r < R; ++r)
            dst[r] = live ? load_weights16(row[r] + (size_t)s * T::kStep) : make_uint4(0, 0, 0, 0);
    };
    uint32_t group = warp / ksplit * gridDim.x + blockIdx.x;
    // weights depend on no other kernel: the first ones are requested before the dependency wait
    turn_to(group);
#pragma unroll
    for (int u = 0; u < U; ++u) fetch(part + u * ksplit, cur[u]);
    float *staged = xs + NT * pitch;
    if (row_kind == kRowNorm) stage_norm_weights(in, staged);
    qk::pdl_wait();
#pragma unroll 1
    for (uint32_t t = 0; t < (uint32_t)NT; ++t) {
        float *dst = xs + t * pitch;
        if (t < n_tokens) {
            auto at4 = [&](uint32_t p) -> float4 & { return *reinterpret_cast<float4 *>(dst + T::place(4 * p)); };
            if (row_kind == kRowNorm) build_norm_row(in, t_in + t, writer, staged, at4, red);
            else if (row_kind == kRowPlain) build_plain_row(in, t_in + t, at4);
            else build_input(in, t_in + t, writer, [&](uint32_t i) -> float & { return dst[T::place(i)]; }, red);
        }
        // what lies between k and the pitch meets zero weights; it must only be finite
        for (uint32_t i = (t < n_tokens ? k : 0) + threadIdx.x; i < pitch; i += kVecThreads) dst[T::place(i)] = 0.f;
    }
    __syncthreads();
    uint32_t turn = 0;
#pragma unroll 1
    for (uint32_t first = blockIdx.x; first < groups; first += gridDim.x * per_block, turn ^= 1) {
        const uint32_t next = group + gridDim.x * per_block;
        float acc[R][NT];
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int t = 0; t < NT; ++t) acc[r][t] = 0.f;
#pragma unroll 1
        for (uint32_t b = 0; b < batches; ++b) {
            const bool over = b + 1 == batches;
            if (over) turn_to(next);
            const uint32_t ahead = over ? part : part + (b + 1) * U * ksplit;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                uint4 now[R];
#pragma unroll
                for (int r = 0; r < R; ++r) now[r] = cur[u][r];
                const uint32_t at = part + (b * U + u) * ksplit;
                fetch(ahead + u * ksplit, cur[u]);
                if (at < steps) {
#pragma unroll
                    for (int r = 0; r < R; ++r) vec_fma<W, NT>(acc[r], now[r], xs, pitch, at * T::kStep, lane);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                float a = acc[r][t];
                for (int off = 16; off > 0; off >>= 1) a += __shfl_xor_sync(0xffffffffu, a, off);
                acc[r][t] = a;
            }
        if (ksplit > 1) {  // (two buffers: the turn after the next finds this one read)
            if (lane == 0) {
#pragma unroll
                for (int r = 0; r < R; ++r)
#pragma unroll
                    for (int t = 0; t < NT; ++t) part_sum[turn][warp][r * NT + t] = acc[r][t];
            }
            __syncthreads();
            if (part == 0) {
#pragma unroll
                for (int r = 0; r < R; ++r)
#pragma unroll
                    for (int t = 0; t < NT; ++t)
                        for (uint32_t p = 1; p < ksplit; ++p) acc[r][t] += part_sum[turn][warp + p][r * NT + t];
            }
        }
        if (part == 0) {
            if (pair) {
                if constexpr (R >= 2) {
#pragma unroll
                    for (int r = 0; r < R / 2; ++r)
#pragma unroll
                        for (int t = 0; t < NT; ++t) {
                            const uint32_t j = group * (R / 2) + r;
                            if (lane == (uint32_t)(r * NT + t) && (uint32_t)t < n_tokens && j < rows / 2)
                                finish_pair(out, t_out + t, j, acc[r][t], acc[r + R / 2][t]);
                        }
                }
            } else {
#pragma unroll
                for (int r = 0; r < R; ++r)
#pragma unroll
                    for (int t = 0; t < NT; ++t)
                        if (lane == (uint32_t)(r * NT + t) && (uint32_t)t < n_tokens && group * R + r < rows)
                            finish(out, t_out + t, group * R + r, acc[r][t]);
            }
        }
        group = next;
    }
    if (in.append.src && blockIdx.x == gridDim.x - 1)
        for (uint32_t t = 0; t < n_tokens; ++t) append_latent(in, t, red);
}

// ------------------------------------------------------------------ input rows of the matrix forms
template <typename A>
__global__ void __launch_bounds__(256)
dense_input_kernel(InputArgs in, A *__restrict__ dst, int row_kind) {
    qk::pdl_launch();
    extern __shared__ __align__(16) float row_smem[];  // [k], staged norm weights [2][width]
    __shared__ float red[8];
    const uint32_t t = blockIdx.x;
    if (row_kind == kRowNorm) stage_norm_weights(in, row_smem + in.k);
    qk::pdl_wait();
    if (dst) {
        if (row_kind == kRowNorm)
            build_norm_row(in, t, true, row_smem + in.k,
                           [&](uint32_t p) -> float4 & { return *reinterpret_cast<float4 *>(row_smem + 4 * p); }, red);
        else
            build_input(in, t, true, [&](uint32_t i) -> float & { return row_smem[i]; }, red);
        for (uint32_t j = 0; j < (in.places ? in.top : 1u); ++j) {
            A *o = dst + (size_t)(in.places ? (uint32_t)in.places[t * in.top + j] : t) * in.k;
            if constexpr (sizeof(A) == 2) {
                for (uint32_t i = threadIdx.x * 2; i < in.k; i += 512) {  // (k is a multiple of 8)
                    const uint32_t lo = float_to_bf16_bits(row_smem[i]), hi = float_to_bf16_bits(row_smem[i + 1]);
                    *reinterpret_cast<uint32_t *>(o + i) = lo | (hi << 16);
                }
            } else {
                for (uint32_t i = threadIdx.x; i < in.k; i += 256) o[i] = row_smem[i];
            }
        }
    }
    if (in.append.src) append_latent(in, t, red);
}

// ------------------------------------------------------------------ float32 form
constexpr int kFTile = 64, kFK = 16;
__global__ void __launch_bounds__(256)
dense_f32_kernel(const float *__restrict__ x, uint32_t x_stride, uint32_t k, const float *__restrict__ w,
                 uint32_t rows, uint32_t w_stride, uint32_t n_tokens, OutputArgs out, const int32_t *__restrict__ tiles) {
    qk::pdl_launch();
    qk::pdl_wait();
    __shared__ float xt[kFK][kFTile + 1], wt[kFK][kFTile + 1];
    const uint32_t tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    uint32_t t0 = blockIdx.y * kFTile;
    const uint32_t n0 = blockIdx.x * kFTile;
    if (tiles) {  // rows sorted by expert
        if (blockIdx.y >= (uint32_t)tiles[0]) return;
        const int32_t *tile = tiles + 1 + kRouteTile * blockIdx.y;
        w += (size_t)tile[0] * rows * w_stride;
        t0 = (uint32_t)tile[1];
        n_tokens = (uint32_t)tile[2];
    }
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < k; k0 += kFK) {
        for (uint32_t i = threadIdx.x; i < kFTile * kFK; i += 256) {
            const uint32_t kk = i % kFK, r = i / kFK;
            const bool in_k = k0 + kk < k;
            xt[kk][r] = in_k && t0 + r < n_tokens ? x[(size_t)(t0 + r) * x_stride + k0 + kk] : 0.f;
            wt[kk][r] = in_k && n0 + r < rows ? w[(size_t)(n0 + r) * w_stride + k0 + kk] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < kFK; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = xt[kk][ty + 16 * i], b[i] = wt[kk][tx + 16 * i];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const uint32_t t = t0 + ty + 16 * i;
        if (t >= n_tokens) continue;
        if (out.kind == QK_OUTPUT_GLU) {  // one block of 32 gate rows and 32 up rows per tile
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const uint32_t o = blockIdx.x * 32 + tx + 16 * j;
                if (o < rows / 2) finish_pair(out, t, o, acc[i][j], acc[i][j + 2]);
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tx + 16 * j < rows) finish(out, t, n0 + tx + 16 * j, acc[i][j]);
        }
    }
}

// ------------------------------------------------------------------ tcgen05 form
// D[128 rows of x][BN weight rows]: x on the M side (an accumulator lane is a token, so that an
// epilogue thread holds consecutive outputs of one token), W on the N side; both K-major tiles of
// 64 k brought in by TMA with the 128-byte swizzle.  One persistent CTA per SM walks over the
// tiles (token tiles fastest: neighbouring CTAs share the weight tile in L2).  Warp 0 issues the
// copies, warp 1 the MMAs, warps 2..5 run the epilogue of one of two tensor-memory accumulators
// while the next tile is multiplied into the other.  Every wait is bounded; a CTA that gives up
// drains its copies and products in flight before it frees tensor memory.
constexpr int kTcM = 128, kTcK = 64, kTcThreads = 192, kTcEpiWarps = 4;
constexpr uint32_t kTcWaitDefault = 1u << 22;
template <int BN> struct TcShape {
    static constexpr uint32_t kABytes = kTcM * kTcK * 2, kBBytes = BN * kTcK * 2, kStage = kABytes + kBBytes;
    static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 6 : 8;
    static constexpr uint32_t kTmemCols = 2 * BN;
    static constexpr size_t kSmem = 1024 + kStages * kStage + kTcEpiWarps * 32 * 36 * 4 + (2 * kStages + 5) * 8 + 32;
    static_assert(kSmem <= 227 * 1024, "the stages must fit the shared memory of a CTA");
};
struct TcArgs {
    uint32_t n_tokens, rows, k_chunks, m_tiles, tiles, wait_limit;
    int *error;
    const int32_t *expert_tiles;  // rows sorted by expert: the token tiles (qk_route); null: one matrix
};
// Tile `tile` of the walk over weight tiles and, fastest, the token tiles that share one; with experts
// the walk goes from expert to expert.
struct TcTile {
    uint32_t t0, t_end, n0, w0;  // rows of x, first output column, first row of W
};
template <int BN>
__device__ __forceinline__ TcTile tc_tile(const TcArgs &g, uint32_t tile) {
    if (!g.expert_tiles) {
        const uint32_t n0 = (tile / g.m_tiles) * BN;
        return {(tile % g.m_tiles) * kTcM, g.n_tokens, n0, n0};
    }
    const uint32_t per_row = (g.rows + BN - 1) / BN;
    const int32_t *any = g.expert_tiles + 1 + kRouteTile * (tile / per_row);  // (a tile of the same expert)
    const uint32_t first = (uint32_t)any[3], count = (uint32_t)any[4], at = tile - first * per_row, n0 = at / count * BN;
    const int32_t *e = g.expert_tiles + 1 + kRouteTile * (first + at % count);
    return {(uint32_t)e[1], (uint32_t)e[2], n0, (uint32_t)e[0] * g.rows + n0};
}
__device__ __forceinline__ uint32_t tc_idesc(uint32_t bn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((bn >> 3) << 17) | ((uint32_t)(kTcM >> 4) << 24);
}
__device__ __forceinline__ bool tc_epilogue_vote(bool ok) {
    uint32_t all;
    asm volatile(
        "{\n .reg .pred p, q;\n setp.ne.b32 p, %1, 0;\n"
        " barrier.cta.red.and.pred q, 1, %2, p;\n selp.u32 %0, 1, 0, q;\n}"
        : "=r"(all)
        : "r"((uint32_t)ok), "r"(kTcEpiWarps * 32)
        : "memory");
    return all != 0;
}

// 16 consecutive 32-bit columns of this thread's tensor-memory lane.
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
          "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
        : "r"(taddr)
        : "memory");
}

// A warp's 32 rows x 32 columns go through shared memory, so that eight lanes hold 32 consecutive
// columns of a row, four each: whole lines for every load and store of the epilogue.
constexpr int kEpiPitch = 36;  // floats per staged row
// Element by element: unaligned buffers and ragged column ends.  Out of line, so that the usual
// path stays short enough for the instruction cache.
__device__ __noinline__ void tc_store_slow(const OutputArgs &o, uint32_t t0, uint32_t n_tokens, uint32_t n0, uint32_t limit,
                                           const float *stage, uint32_t lane, bool raw) {
    for (uint32_t r = 0; r < 32 && t0 + r < n_tokens; ++r)
        if (n0 + lane < limit) {
            const float v = stage[r * kEpiPitch + lane];
            if (raw) put(o.out, o.out_bf16, (size_t)(t0 + r) * o.out_stride + n0 + lane, v);
            else finish(o, t0 + r, n0 + lane, v);
        }
}
template <int KIND>
__device__ __forceinline__ void tc_store_tile(const OutputArgs &o, uint32_t t0, uint32_t n_tokens, uint32_t n0,
                                              uint32_t limit, const float (&v)[32], float *stage, uint32_t lane, bool vec) {
    __syncwarp();
#pragma unroll
    for (int j = 0; j < 32; j += 4)
        *reinterpret_cast<float4 *>(stage + lane * kEpiPitch + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
    __syncwarp();
    if (!vec || n0 + 32 > limit) {
        tc_store_slow(o, t0, n_tokens, n0, limit, stage, lane, KIND == QK_OUTPUT_GLU);
        return;
    }
    const uint32_t c = (lane % 8) * 4, n = n0 + c;
    float4 scale = make_float4(1.f, 1.f, 1.f, 1.f);
    float4 old[KIND == QK_OUTPUT_RESIDUAL ? 8 : 1];
    if constexpr (KIND == QK_OUTPUT_RESIDUAL) {
        if (o.scale) scale = *reinterpret_cast<const float4 *>(o.scale + n);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const uint32_t t = min(t0 + i * 4 + lane / 8, n_tokens - 1);
            old[i] = *reinterpret_cast<const float4 *>(o.residual + (size_t)t * o.residual_stride + n);
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const uint32_t r = i * 4 + lane / 8, t = t0 + r;
        if (t >= n_tokens) continue;
        float4 x = *reinterpret_cast<const float4 *>(stage + r * kEpiPitch + c);
        if constexpr (KIND == QK_OUTPUT_RESIDUAL) {
            x = make_float4(fmaf(x.x, scale.x, old[i].x), fmaf(x.y, scale.y, old[i].y), fmaf(x.z, scale.z, old[i].z),
                            fmaf(x.w, scale.w, old[i].w));
            *reinterpret_cast<float4 *>(o.residual + (size_t)t * o.residual_stride + n) = x;
            if (!o.out) continue;
        } else if constexpr (KIND == QK_OUTPUT_SIDE) {
            x = make_float4(activate(o.act, x.x) * side_value(o, t, n), activate(o.act, x.y) * side_value(o, t, n + 1),
                            activate(o.act, x.z) * side_value(o, t, n + 2), activate(o.act, x.w) * side_value(o, t, n + 3));
        }
        const size_t at = (size_t)t * o.out_stride + n;
        if (o.out_bf16) {
            const uint32_t lo = (uint32_t)float_to_bf16_bits(x.x) | ((uint32_t)float_to_bf16_bits(x.y) << 16);
            const uint32_t hi = (uint32_t)float_to_bf16_bits(x.z) | ((uint32_t)float_to_bf16_bits(x.w) << 16);
            *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(o.out) + at) = make_uint2(lo, hi);
        } else {
            *reinterpret_cast<float4 *>(static_cast<float *>(o.out) + at) = x;
        }
    }
}

template <int BN, int KIND>
__global__ void __launch_bounds__(kTcThreads, 1)
dense_tc_kernel(const __grid_constant__ CUtensorMap x_map, const __grid_constant__ CUtensorMap w_map, TcArgs g,
                OutputArgs out, int vec) {
    using S = TcShape<BN>;
    qk::pdl_launch();
    extern __shared__ __align__(1024) uint8_t tc_smem[];
    uint8_t *tiles = reinterpret_cast<uint8_t *>(((uintptr_t)tc_smem + 1023) & ~(uintptr_t)1023);
    float *epi = reinterpret_cast<float *>(tiles + S::kStages * S::kStage);  // [epilogue warp][32][kEpiPitch]
    uint64_t *full = reinterpret_cast<uint64_t *>(epi + kTcEpiWarps * 32 * kEpiPitch);
    uint64_t *empty = full + S::kStages;
    uint64_t *acc_full = empty + S::kStages;
    uint64_t *acc_empty = acc_full + 2;
    uint64_t *drain = acc_empty + 2;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(drain + 1);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    volatile int *never = reinterpret_cast<volatile int *>(tmem_slot + 2);
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    if (threadIdx.x == 0) {
        for (int s = 0; s < S::kStages; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        for (int a = 0; a < 2; ++a) {
            mbar_init(&acc_full[a], 1);
            mbar_init(&acc_empty[a], kTcEpiWarps);
        }
        mbar_init(drain, 1);
        *abort_flag = 0;
        *never = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&x_map) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&w_map) : "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)),
                     "r"(S::kTmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    qk::pdl_wait();
    const uint32_t tmem_base = *tmem_slot;
    const uint32_t n_tiles = g.expert_tiles ? (uint32_t)g.expert_tiles[0] * ((g.rows + BN - 1) / BN) : g.tiles;

    if (warp == 0) {
        uint32_t gc = 0;
        bool dead = false;
        for (uint32_t tile = blockIdx.x; tile < n_tiles && !dead; tile += gridDim.x) {
            const TcTile at = tc_tile<BN>(g, tile);
            for (uint32_t kc = 0; kc < g.k_chunks; ++kc, ++gc) {
                const uint32_t s = gc % S::kStages;
                if (!mbar_wait(&empty[s], ((gc / S::kStages) & 1) ^ 1, abort_flag, g.wait_limit)) {
                    dead = true;
                    break;
                }
                if (lane == 0) {
                    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(&full[s])),
                                 "r"(S::kStage)
                                 : "memory");
                    const uint32_t a = smem_u32(tiles + s * S::kStage);
                    tma_load_2d(a, &x_map, kc * kTcK, at.t0, &full[s]);
                    tma_load_2d(a + S::kABytes, &w_map, kc * kTcK, at.w0, &full[s]);
                }
                __syncwarp();
            }
        }
        if (dead) {
            *abort_flag = 1;
            // the copies still in flight
            for (uint32_t i = gc > (uint32_t)S::kStages ? gc - S::kStages : 0; i < gc; ++i)
                (void)mbar_wait(&full[i % S::kStages], (i / S::kStages) & 1, never, g.wait_limit);
        } else if (*abort_flag) {
            for (uint32_t i = gc > (uint32_t)S::kStages ? gc - S::kStages : 0; i < gc; ++i)
                (void)mbar_wait(&full[i % S::kStages], (i / S::kStages) & 1, never, g.wait_limit);
        }
    } else if (warp == 1) {
        const uint32_t idesc = tc_idesc(BN);
        uint32_t gc = 0, seg = 0;
        bool dead = false;
        for (uint32_t tile = blockIdx.x; tile < n_tiles && !dead; tile += gridDim.x, ++seg) {
            const uint32_t acc = seg & 1;
            if (!mbar_wait(&acc_empty[acc], ((seg >> 1) & 1) ^ 1, abort_flag, g.wait_limit)) {
                dead = true;
                break;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t d_tmem = tmem_base + acc * BN;
            for (uint32_t kc = 0; kc < g.k_chunks; ++kc, ++gc) {
                const uint32_t s = gc % S::kStages;
                if (!mbar_wait(&full[s], (gc / S::kStages) & 1, abort_flag, g.wait_limit)) {
                    dead = true;
                    break;
                }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lane == 0) {
                    const uint32_t a_addr = smem_u32(tiles + s * S::kStage), b_addr = a_addr + S::kABytes;
#pragma unroll
                    for (int k = 0; k < kTcK / 16; ++k) {
                        const uint64_t ad = umma_desc(a_addr + k * 32), bd = umma_desc(b_addr + k * 32);
                        const uint32_t accumulate = (kc != 0 || k != 0) ? 1u : 0u;
                        asm volatile(
                            "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
                            " tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}" ::"r"(d_tmem),
                            "l"(ad), "l"(bd), "r"(idesc), "r"(accumulate)
                            : "memory");
                    }
                    umma_commit(&empty[s]);
                }
                __syncwarp();
            }
            if (!dead && lane == 0) umma_commit(&acc_full[acc]);
            __syncwarp();
        }
        if (dead) {
            *abort_flag = 1;
            if (lane == 0) umma_commit(drain);  // the products still in flight
            __syncwarp();
            (void)mbar_wait(drain, 0, never, g.wait_limit);
        }
    } else {
        const uint32_t quarter = warp % 4;
        uint32_t seg = 0;
        for (uint32_t tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++seg) {
            const uint32_t acc = seg & 1;
            const TcTile at = tc_tile<BN>(g, tile);
            const uint32_t t0 = at.t0 + quarter * 32, n0 = at.n0;
            float *stage = epi + (warp - 2) * 32 * kEpiPitch;
            if (!tc_epilogue_vote(mbar_wait(&acc_full[acc], (seg >> 1) & 1, abort_flag, g.wait_limit))) {
                *abort_flag = 1;
                break;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t lane_addr = tmem_base + acc * BN + ((quarter * 32) << 16);
#pragma unroll 1
            for (uint32_t c = 0; c < BN && n0 + c < g.rows; c += KIND == QK_OUTPUT_GLU ? 64 : 32) {  // warp-uniform
                uint32_t a[32];
                float v[32];
                tmem_ld32(lane_addr + c, a);
                if constexpr (KIND == QK_OUTPUT_GLU) {
                    uint32_t b[32];
                    tmem_ld32(lane_addr + c + 32, b);
                    tmem_ld_wait();
                    if (out.act == QK_ACT_RELU) {
#pragma unroll
                        for (int j = 0; j < 32; ++j) v[j] = fmaxf(__uint_as_float(a[j]), 0.f) * __uint_as_float(b[j]);
                    } else if (out.act == QK_ACT_SILU) {
#pragma unroll
                        for (int j = 0; j < 32; ++j) v[j] = silu_f(__uint_as_float(a[j])) * __uint_as_float(b[j]);
                    } else {
#pragma unroll
                        for (int j = 0; j < 32; ++j) v[j] = gelu_tanh_f(__uint_as_float(a[j])) * __uint_as_float(b[j]);
                    }
                    tc_store_tile<KIND>(out, t0, at.t_end, (n0 + c) / 2, g.rows / 2, v, stage, lane, vec != 0);
                } else {
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; ++j) v[j] = __uint_as_float(a[j]);
                    tc_store_tile<KIND>(out, t0, at.t_end, n0 + c, g.rows, v, stage, lane, vec != 0);
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[acc]);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(S::kTmemCols)
                     : "memory");
    if (threadIdx.x == 0 && *abort_flag) atomicOr(g.error, 1);
}

// The same rows for a normed or concatenated input whose rows are 16-byte aligned, bfloat16 out: a
// thread keeps its kV pieces of four entries in registers, all loads of the row go out together.
template <int kV>
__global__ void __launch_bounds__(256)
dense_norm_rows_kernel(InputArgs in, uint16_t *__restrict__ dst) {
    qk::pdl_launch();
    qk::pdl_wait();
    __shared__ float red[8];
    const uint32_t t = blockIdx.x, n = in.width, pieces = n / 4;
    const float4 *xr = reinterpret_cast<const float4 *>(in.x + (size_t)t * in.x_stride);
    float4 h[kV];
#pragma unroll
    for (int j = 0; j < kV; ++j) {
        const uint32_t p = threadIdx.x + 256 * j;
        h[j] = p < pieces ? xr[p] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (in.pending) {
        const uint32_t parts = in.pending_top ? in.pending_top : 1;
        float4 y[kV];
        float ps = 0.f;
        for (uint32_t c = 0; c < parts; ++c) {
            const float4 *pr = reinterpret_cast<const float4 *>(
                in.pending_top ? pending_row(in, t, c) : in.pending + (size_t)t * in.pending_stride);
#pragma unroll
            for (int j = 0; j < kV; ++j) {
                const uint32_t p = threadIdx.x + 256 * j;
                const float4 v = p < pieces ? pr[p] : make_float4(0.f, 0.f, 0.f, 0.f);
                y[j] = c ? make_float4(y[j].x + v.x, y[j].y + v.y, y[j].z + v.z, y[j].w + v.w) : v;
            }
        }
        const float share = in.pending_top ? in.pending_scale : 1.f;
#pragma unroll
        for (int j = 0; j < kV; ++j) {
            y[j] = make_float4(y[j].x * share, y[j].y * share, y[j].z * share, y[j].w * share);
            ps += y[j].x * y[j].x + y[j].y * y[j].y + y[j].z * y[j].z + y[j].w * y[j].w;
        }
        const float inv = 1.0f / sqrtf(in_block_sum(ps, red) / (float)n + in.pending_eps);
        const float4 *pw = reinterpret_cast<const float4 *>(in.pending_weight);
        float4 *xo = in.x_out ? reinterpret_cast<float4 *>(in.x_out + (size_t)t * in.x_stride) : nullptr;
#pragma unroll
        for (int j = 0; j < kV; ++j) {
            const uint32_t p = threadIdx.x + 256 * j;
            if (p >= pieces) continue;
            const float4 w = pw[p];
            h[j].x += y[j].x * inv * w.x;
            h[j].y += y[j].y * inv * w.y;
            h[j].z += y[j].z * inv * w.z;
            h[j].w += y[j].w * inv * w.w;
            if (xo) xo[p] = h[j];
        }
    }
    float mean = 0.f, inv = 1.f;
    if (in.norm == QK_NORM_LAYER) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < kV; ++j) s += h[j].x + h[j].y + h[j].z + h[j].w;
        mean = in_block_sum(s, red) / (float)n;
    }
    if (in.norm != QK_NORM_NONE) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < kV; ++j) {
            if (threadIdx.x + 256 * j >= pieces) continue;
            const float a = h[j].x - mean, b = h[j].y - mean, c = h[j].z - mean, d = h[j].w - mean;
            s += a * a + b * b + c * c + d * d;
        }
        inv = 1.0f / sqrtf(in_block_sum(s, red) / (float)n + in.norm_eps);
    }
    const uint32_t copies = in.places ? in.top : 1;
    const float4 *nw = reinterpret_cast<const float4 *>(in.norm_weight);
    const uint32_t half = (in.kind == QK_INPUT_CONCAT ? in.k / 2 : in.k) / 4;
    const float4 *second = reinterpret_cast<const float4 *>(in.second ? in.second + (size_t)t * in.x_stride : nullptr);
    auto pack = [](float4 v) {
        return make_uint2((uint32_t)float_to_bf16_bits(v.x) | ((uint32_t)float_to_bf16_bits(v.y) << 16),
                          (uint32_t)float_to_bf16_bits(v.z) | ((uint32_t)float_to_bf16_bits(v.w) << 16));
    };
#pragma unroll
    for (int j = 0; j < kV; ++j) {
        const uint32_t p = threadIdx.x + 256 * j;
        if (p >= half) continue;  // (pieces past the width are zeros)
        float4 v = h[j];
        if (in.norm != QK_NORM_NONE && p < pieces) {
            const float4 w = nw[p];
            v = make_float4((v.x - mean) * inv * w.x, (v.y - mean) * inv * w.y, (v.z - mean) * inv * w.z,
                            (v.w - mean) * inv * w.w);
        }
        for (uint32_t c = 0; c < copies; ++c) {
            uint2 *o = reinterpret_cast<uint2 *>(dst + (size_t)(in.places ? (uint32_t)in.places[t * in.top + c] : t) * in.k);
            o[p] = pack(v);
            if (in.kind == QK_INPUT_CONCAT) o[half + p] = pack(p < pieces ? second[p] : make_float4(0.f, 0.f, 0.f, 0.f));
        }
    }
    if (in.append.src) append_latent(in, t, red);
}

// ------------------------------------------------------------------ narrow form
// Few rows of x (a decode batch): the weights take the M side (128 weight rows per CTA), the rows of
// x the N side, so that a weight byte is read once and the product is bound by reading it.  The k
// range of a tile is shared out over the CTAs of a cluster (up to eight), which then add their
// float32 accumulators through distributed shared memory, each CTA finishing its share of the
// columns.  Weights depend on no other kernel: the first stages' copies start before the
// dependency wait.  Warp 0 issues the copies, warp 1 the MMAs, warps 2..5 finish.
template <int BN> struct NarrowShape {
    static constexpr uint32_t kABytes = 128 * kTcK * 2, kBBytes = BN * kTcK * 2, kStage = kABytes + kBBytes;
    static constexpr int kStages = BN >= 128 ? 6 : 8;
    static constexpr uint32_t kTmemCols = BN < 32 ? 32 : BN;
    static constexpr size_t kSmem = 1024 + kStages * kStage + (2 * kStages + 2) * 8 + 32;
    static_assert(128 * BN * 4 + 2 * 32 * BN * 4 <= kStages * kStage, "the accumulators must fit the drained stages");
};
struct NarrowArgs {
    uint32_t n_tokens, rows, k_chunks, splits, wait_limit;
    int *error;
    const int32_t *offsets;  // rows sorted by expert: [experts + 1]; null: one matrix
    uint32_t tiles;          // weight tiles of an expert
};
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int BN>
__global__ void __launch_bounds__(kTcThreads, 1)
dense_narrow_kernel(const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map,
                    NarrowArgs g, OutputArgs out) {
    using S = NarrowShape<BN>;
    qk::pdl_launch();
    extern __shared__ __align__(1024) uint8_t nr_smem[];
    uint8_t *tiles = reinterpret_cast<uint8_t *>(((uintptr_t)nr_smem + 1023) & ~(uintptr_t)1023);
    uint64_t *full = reinterpret_cast<uint64_t *>(tiles + S::kStages * S::kStage);
    uint64_t *empty = full + S::kStages;
    uint64_t *acc_full = empty + S::kStages;
    uint64_t *drain = acc_full + 1;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(drain + 1);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    volatile int *never = reinterpret_cast<volatile int *>(tmem_slot + 2);
    const uint32_t warp = threadIdx.x / 32, lane = threadIdx.x % 32;
    uint32_t tile = blockIdx.x / g.splits;  // (a cluster is one tile)
    const uint32_t split = blockIdx.x % g.splits;
    uint32_t t0 = 0, n_rows = g.n_tokens, w0 = tile * 128;  // rows of x, first row of W
    if (g.offsets) {
        // (qk_route lets nothing start early: the offsets may be read before the dependency wait)
        const uint32_t e = tile / g.tiles;
        tile %= g.tiles;
        t0 = (uint32_t)g.offsets[e];
        n_rows = (uint32_t)g.offsets[e + 1] - t0;
        w0 = e * g.rows + tile * 128;
        if (n_rows == 0) {  // (the same for the whole cluster)
            qk::pdl_wait();
            return;
        }
    }
    const uint32_t per = (g.k_chunks + g.splits - 1) / g.splits;
    const uint32_t kc0 = min(split * per, g.k_chunks), kc1 = min(kc0 + per, g.k_chunks);
    if (threadIdx.x == 0) {
        for (int s = 0; s < S::kStages; ++s) {
            mbar_init(&full[s], 1);
            mbar_init(&empty[s], 1);
        }
        mbar_init(acc_full, 1);
        mbar_init(drain, 1);
        *abort_flag = 0;
        *never = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)),
                     "r"(S::kTmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t ahead = min((uint32_t)S::kStages, kc1 - kc0);
    if (warp == 0 && lane == 0)
        for (uint32_t i = 0; i < ahead; ++i) {
            asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(&full[i])),
                         "r"(S::kStage)
                         : "memory");
            tma_load_2d(smem_u32(tiles + i * S::kStage), &w_map, (kc0 + i) * kTcK, w0, &full[i]);
        }
    qk::pdl_wait();
    const uint32_t tmem_base = *tmem_slot;
    bool finished = true;  // (epilogue warps: the accumulator is complete)

    if (warp == 0) {
        uint32_t gc = 0;
        bool dead = false;
        for (uint32_t kc = kc0; kc < kc1; ++kc, ++gc) {
            const uint32_t s = gc % S::kStages;
            if (gc >= ahead && !mbar_wait(&empty[s], ((gc / S::kStages) & 1) ^ 1, abort_flag, g.wait_limit)) {
                dead = true;
                break;
            }
            if (lane == 0) {
                const uint32_t a = smem_u32(tiles + s * S::kStage);
                if (gc >= ahead) {
                    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(&full[s])),
                                 "r"(S::kStage)
                                 : "memory");
                    tma_load_2d(a, &w_map, kc * kTcK, w0, &full[s]);
                }
                tma_load_2d(a + S::kABytes, &x_map, kc * kTcK, t0, &full[s]);
            }
            __syncwarp();
        }
        if (dead) *abort_flag = 1;
        if (*abort_flag)  // the copies still in flight
            for (uint32_t i = gc > (uint32_t)S::kStages ? gc - S::kStages : 0; i < gc; ++i)
                (void)mbar_wait(&full[i % S::kStages], (i / S::kStages) & 1, never, g.wait_limit);
    } else if (warp == 1) {
        const uint32_t idesc = tc_idesc(BN);
        uint32_t gc = 0;
        bool dead = false;
        for (uint32_t kc = kc0; kc < kc1; ++kc, ++gc) {
            const uint32_t s = gc % S::kStages;
            if (!mbar_wait(&full[s], (gc / S::kStages) & 1, abort_flag, g.wait_limit)) {
                dead = true;
                break;
            }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (lane == 0) {
                const uint32_t a_addr = smem_u32(tiles + s * S::kStage), b_addr = a_addr + S::kABytes;
#pragma unroll
                for (int k = 0; k < kTcK / 16; ++k) {
                    const uint64_t ad = umma_desc(a_addr + k * 32), bd = umma_desc(b_addr + k * 32);
                    const uint32_t accumulate = (gc != 0 || k != 0) ? 1u : 0u;
                    asm volatile(
                        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
                        " tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}" ::"r"(tmem_base),
                        "l"(ad), "l"(bd), "r"(idesc), "r"(accumulate)
                        : "memory");
                }
                umma_commit(&empty[s]);
            }
            __syncwarp();
        }
        if (!dead && lane == 0) umma_commit(acc_full);
        __syncwarp();
        if (dead) {
            *abort_flag = 1;
            if (lane == 0) umma_commit(drain);  // the products still in flight
            __syncwarp();
            (void)mbar_wait(drain, 0, never, g.wait_limit);
        }
    } else {
        finished = tc_epilogue_vote(mbar_wait(acc_full, 0, abort_flag, g.wait_limit));
        if (!finished) *abort_flag = 1;
    }
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t quarter = warp % 4, row = quarter * 32 + lane;
    float *own = reinterpret_cast<float *>(tiles);  // [BN][128]: the drained stages
    if (g.splits > 1) {
        if (warp >= 2 && finished) {
            const uint32_t lane_addr = tmem_base + ((quarter * 32) << 16);
#pragma unroll
            for (int c0 = 0; c0 < BN; c0 += 16) {
                uint32_t v[16];
                tmem_ld16(lane_addr + c0, v);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 16; ++j)
                    own[(c0 + j) * 128 + row] = kc1 > kc0 ? __uint_as_float(v[j]) : 0.f;
            }
        }
        __syncwarp();
        cluster_sync_all();  // every CTA of the tile has its accumulator in shared memory
    }
    if (warp >= 2 && finished) {
        const bool pair = out.kind == QK_OUTPUT_GLU;
        const uint32_t share = (BN + g.splits - 1) / g.splits;  // columns this CTA finishes
        const uint32_t c_begin = split * share, c_end = min(min(c_begin + share, (uint32_t)BN), n_rows);
        float *ups = own + 128 * BN;  // [2][BN][32]: up rows for their gate rows
        const uint32_t n = tile * 128 + row, lane_addr = tmem_base + ((quarter * 32) << 16);
        auto value = [&](uint32_t c) -> float {  // (splits > 1) the sum over the cluster, in split order
            float v = 0.f;
            for (uint32_t p = 0; p < g.splits; ++p) {
                uint32_t remote;
                float x;
                asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(smem_u32(own + c * 128 + row)), "r"(p));
                asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(x) : "r"(remote) : "memory");
                v += x;
            }
            return v;
        };
        auto done = [&](uint32_t c, float v) {
            if (pair) {
                if (quarter & 1) ups[((quarter >> 1) * BN + c) * 32 + lane] = v;
            } else if (n < g.rows) {
                finish(out, t0 + c, n, v);
            }
        };
        float kept[BN <= 64 ? BN : 1];  // a gate row's values until its up row's arrive
        if (g.splits == 1) {
#pragma unroll
            for (int c0 = 0; c0 < BN; c0 += 16) {
                if ((uint32_t)c0 >= c_end) break;
                uint32_t v[16];
                tmem_ld16(lane_addr + c0, v);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    if constexpr (BN <= 64) kept[c0 + j] = __uint_as_float(v[j]);
                    if ((uint32_t)(c0 + j) < c_end) done(c0 + j, __uint_as_float(v[j]));
                }
            }
        } else if (!pair) {
#pragma unroll 4
            for (uint32_t c = c_begin; c < c_end; ++c) done(c, value(c));
        } else if (quarter & 1) {
#pragma unroll 4
            for (uint32_t c = c_begin; c < c_end; ++c) done(c, value(c));
        }
        if (pair) {
            asm volatile("bar.sync 1, %0;" ::"r"(kTcEpiWarps * 32) : "memory");
            const uint32_t j = tile * 64 + (quarter >> 1) * 32 + lane;
            if (!(quarter & 1) && j < g.rows / 2) {
                if (g.splits == 1) {
#pragma unroll
                    for (int c0 = 0; c0 < BN; c0 += 16) {
                        if ((uint32_t)c0 >= c_end) break;
                        uint32_t v[16];
                        if constexpr (BN > 64) {
                            tmem_ld16(lane_addr + c0, v);
                            tmem_ld_wait();
                        }
#pragma unroll
                        for (int e = 0; e < 16; ++e) {
                            const uint32_t c = c0 + e;
                            float gate;
                            if constexpr (BN > 64) gate = __uint_as_float(v[e]);
                            else gate = kept[c0 + e];
                            if (c < c_end) finish_pair(out, t0 + c, j, gate, ups[((quarter >> 1) * BN + c) * 32 + lane]);
                        }
                    }
                } else {
#pragma unroll 4
                    for (uint32_t c = c_begin; c < c_end; ++c)
                        finish_pair(out, t0 + c, j, value(c), ups[((quarter >> 1) * BN + c) * 32 + lane]);
                }
            }
        }
    }
    __syncwarp();
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    if (g.splits > 1) cluster_sync_all();  // no CTA leaves while another still reads its shared memory
    else __syncthreads();
    if (warp == 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(S::kTmemCols)
                     : "memory");
    if (threadIdx.x == 0 && *abort_flag) atomicOr(g.error, 1);
}

// rows x k bfloat16 entries, `stride` entries from row to row; boxes of 64 k x box_rows.
qk_status encode_map(const void *base, size_t rows, size_t k, size_t stride, uint32_t box_rows, CUtensorMap *out) {
    const cuuint64_t dims[2] = {k, rows}, strides[1] = {stride * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kTcK, box_rows};
    return encode_bf16_map(base, 2, dims, strides, box, out);
}

// Rows of x and of W as the matrix forms see them, and their row tiles.
size_t input_rows(const qk_dense_call &d) { return d.experts ? d.tokens * d.top : d.tokens; }
size_t weight_rows(const qk_dense_call &d) { return d.experts ? d.rows * d.experts : d.rows; }
size_t row_tiles(const qk_dense_call &d, size_t tile) {
    return qk::ceil_div(input_rows(d), tile) + (d.experts ? std::min(d.experts, input_rows(d)) : 0);
}

// Weight rows per tile: the width whose number of waves over the SMs costs least.
int pick_tile(size_t m_tiles, size_t rows, size_t sms) {
    int best = 64;
    size_t best_cost = ~(size_t)0;
    for (int bn : {256, 128, 64}) {
        const size_t waves = qk::ceil_div(m_tiles * qk::ceil_div(rows, bn), sms);
        const size_t cost = waves * (bn + 48);  // (48: what a tile costs whatever its width)
        if (cost < best_cost) best = bn, best_cost = cost;
    }
    return best;
}

template <int BN, int KIND>
qk_status launch_tc_kind(qk_ctx *c, const void *x, size_t x_stride, const qk_dense_call &d, const OutputArgs &out,
                    int vec) {
    using S = TcShape<BN>;
    CUtensorMap xm, wm;
    qk_status st;
    if ((st = encode_map(x, input_rows(d), d.k, x_stride, kTcM, &xm)) != QK_OK) return st;
    if ((st = encode_map(d.w, weight_rows(d), d.k, d.w_stride, BN, &wm)) != QK_OK) return st;
    TcArgs g{};
    g.n_tokens = (uint32_t)d.tokens;
    g.rows = (uint32_t)d.rows;
    g.k_chunks = (uint32_t)qk::ceil_div(d.k, kTcK);
    g.m_tiles = (uint32_t)row_tiles(d, kTcM);  // (with experts: the most there can be)
    g.tiles = g.m_tiles * (uint32_t)qk::ceil_div(d.rows, BN);
    g.expert_tiles = d.experts ? d.tiles : nullptr;
    g.wait_limit = c->wait_limit ? c->wait_limit : kTcWaitDefault;
    g.error = (int *)c->d_err.ptr;
    QK_CUDA(cudaFuncSetAttribute((dense_tc_kernel<BN, KIND>), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::kSmem));
    (void)qk::launch_pdl(c->pdl, (dense_tc_kernel<BN, KIND>), dim3(std::min(g.tiles, (uint32_t)c->sm_count)),
                         dim3(kTcThreads), S::kSmem, c->stream, xm, wm, g, out, vec);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    c->err_armed = true;
    return QK_OK;
}

// CTAs per tile: enough to occupy the SMs without splitting the k range finer than four chunks.
uint32_t narrow_splits(size_t tiles, size_t k_chunks, size_t sms) {
    uint32_t best = 1;
    size_t best_cost = ~(size_t)0;
    for (uint32_t s : {1u, 2u, 4u, 8u}) {
        if (s > 1 && k_chunks / s < 4) break;
        // (a cluster of CTAs does not find room on every SM)
        const size_t room = s == 1 ? sms : s == 2 ? sms - 4 : sms - 20;
        const size_t waves = qk::ceil_div(tiles * s, room);
        const size_t cost = waves * (qk::ceil_div(k_chunks, s) + 10) + (s > 1 ? 6 : 0);
        if (cost < best_cost) best = s, best_cost = cost;
    }
    return best;
}

template <int BN>
qk_status launch_narrow(qk_ctx *c, const void *x, size_t x_stride, const qk_dense_call &d, const OutputArgs &out) {
    using S = NarrowShape<BN>;
    CUtensorMap xm, wm;
    qk_status st;
    if ((st = encode_map(x, input_rows(d), d.k, x_stride, BN, &xm)) != QK_OK) return st;
    if ((st = encode_map(d.w, weight_rows(d), d.k, d.w_stride, 128, &wm)) != QK_OK) return st;
    NarrowArgs g{};
    g.n_tokens = (uint32_t)d.tokens;
    g.rows = (uint32_t)d.rows;
    g.k_chunks = (uint32_t)qk::ceil_div(d.k, kTcK);
    const uint32_t per_matrix = (uint32_t)qk::ceil_div(d.rows, 128);
    const uint32_t tiles = per_matrix * (uint32_t)(d.experts ? d.experts : 1);
    g.offsets = d.experts ? d.offsets : nullptr;
    g.tiles = per_matrix;
    g.splits = narrow_splits(per_matrix * (d.experts ? std::min(d.experts, input_rows(d)) : 1), g.k_chunks,
                             (size_t)c->sm_count);
    g.wait_limit = c->wait_limit ? c->wait_limit : kTcWaitDefault;
    g.error = (int *)c->d_err.ptr;
    QK_CUDA(cudaFuncSetAttribute(dense_narrow_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::kSmem));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles * g.splits);
    cfg.blockDim = dim3(kTcThreads);
    cfg.dynamicSmemBytes = S::kSmem;
    cfg.stream = c->stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = c->pdl ? 1 : 0;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = g.splits;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    QK_CUDA(cudaLaunchKernelEx(&cfg, dense_narrow_kernel<BN>, wm, xm, g, out));
    c->launches++;
    c->err_armed = true;
    return QK_OK;
}

template <int BN>
qk_status launch_tc(qk_ctx *c, const void *x, size_t x_stride, const qk_dense_call &d, const OutputArgs &out, int vec) {
    switch (d.output) {
        case QK_OUTPUT_RESIDUAL: return launch_tc_kind<BN, QK_OUTPUT_RESIDUAL>(c, x, x_stride, d, out, vec);
        case QK_OUTPUT_GLU: return launch_tc_kind<BN, QK_OUTPUT_GLU>(c, x, x_stride, d, out, vec);
        case QK_OUTPUT_SIDE: return launch_tc_kind<BN, QK_OUTPUT_SIDE>(c, x, x_stride, d, out, vec);
        default: return launch_tc_kind<BN, QK_OUTPUT_STORE>(c, x, x_stride, d, out, vec);
    }
}

// Which of the faster ways to read the input rows applies.
int row_kind_of(const InputArgs &a) {
    auto aligned = [](const void *p) { return ((uintptr_t)p & 15) == 0; };
    if (a.width % 4 || a.k % 4 || a.x_stride % 4 || !aligned(a.x)) return kRowAny;
    if (a.kind == QK_INPUT_PLAIN) return kRowPlain;
    if (a.kind != QK_INPUT_NORM || a.width > 1024 * kNormPieces || !aligned(a.x_out)) return kRowAny;
    if (a.norm != QK_NORM_NONE && !aligned(a.norm_weight)) return kRowAny;
    if (a.pending && (a.pending_stride % 4 || !aligned(a.pending) || !aligned(a.pending_weight))) return kRowAny;
    return kRowNorm;
}

template <typename W, int NT, int R>
qk_status launch_vector_r(qk_ctx *c, const InputArgs &in, const OutputArgs &out, const qk_dense_call &d,
                          size_t n_tokens, uint32_t ks) {
    const size_t step = VecTraits<W>::kStep;
    int kind = row_kind_of(in);
    size_t smem = NT * qk::ceil_div(d.k, step) * step * 4;
    if (kind == kRowNorm && smem + 8 * d.width > kVecSmemMax) kind = kRowAny;
    if (kind == kRowNorm) smem += 8 * d.width;
    const size_t groups = d.output == QK_OUTPUT_GLU ? qk::ceil_div(d.rows / 2, R / 2 ? R / 2 : 1)
                                                    : qk::ceil_div(d.rows, R);
    QK_CUDA(cudaFuncSetAttribute(dense_vector_kernel<W, NT, R>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)std::max(smem, (size_t)48 * 1024)));
    ChoiceArgs ch{};
    if (d.experts) ch = ChoiceArgs{d.table, d.ids, (uint32_t)d.top, (uint32_t)d.vocab, d.by_choice ? 1u : 0u};
    const size_t choices = d.experts ? input_rows(d) : 1;
    // the blocks that stay resident, shared out evenly among the choices
    const size_t per_sm = std::max<size_t>(1, std::min<size_t>(vec_blocks(NT, R), kVecSmemSm / (smem + 2048)));
    const size_t resident = std::max<size_t>(1, per_sm * (size_t)c->sm_count / choices);
    (void)qk::launch_pdl(c->pdl, dense_vector_kernel<W, NT, R>, dim3((unsigned)std::min(groups, resident), (unsigned)choices),
                         dim3(kVecThreads), smem, c->stream, in, out, (const W *)d.w, (uint32_t)d.rows,
                         (uint32_t)d.w_stride, (uint32_t)n_tokens, ks, ch, kind);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
}
template <typename W, int NT>
qk_status launch_vector(qk_ctx *c, const InputArgs &in, const OutputArgs &out, const qk_dense_call &d,
                        size_t n_tokens) {
    // rows per warp and warps per row group
    const size_t steps = qk::ceil_div(d.k, VecTraits<W>::kStep);
    const bool pair = d.output == QK_OUTPUT_GLU;
    if (d.experts) {
        // The blocks are shared out among the choices, so that a few turns over the rows are usual: what
        // takes the fewest batches of four steps one after the other (a turn costs a little on its own).
        const size_t choices = input_rows(d);
        int best_r = 2;
        uint32_t best_ks = 1;
        size_t best_cost = ~(size_t)0;
        for (int r = pair ? 2 : 1; r <= 2; ++r) {
            const size_t warps = std::max<size_t>(1, (size_t)vec_blocks(NT, r) * (size_t)c->sm_count / choices) * kVecWarps;
            const size_t groups = pair ? d.rows / 2 : qk::ceil_div(d.rows, r);
            for (uint32_t ks = 1; ks <= (uint32_t)kVecWarps && (ks == 1 || ks * 2 <= steps); ks *= 2) {
                const size_t turns = qk::ceil_div(groups * ks, warps), batches = qk::ceil_div(steps, 4 * ks);
                const size_t cost = turns * (4 * batches + (ks > 1 ? 2 : 1));
                if (cost < best_cost) best_r = r, best_ks = ks, best_cost = cost;
            }
        }
        return best_r == 2 ? launch_vector_r<W, NT, 2>(c, in, out, d, n_tokens, best_ks)
                           : launch_vector_r<W, NT, 1>(c, in, out, d, n_tokens, best_ks);
    }
    // one matrix: about two blocks per SM or more (one, where a block has a long vector to stage
    // first); measured in a whole step, splitting the k range further costs more than it evens out
    const size_t want = (d.k > 8192 ? 1 : 2) * (size_t)c->sm_count * kVecWarps;
    if (NT > 1 && d.rows / 4 >= want) return launch_vector_r<W, NT, 4>(c, in, out, d, n_tokens, 1);
    if (d.rows / 2 >= want || pair) {
        uint32_t ks = 1;
        while (ks < kVecWarps && d.rows / 2 * ks < want && ks * 4 <= steps) ks *= 2;
        return launch_vector_r<W, NT, 2>(c, in, out, d, n_tokens, ks);
    }
    uint32_t ks = 1;
    while (ks < kVecWarps && d.rows * ks < want && ks * 4 <= steps) ks *= 2;
    return launch_vector_r<W, NT, 1>(c, in, out, d, n_tokens, ks);
}

InputArgs input_args(const qk_dense_call &d) {
    InputArgs a{};
    a.x = (const float *)d.x;
    a.pending = d.pending;
    a.pending_weight = d.pending_weight;
    a.second = d.second;
    a.norm_weight = d.norm_weight;
    a.gate = d.gate;
    a.x_out = d.x_out;
    a.positions = d.positions;
    a.slots = d.slots;
    a.x_stride = (uint32_t)d.x_stride;
    a.pending_stride = (uint32_t)d.pending_stride;
    a.gate_stride = (uint32_t)d.gate_stride;
    a.width = (uint32_t)d.width;
    a.k = (uint32_t)d.k;
    a.group = (uint32_t)d.group;
    a.pending_eps = d.pending_eps;
    a.norm_eps = d.norm_eps;
    a.kind = d.input;
    a.norm = d.norm;
    a.append = AppendArgs{d.append.src, d.append.weight, d.append.cache, (uint32_t)d.append.src_stride,
                          (uint32_t)d.append.width, (uint32_t)d.append.ring, (uint32_t)d.append.stride, d.append.eps,
                          d.append.cache_dtype == QK_BF16};
    a.pending_rows = d.pending_rows;
    a.pending_top = (uint32_t)d.pending_top;
    a.pending_scale = d.pending_scale;
    return a;
}
OutputArgs output_args(const qk_dense_call &d) {
    OutputArgs o{};
    o.out = d.out;
    o.residual = d.residual;
    o.scale = d.out_scale;
    o.side = d.side;
    o.ids = d.ids;
    o.out_stride = (uint32_t)d.out_stride;
    o.residual_stride = (uint32_t)d.residual_stride;
    o.side_stride = (uint32_t)d.side_stride;
    o.side_offset = (uint32_t)d.side_offset;
    o.vocab = (uint32_t)d.vocab;
    o.kind = d.output;
    o.act = d.activation;
    o.out_bf16 = d.out_dtype == QK_BF16;
    o.side_bf16 = d.side_dtype == QK_BF16;
    return o;
}
void advance(InputArgs &a, OutputArgs &o, size_t t) {  // the same call from row t on
    a.x += t * a.x_stride;
    if (a.pending && a.pending_rows) a.pending_rows += t * a.pending_top;
    else if (a.pending) a.pending += t * (a.pending_top ? a.pending_top : 1) * a.pending_stride;
    if (a.second) a.second += t * a.x_stride;
    if (a.gate) a.gate += t * a.gate_stride;
    if (a.x_out) a.x_out += t * a.x_stride;
    if (a.positions) a.positions += t;
    if (a.slots) a.slots += t;
    if (a.append.src) a.append.src += t * a.append.src_stride;
    if (o.out) o.out = (uint8_t *)o.out + t * o.out_stride * (o.out_bf16 ? 2 : 4);
    if (o.residual) o.residual += t * o.residual_stride;
    if (o.ids) o.ids += t;
}

qk_status validate(const qk_dense_call *d, bool with_weights) {
    if (!d || !d->x) return qk::fail(QK_ERR_VALUE, "qk_dense: null argument");
    if (d->k == 0 || d->k % 8 || d->width > d->k || d->width == 0)
        return qk::fail(QK_ERR_VALUE, "qk_dense: %zu input columns for vectors of %zu (a multiple of 8 is needed)",
                        d->k, d->width);
    if (d->input < QK_INPUT_PLAIN || d->input > QK_INPUT_GATED)
        return qk::fail(QK_ERR_VALUE, "qk_dense: unknown input kind %d", d->input);
    if (d->x_dtype == QK_BF16 && d->input != QK_INPUT_PLAIN)
        return qk::fail(QK_ERR_VALUE, "qk_dense: bfloat16 input rows must be plain");
    if (d->x_dtype != QK_BF16 && d->x_dtype != QK_F32)
        return qk::fail(QK_ERR_VALUE, "qk_dense: input dtype must be float32 or bfloat16, got tag %d", d->x_dtype);
    if (d->input == QK_INPUT_CONCAT && (!d->second || d->k % 2 || d->width > d->k / 2))
        return qk::fail(QK_ERR_VALUE, "qk_dense: a concatenated input needs a second vector and two equal halves");
    if (d->input == QK_INPUT_GATED &&
        (!d->gate || !d->norm_weight || d->group == 0 || d->width % d->group))
        return qk::fail(QK_ERR_VALUE, "qk_dense: a gated input needs a gate and whole groups");
    if (d->norm != QK_NORM_NONE && !d->norm_weight && d->input != QK_INPUT_PLAIN)
        return qk::fail(QK_ERR_VALUE, "qk_dense: a norm needs its weight");
    if (d->x_out && d->x_out == d->x) return qk::fail(QK_ERR_VALUE, "qk_dense: x_out must be another buffer than x");
    if (d->pending && !d->pending_weight) return qk::fail(QK_ERR_VALUE, "qk_dense: a pending residual needs its weight");
    if (d->append.src && (!d->append.cache || !d->positions || !d->slots || d->append.ring == 0 ||
                          d->append.width > d->append.stride))
        return qk::fail(QK_ERR_VALUE, "qk_dense: an append needs a cache, positions and slots");
    if (d->input != QK_INPUT_PLAIN && d->k * 4 > kVecSmemMax)
        return qk::fail(QK_ERR_VALUE, "qk_dense: an input vector of %zu entries does not fit shared memory", d->k);
    if (!with_weights) return QK_OK;
    if (!d->w || d->rows == 0 || d->w_stride < d->k || d->w_stride % 8)
        return qk::fail(QK_ERR_VALUE, "qk_dense: %zu weight rows of stride %zu for %zu columns", d->rows, d->w_stride,
                        d->k);
    if (d->w_dtype != QK_F32 && d->w_dtype != QK_BF16)
        return qk::fail(QK_ERR_VALUE, "qk_dense: weight dtype must be float32 or bfloat16, got tag %d", d->w_dtype);
    if (d->output < QK_OUTPUT_STORE || d->output > QK_OUTPUT_SIDE)
        return qk::fail(QK_ERR_VALUE, "qk_dense: unknown output kind %d", d->output);
    if (d->output == QK_OUTPUT_RESIDUAL ? !d->residual : !d->out)
        return qk::fail(QK_ERR_VALUE, "qk_dense: no output buffer");
    if (d->output == QK_OUTPUT_GLU && d->rows % 64)
        return qk::fail(QK_ERR_VALUE, "qk_dense: gated pairs come in blocks of 64 rows, got %zu", d->rows);
    if (d->experts) {
        if (!d->ids || !d->table || d->vocab == 0 || d->top == 0 || d->top > d->experts)
            return qk::fail(QK_ERR_VALUE, "qk_dense: %zu of %zu experts need token ids and a table", d->top, d->experts);
        if (d->output != QK_OUTPUT_STORE && d->output != QK_OUTPUT_GLU)
            return qk::fail(QK_ERR_VALUE, "qk_dense: the rows of experts are stored, not added to a stream");
        if (d->by_choice && d->input != QK_INPUT_PLAIN)
            return qk::fail(QK_ERR_VALUE, "qk_dense: input rows by choice must be plain");
        if (d->append.src) return qk::fail(QK_ERR_VALUE, "qk_dense: no append beside experts");
    }
    if (d->output == QK_OUTPUT_SIDE && (!d->side || !d->ids || d->vocab == 0))
        return qk::fail(QK_ERR_VALUE, "qk_dense: a side product needs its table and token ids");
    return QK_OK;
}

// ------------------------------------------------------------------ choices sorted by expert
constexpr int kRouteThreads = 1024;
__global__ void __launch_bounds__(kRouteThreads)
route_kernel(const qk_route_job *__restrict__ jobs, const int32_t *__restrict__ ids, uint32_t tokens, uint32_t vocab,
             uint32_t tile_rows) {
    qk::pdl_wait();
    const qk_route_job j = jobs[blockIdx.x];
    const uint32_t top = (uint32_t)j.top, experts = (uint32_t)j.experts, n = tokens * top;
    extern __shared__ uint32_t route_smem[];  // [experts]: counts, then each expert's next place
    uint32_t *next = route_smem;
    for (uint32_t e = threadIdx.x; e < experts; e += kRouteThreads) next[e] = 0;
    __syncthreads();
    auto expert = [&](uint32_t i) {
        const uint32_t id = (uint32_t)min(max(ids[i / top], 0), (int)vocab - 1);
        return (uint32_t)j.table[(size_t)id * top + i % top];
    };
    for (uint32_t i = threadIdx.x; i < n; i += kRouteThreads) atomicAdd(&next[expert(i)], 1u);
    __syncthreads();
    if (threadIdx.x < 32) {  // running sums of the counts and of the tiles, 32 experts at a time
        uint32_t places = 0, tiles = 0;
        for (uint32_t e0 = 0; e0 < experts; e0 += 32) {
            const uint32_t e = e0 + threadIdx.x, count = e < experts ? next[e] : 0;
            const uint32_t own = (count + tile_rows - 1) / tile_rows;
            uint32_t p = count, q = own;
            for (int off = 1; off < 32; off *= 2) {
                const uint32_t a = __shfl_up_sync(0xffffffffu, p, off), b = __shfl_up_sync(0xffffffffu, q, off);
                if (threadIdx.x >= (uint32_t)off) p += a, q += b;
            }
            const uint32_t first = places + p - count, tile0 = tiles + q - own;
            if (e < experts) {
                next[e] = first;
                j.offsets[e] = (int32_t)first;
                for (uint32_t k = 0; k < own; ++k) {
                    int32_t *t = j.tiles + 1 + kRouteTile * (tile0 + k);
                    t[0] = (int32_t)e;
                    t[1] = (int32_t)(first + k * tile_rows);
                    t[2] = (int32_t)min(first + (k + 1) * tile_rows, first + count);
                    t[3] = (int32_t)tile0;
                    t[4] = (int32_t)own;
                }
            }
            places += __shfl_sync(0xffffffffu, p, 31);
            tiles += __shfl_sync(0xffffffffu, q, 31);
        }
        if (threadIdx.x == 0) {
            j.offsets[experts] = (int32_t)places;
            j.tiles[0] = (int32_t)tiles;
        }
    }
    __syncthreads();
    // (the order of an expert's places is free: no row's result depends on its place)
    for (uint32_t i = threadIdx.x; i < n; i += kRouteThreads) j.places[i] = (int32_t)atomicAdd(&next[expert(i)], 1u);
}

template <typename A>
qk_status launch_input(qk_ctx *c, const InputArgs &in, size_t tokens, A *dst) {
    auto aligned = [](const void *p) { return ((uintptr_t)p & 15) == 0; };
    const size_t half = in.kind == QK_INPUT_CONCAT ? in.k / 2 : in.k;
    if (sizeof(A) == 2 && dst && (in.kind == QK_INPUT_NORM || in.kind == QK_INPUT_CONCAT) && in.width % 4 == 0 &&
        half % 4 == 0 && half <= 8192 && in.x_stride % 4 == 0 && aligned(in.x) && aligned(in.x_out) && aligned(dst) &&
        (!in.pending || (in.pending_stride % 4 == 0 && aligned(in.pending) && aligned(in.pending_weight))) &&
        aligned(in.second) && aligned(in.norm_weight)) {
        uint16_t *o = reinterpret_cast<uint16_t *>(dst);
        const dim3 grid((unsigned)tokens), block(256);
        if (half <= 1024) (void)qk::launch_pdl(c->pdl, dense_norm_rows_kernel<1>, grid, block, 0, c->stream, in, o);
        else if (half <= 2048) (void)qk::launch_pdl(c->pdl, dense_norm_rows_kernel<2>, grid, block, 0, c->stream, in, o);
        else if (half <= 4096) (void)qk::launch_pdl(c->pdl, dense_norm_rows_kernel<4>, grid, block, 0, c->stream, in, o);
        else (void)qk::launch_pdl(c->pdl, dense_norm_rows_kernel<8>, grid, block, 0, c->stream, in, o);
        QK_CUDA(cudaGetLastError());
        c->launches++;
        return QK_OK;
    }
    const int kind = dst && in.k % 4 == 0 && row_kind_of(in) == kRowNorm ? kRowNorm : kRowAny;
    const size_t smem = dst ? (size_t)in.k * 4 + (kind == kRowNorm ? in.width * 8 : 0) : 0;
    if (smem > kVecSmemMax) return qk::fail(QK_ERR_VALUE, "qk_dense: an input vector of %u entries does not fit shared memory", in.k);
    QK_CUDA(cudaFuncSetAttribute(dense_input_kernel<A>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)std::max(smem, (size_t)48 * 1024)));
    (void)qk::launch_pdl(c->pdl, dense_input_kernel<A>, dim3((unsigned)tokens), dim3(256), smem, c->stream, in, dst, kind);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
}

}  // namespace

extern "C" {

int32_t qk_dense_form(size_t tokens, size_t k, int32_t w_dtype) {
    if (tokens <= (size_t)kVectorTokens && k * 4 <= kVecSmemMax) return QK_FORM_VECTOR;
    if (w_dtype == QK_F32) return QK_FORM_F32;
    return tokens <= (size_t)kNarrowTokens ? QK_FORM_NARROW : QK_FORM_TCGEN05;
}

size_t qk_route_tile_rows(size_t tokens, size_t k, int32_t w_dtype) {
    return qk_dense_form(tokens, k, w_dtype) == QK_FORM_F32 ? kFTile : kTcM;
}

qk_status qk_route(qk_ctx *ctx, const qk_route_job *device_jobs, size_t n_jobs, size_t max_experts, const int32_t *ids,
                   size_t tokens, size_t vocab, size_t tile_rows) {
    qk_ctx *c;
    qk_status st = qk::resolve_ctx(ctx, &c);
    if (st != QK_OK) return st;
    QK_CUDA(cudaSetDevice(c->device));
    if (!device_jobs || !ids || vocab == 0 || tile_rows == 0) return qk::fail(QK_ERR_VALUE, "qk_route: bad arguments");
    if (max_experts * 4 > 48 * 1024) return qk::fail(QK_ERR_VALUE, "qk_route: %zu experts do not fit shared memory", max_experts);
    if (tokens == 0 || n_jobs == 0) return QK_OK;
    (void)qk::launch_pdl(c->pdl, route_kernel, dim3((unsigned)n_jobs), dim3(kRouteThreads), max_experts * 4, c->stream,
                         device_jobs, ids, (uint32_t)tokens, (uint32_t)vocab, (uint32_t)tile_rows);
    QK_CUDA(cudaGetLastError());
    c->launches++;
    return QK_OK;
}

qk_status qk_dense_input(qk_ctx *ctx, const qk_dense_call *d) {
    qk_ctx *c;
    qk_status st = qk::resolve_ctx(ctx, &c);
    if (st != QK_OK) return st;
    QK_CUDA(cudaSetDevice(c->device));
    if ((st = validate(d, false)) != QK_OK) return st;
    if (d->tokens == 0) return QK_OK;
    if (d->x_dtype != QK_F32) return qk::fail(QK_ERR_VALUE, "qk_dense_input: the rows must be float32");
    const InputArgs in = input_args(*d);
    return d->out_dtype == QK_BF16 ? launch_input<uint16_t>(c, in, d->tokens, (uint16_t *)d->out)
                                   : launch_input<float>(c, in, d->tokens, (float *)d->out);
}

qk_status qk_dense(qk_ctx *ctx, const qk_dense_call *d) {
    qk_ctx *c;
    qk_status st = qk::resolve_ctx(ctx, &c);
    if (st != QK_OK) return st;
    QK_CUDA(cudaSetDevice(c->device));
    if ((st = validate(d, true)) != QK_OK) return st;
    if (d->tokens == 0) return QK_OK;
    const bool bf16 = d->w_dtype == QK_BF16;
    const int32_t form = qk_dense_form(d->tokens, d->k, d->w_dtype);
    InputArgs in = input_args(*d);
    OutputArgs out = output_args(*d);
    if (form == QK_FORM_VECTOR && d->x_dtype == QK_F32) {
        if (d->experts) return bf16 ? launch_vector<uint16_t, 1>(c, in, out, *d, 1) : launch_vector<float, 1>(c, in, out, *d, 1);
        // as many rows per launch as fit shared memory
        for (size_t t = 0; t < d->tokens;) {
            const size_t left = d->tokens - t;
            const int nt = left >= 3 && d->k * 16 <= kVecSmemMax ? 4 : left >= 2 && d->k * 8 <= kVecSmemMax ? 2 : 1;
            const size_t n = std::min(left, (size_t)nt);
            if (bf16)
                st = nt == 4 ? launch_vector<uint16_t, 4>(c, in, out, *d, n)
                     : nt == 2 ? launch_vector<uint16_t, 2>(c, in, out, *d, n)
                               : launch_vector<uint16_t, 1>(c, in, out, *d, n);
            else
                st = nt == 4 ? launch_vector<float, 4>(c, in, out, *d, n)
                     : nt == 2 ? launch_vector<float, 2>(c, in, out, *d, n)
                               : launch_vector<float, 1>(c, in, out, *d, n);
            if (st != QK_OK) return st;
            advance(in, out, n);
            t += n;
        }
        return QK_OK;
    }
    // the input rows in the weights' dtype
    const void *rows = d->x;
    size_t stride = d->x_stride;
    const bool direct = d->input == QK_INPUT_PLAIN && (!d->experts || d->by_choice) && d->x_dtype == d->w_dtype && d->x_stride >= d->k &&
                        d->x_stride % 8 == 0 && ((uintptr_t)d->x & 15) == 0;
    if (d->x_dtype == QK_BF16 && !direct)
        return qk::fail(QK_ERR_VALUE, "qk_dense: bfloat16 rows of stride %zu cannot feed %zu columns", d->x_stride, d->k);
    if (d->experts && (!d->offsets || !d->tiles || (!d->places && !d->by_choice)))
        return qk::fail(QK_ERR_VALUE, "qk_dense: the matrix forms need the choices sorted by expert");
    if (!direct) {
        if (d->by_choice) return qk::fail(QK_ERR_VALUE, "qk_dense: rows by choice must be of the weights' dtype");
        if (d->experts) in.places = d->places, in.top = (uint32_t)d->top;
        const size_t need = input_rows(*d) * d->k * (bf16 ? 2 : 4);
        if (!d->scratch || d->scratch_bytes < need)
            return qk::fail(QK_ERR_VALUE, "qk_dense: %zu bytes of scratch are needed, %zu given", need,
                            d->scratch_bytes);
        st = bf16 ? launch_input<uint16_t>(c, in, d->tokens, (uint16_t *)d->scratch)
                  : launch_input<float>(c, in, d->tokens, (float *)d->scratch);
        if (st != QK_OK) return st;
        rows = d->scratch;
        stride = d->k;
    } else if (d->append.src) {
        if ((st = launch_input<float>(c, in, d->tokens, nullptr)) != QK_OK) return st;
    }
    if (!bf16) {
        dim3 grid((unsigned)qk::ceil_div(d->rows, kFTile), (unsigned)row_tiles(*d, kFTile));
        (void)qk::launch_pdl(c->pdl, dense_f32_kernel, grid, dim3(256), 0, c->stream, (const float *)rows,
                             (uint32_t)stride, (uint32_t)d->k, (const float *)d->w, (uint32_t)d->rows,
                             (uint32_t)d->w_stride, (uint32_t)d->tokens, out, d->experts ? d->tiles : nullptr);
        QK_CUDA(cudaGetLastError());
        c->launches++;
        return QK_OK;
    }
    if ((st = qk::error_word(c)) != QK_OK) return st;
    if (d->tokens <= (size_t)kNarrowTokens) {
        if (d->tokens <= 16) return launch_narrow<16>(c, rows, stride, *d, out);
        if (d->tokens <= 32) return launch_narrow<32>(c, rows, stride, *d, out);
        if (d->tokens <= 64) return launch_narrow<64>(c, rows, stride, *d, out);
        return launch_narrow<128>(c, rows, stride, *d, out);
    }
    const int vec = (!d->out || (((uintptr_t)d->out & 15) == 0 && d->out_stride % 4 == 0)) &&
                    (!d->residual || (((uintptr_t)d->residual & 15) == 0 && d->residual_stride % 4 == 0)) &&
                    ((uintptr_t)d->out_scale & 15) == 0;
    switch (pick_tile(row_tiles(*d, kTcM), d->rows, (size_t)c->sm_count)) {
        case 256: return launch_tc<256>(c, rows, stride, *d, out, vec);
        case 128: return launch_tc<128>(c, rows, stride, *d, out, vec);
        default: return launch_tc<64>(c, rows, stride, *d, out, vec);
    }
}

}  // extern "C"
