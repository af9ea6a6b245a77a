// Fragment helpers of the mma.sync attention kernels: ldmatrix, 16-byte asynchronous copies with
// zero fill, bfloat16 packing and splitting.
#pragma once

#include <cstdint>

#include "qk_decoder_dev.cuh"

namespace {

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void mma16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    mma_bf16_full(c, a[0], a[1], a[2], a[3], b0, b1);
}
__device__ __forceinline__ void copy16(void *smem, const void *gmem, uint32_t bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)),
                 "l"(gmem), "r"(bytes)
                 : "memory");
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    return (uint32_t)float_to_bf16_bits(lo) | ((uint32_t)float_to_bf16_bits(hi) << 16);
}
// x as two bfloat16 terms, packed for two neighbouring values
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t &hi, uint32_t &lo) {
    const uint16_t ah = float_to_bf16_bits(a), bh = float_to_bf16_bits(b);
    hi = (uint32_t)ah | ((uint32_t)bh << 16);
    lo = pack_bf16(a - bf16_bits_to_float(ah), b - bf16_bits_to_float(bh));
}

}  // namespace
