// What the flash-attention kernels on tcgen05 share: geometry of the tiles in tensor memory, and the softmax of one block.
//
// A CTA works on two tiles of 128 query rows that take turns on the tensor cores.  S = Q K^T of tile w accumulates in the
// 128 columns at 128 w; the weights go back into the columns S came from as two bf16 terms (p = hi + lo, both multiplied:
// 16 bits of mantissa), as the A operand of O += P V; O of tile w is at 256 + 128 w.  Row maxima are only moved when they
// grow by 2^8 (then O and the sum are rescaled).
#pragma once

#include "stack.cuh"
#include "tc05.cuh"

namespace tbl {
namespace stack {
namespace flash {

using namespace tc05;

constexpr int kBlock = 128;                  // context tokens per block (and queries per tile)
constexpr int kSubBytes = 128 * 128;         // a sub-tile: 128 rows x 64 bf16
constexpr int kSoftWarps = 8;                // warps 0-3 and 4-7: softmax of tile 0 and 1, a thread per query row
constexpr int kTmaWarp = kSoftWarps, kMmaWarp = kSoftWarps + 1;
constexpr int kThreads = 32 * (kSoftWarps + 2);
constexpr int kOCol = 256;
constexpr float kRescale = 8.0f;

// two fp32 numbers per instruction
__device__ __forceinline__ uint64_t pair_of(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void unpair(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
    float r;
    asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
    return r;
}

// d += a b^T over n steps of 16; a and b walk 64-element sub-tiles (a descriptor counts 16-byte units)
__device__ __forceinline__ void products(uint32_t d_tmem, uint64_t a, uint64_t b, int n, uint32_t idesc, uint32_t acc) {
    for (; n >= 4; n -= 4, a += kSubBytes / 16, b += kSubBytes / 16, acc = 1) {
        umma_f16(d_tmem, a, b, idesc, acc);
        umma_f16(d_tmem, a + 2, b + 2, idesc, 1);
        umma_f16(d_tmem, a + 4, b + 4, idesc, 1);
        umma_f16(d_tmem, a + 6, b + 6, idesc, 1);
    }
    for (; n > 0; --n, a += 2, b += 2, acc = 1) umma_f16(d_tmem, a, b, idesc, acc);
}

// One block of 128 scores of this thread's row -> weights in place; columns past `last` are not visible.  c = scale log2 e,
// m the row's maximum (times c), l its sum.  vd: output columns to rescale.  p_full: two barriers, one for each half of the
// weights, so that the second product starts under the second half's exponentials.
__device__ __forceinline__ void softmax_block(uint32_t s_col, uint32_t o_col, int vd, int last, float c, bool first, float& m, float& l,
                                              uint64_t* p_full, int lane) {
    const bool edge = __any_sync(0xffffffffu, last < kBlock - 1);
    // the whole row at once: 128 scores in registers
    uint32_t x[4][32];
#pragma unroll
    for (int ch = 0; ch < 4; ++ch) tmem_ld32(s_col + ch * 32, x[ch]);
    tmem_ld_wait();
    if (edge) {
#pragma unroll
        for (int ch = 0; ch < 4; ++ch)
#pragma unroll
            for (int i = 0; i < 32; ++i)
                if (ch * 32 + i > last) x[ch][i] = 0xff800000u;         // -inf
    }
    float mx[4];
#pragma unroll
    for (int ch = 0; ch < 4; ++ch) {
        mx[ch] = fmaxf(__uint_as_float(x[ch][0]), __uint_as_float(x[ch][1]));
#pragma unroll
        for (int i = 2; i < 32; i += 2) mx[ch] = max3(mx[ch], __uint_as_float(x[ch][i]), __uint_as_float(x[ch][i + 1]));
    }
    const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * c;
    if (first) {
        m = top;
    } else if (__any_sync(0xffffffffu, top > m + kRescale)) {
        const float mn = fmaxf(m, top), f = ex2(m - mn);
        m = mn;
        l *= f;
#pragma unroll 1
        for (int ch = 0; ch * 32 < vd; ++ch) {             // columns past vd are unused tensor memory
            uint32_t y[32];
            tmem_ld32(o_col + ch * 32, y);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) y[i] = __float_as_uint(__uint_as_float(y[i]) * f);
            tmem_st32(o_col + ch * 32, y);
        }
    }
    const uint64_t cc = pair_of(c, c), mm = pair_of(-m, -m);
    uint64_t sums[2] = {0, 0};
#pragma unroll
    for (int ch = 0; ch < 4; ++ch) {
        uint32_t y[32];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float p0, p1;
            unpair(fma2(pair_of(__uint_as_float(x[ch][2 * i]), __uint_as_float(x[ch][2 * i + 1])), cc, mm), p0, p1);
            p0 = ex2(p0);
            p1 = ex2(p1);
            const uint64_t p = pair_of(p0, p1);
            sums[i & 1] = add2(sums[i & 1], p);
            // the high term cut off, the low term the (exact) rest rounded
            const uint32_t b0 = __float_as_uint(p0), b1 = __float_as_uint(p1);
            y[i] = __byte_perm(b0, b1, 0x7632);
            float r0, r1;
            unpair(add2(p, pair_of(-__uint_as_float(b0 & 0xffff0000u), -__uint_as_float(b1 & 0xffff0000u))), r0, r1);
            y[16 + i] = pack_bf16(r0, r1);
        }
        tmem_st32(s_col + ch * 32, y);
        if (ch & 1) {
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + (ch >> 1));
        }
    }
    float a0, a1;
    unpair(add2(sums[0], sums[1]), a0, a1);
    l += a0 + a1;
}

}  // namespace flash
}  // namespace stack
}  // namespace tbl
