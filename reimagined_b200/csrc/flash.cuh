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

__device__ __forceinline__ float pow2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }

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
// m the row's maximum (times c), l its sum.  vd: output columns to rescale.
__device__ __forceinline__ void softmax_block(uint32_t s_col, uint32_t o_col, int vd, int last, float c, bool first, float& m, float& l) {
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
        mx[ch] = __uint_as_float(x[ch][0]);
#pragma unroll
        for (int i = 1; i < 32; ++i) mx[ch] = fmaxf(mx[ch], __uint_as_float(x[ch][i]));
    }
    const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * c;
    if (first) {
        m = top;
    } else if (__any_sync(0xffffffffu, top > m + kRescale)) {
        const float mn = fmaxf(m, top), f = pow2(m - mn);
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
    float sum = 0.0f;
#pragma unroll
    for (int ch = 0; ch < 4; ++ch) {
        float a0 = 0.0f, a1 = 0.0f;
        uint32_t y[32];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            const float p0 = pow2(fmaf(__uint_as_float(x[ch][2 * i]), c, -m)), p1 = pow2(fmaf(__uint_as_float(x[ch][2 * i + 1]), c, -m));
            a0 += p0;
            a1 += p1;
            const uint32_t hi = pack_bf16(p0, p1);
            y[i] = hi;
            y[16 + i] = pack_bf16(p0 - bf_lo(hi), p1 - bf_hi(hi));
        }
        sum += a0 + a1;
        tmem_st32(s_col + ch * 32, y);
    }
    l += sum;
    tmem_st_wait();
}

}  // namespace flash
}  // namespace stack
}  // namespace tbl
