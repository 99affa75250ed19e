// Linear layers over a few bf16 rows (decode): the weights stream from memory once, straight into the A fragments of
// warp-level MMAs (16 weight rows x 16 of K), the activation rows are the B operand (8 rows per MMA).
//
// The order of K inside an MMA is free as long as both operands agree, so a lane's fragments are plain 16-byte loads:
// of weight rows g and g + 8 and of activation row g (g = lane / 4) it takes elements 8t .. 8t + 7 of every 32 (t =
// lane % 4) and feeds two MMAs with them.  No shared-memory staging; the activations stay in L1.
// A CTA's eight warps share WK-way the K range of 8 / WK row units (so that short matrices still fill the GPU); the
// partial sums meet in shared memory, where the epilogue adds bias and residual, gates, or pairs.  The first weight
// loads are issued before the wait on the preceding kernel of the step.
#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

constexpr int kWarps = 8;

__device__ __forceinline__ uint4 ld_stream(const bf16* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// TA: 16-row weight tiles per warp (a gated layer: the gate tile and its up tile).  NB: blocks of 8 activation rows.
template <int TA, int NB>
__global__ void __launch_bounds__(32 * kWarps) dense_rows_kernel(const DenseCall c, const int wk) {
    constexpr int U = TA == 1 ? 4 : 2;                     // steps of 32 in flight per batch of loads
    constexpr int LDP = NB * 8 + 1;
    extern __shared__ float part[];                        // [warps][TA * 16][LDP]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int units = kWarps / wk, ks = warp % wk;
    const int unit = blockIdx.x * units + warp / wk;
    const int m0 = blockIdx.z * NB * 8, M = min(c.M - m0, NB * 8);
    const bool pair = c.pair_cols > 0;
    const bf16* w = c.w + blockIdx.y * c.batch_w;
    const bf16* wp[TA][2];
#pragma unroll
    for (int i = 0; i < TA; ++i) {
        const int n0 = pair ? unit * 16 / TBL_PAIR_BLOCK * 2 * TBL_PAIR_BLOCK + unit * 16 % TBL_PAIR_BLOCK + i * TBL_PAIR_BLOCK
                            : (unit * TA + i) * 16;
        wp[i][0] = w + static_cast<size_t>(min(n0 + g, c.N - 1)) * c.ldw + t * 8;
        wp[i][1] = w + static_cast<size_t>(min(n0 + g + 8, c.N - 1)) * c.ldw + t * 8;
    }
    const int steps = (c.K + 31) / 32, per = (steps + wk - 1) / wk;
    const int s0 = ks * per, s1 = min(steps, s0 + per);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    uint4 a[U][TA][2], an[U][TA][2];
    auto load_w = [&](uint4 (&d)[U][TA][2], int s) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const bool ok = s + u < s1 && (s + u) * 32 + t * 8 < c.K;
#pragma unroll
            for (int i = 0; i < TA; ++i)
#pragma unroll
                for (int h = 0; h < 2; ++h) d[u][i][h] = ok ? ld_stream(wp[i][h] + (s + u) * 32) : zero;
        }
    };
    load_w(a, s0);
    pdl_launch_dependents();
    pdl_wait();
    const bf16* x = static_cast<const bf16*>(c.x) + blockIdx.y * c.batch_x + static_cast<size_t>(m0) * c.ldx + t * 8;
    float acc[TA][NB][4] = {};
    for (int s = s0; s < s1; s += U) {
        uint4 b[U][NB];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const bool ok = s + u < s1 && (s + u) * 32 + t * 8 < c.K;
#pragma unroll
            for (int n = 0; n < NB; ++n)
                b[u][n] = ok && n * 8 + g < M ? *reinterpret_cast<const uint4*>(x + static_cast<size_t>(n * 8 + g) * c.ldx + (s + u) * 32) : zero;
        }
        load_w(an, s + U);
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int i = 0; i < TA; ++i)
#pragma unroll
                for (int n = 0; n < NB; ++n) {
                    mma16816(acc[i][n], a[u][i][0].x, a[u][i][1].x, a[u][i][0].y, a[u][i][1].y, b[u][n].x, b[u][n].y);
                    mma16816(acc[i][n], a[u][i][0].z, a[u][i][1].z, a[u][i][0].w, a[u][i][1].w, b[u][n].z, b[u][n].w);
                }
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int i = 0; i < TA; ++i) { a[u][i][0] = an[u][i][0]; a[u][i][1] = an[u][i][1]; }
    }
    float* mine = part + warp * TA * 16 * LDP;
#pragma unroll
    for (int i = 0; i < TA; ++i)
#pragma unroll
        for (int n = 0; n < NB; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) mine[(i * 16 + g + (e >> 1) * 8) * LDP + n * 8 + 2 * t + (e & 1)] = acc[i][n][e];
    __syncthreads();
    const int cols = pair ? 16 : 16 * TA;                  // output columns per unit
    const int ncols = pair ? c.pair_cols : c.N;
    for (int e = threadIdx.x; e < units * cols * M; e += 32 * kWarps) {
        const int m = e / (units * cols), r = e - m * units * cols;
        const int un = r / cols, col = r - un * cols;
        const int n = (blockIdx.x * units + un) * cols + col;
        if (n >= ncols) continue;
        const float* src = part + un * wk * TA * 16 * LDP + col * LDP + m;
        float v = 0.0f, up = 0.0f;
        for (int k = 0; k < wk; ++k) v += src[k * TA * 16 * LDP];
        if (pair) {
            for (int k = 0; k < wk; ++k) up += src[k * TA * 16 * LDP + 16 * LDP];
            const int gr = n / TBL_PAIR_BLOCK * 2 * TBL_PAIR_BLOCK + n % TBL_PAIR_BLOCK;
            if (c.bias) { v += __ldg(c.bias + gr); up += __ldg(c.bias + gr + TBL_PAIR_BLOCK); }
            v = activate(activation_of(c.act), v) * up;
        } else {
            if (c.bias) v += __ldg(c.bias + n);
        }
        if (c.gate) v *= sigmoid_f(c.gate[static_cast<size_t>(m0 + m) * c.ldg + blockIdx.y * c.batch_gate + n]);
        const size_t o = static_cast<size_t>(m0 + m) * c.ldo + blockIdx.y * c.batch_out + n;
        if (c.out_f32) c.out_f32[o] = c.residual ? c.residual[o] + v : v;
        else c.out_b16[o] = __float2bfloat16_rn(v);
    }
}

template <int TA, int NB>
cudaError_t launch(const DenseCall& c, cudaStream_t st) {
    static bool done[64] = {};
    const size_t smem = sizeof(float) * kWarps * TA * 16 * (NB * 8 + 1);
    const cudaError_t e = allow_smem(dense_rows_kernel<TA, NB>, smem, done);
    if (e != cudaSuccess) return e;
    const int batch = c.batch > 0 ? c.batch : 1;
    const int units = c.pair_cols ? ceil_div(c.pair_cols, 16) : ceil_div(c.N, 16 * TA);
    int wk = 1;
    while (wk < kWarps && static_cast<long long>(units) * batch * wk < 148 * 14 && c.K >= 256 * wk) wk *= 2;
    return launch_dependent(dense_rows_kernel<TA, NB>, dim3(ceil_div(units, kWarps / wk), batch, ceil_div(c.M, NB * 8)), dim3(32 * kWarps), smem, st,
                            c, wk);
}

template <int TA>
cudaError_t launch_ta(const DenseCall& c, cudaStream_t st) {
    if (c.M <= 8) return launch<TA, 1>(c, st);
    if (c.M <= 16) return launch<TA, 2>(c, st);
    if (c.M <= 32) return launch<TA, 4>(c, st);
    return launch<TA, 8>(c, st);
}

}  // namespace

bool dense_rows_supported(const DenseCall& c) {
    return c.K % 8 == 0 && c.ldx % 8 == 0 && c.ldw % 8 == 0 && c.batch_w % 8 == 0 && c.batch_x % 8 == 0 && c.batch <= 65535 && c.M <= 65535 * 64 &&
           (reinterpret_cast<uintptr_t>(c.x) & 15) == 0 && (reinterpret_cast<uintptr_t>(c.w) & 15) == 0;
}

cudaError_t launch_dense_rows(const DenseCall& c, cudaStream_t st) {
    // two weight tiles per warp where the matrix is tall enough to fill the GPU with them
    const bool two = c.pair_cols || static_cast<long long>(c.N) * (c.batch > 0 ? c.batch : 1) >= 32LL * 148 * 8;
    return two ? launch_ta<2>(c, st) : launch_ta<1>(c, st);
}

}  // namespace stack
}  // namespace tbl
