// y[M,N] = x[M,K] (bf16) x w[N,K]^T (bf16) on the 5th-generation tensor cores: the dense counterpart of
// gemm_tcgen05.cu, with the same roles and the same operand geometry (a stage is 128 bytes of K per row, i.e. 64
// bf16, in the 128-byte-swizzled K-major layout TMA writes; an MMA takes 32 bytes of K).
//
// One persistent CTA per SM, ten warps: TMA producer, MMA issuer (tcgen05.mma kind::f16, fp32 accumulators in TMEM,
// two buffers of BN columns), eight epilogue warps.  128 x BN tiles; the two accumulators double-buffer tiles.  (256 x
// 256 tiles, which the int8 kernel uses for large problems, gain nothing here: these epilogues -- residual, gated pair --
// are longer, and a tall tile cannot hide them.)
// The epilogue adds the bias and either adds the fp32 residual and stores fp32, stores bf16, or -- for a gated
// feed-forward, whose weight rows alternate in blocks of 32 gate and 32 up rows -- combines two neighbouring
// 32-column blocks into act(gate) * up and stores that.
// Every wait is bounded: on a timeout the role records the status word and falls through to the common exit, where
// TMEM is released.
#include <cuda.h>

#include "stack.cuh"
#include "tc05.cuh"

namespace tbl {
namespace stack {
namespace {

using namespace tc05;

constexpr int BM = 128;             // activation rows per MMA
constexpr int BKB = 128;            // bytes of K per stage
constexpr int BKE = BKB / 2;        // the same in elements
constexpr int kGroupM = 16;         // row tiles per group of the tile walk
constexpr int kMaxStages = 8;
constexpr int kEpiWarps = 8;
constexpr int kThreads = 32 * (2 + kEpiWarps);

__host__ __device__ constexpr int stages_for(int bn) { return bn >= 256 ? 4 : (bn >= 128 ? 6 : 8); }
constexpr size_t smem_for(int bn) {
    return 1024 + static_cast<size_t>(stages_for(bn)) * (BM * BKB + bn * BKB) + kEpiWarps * 4096 + 256;
}

struct Params {
    DenseCall c;
    int tiles_m, tiles_n;
    int vec;                // outputs (and residual) take 4-column vector accesses
    int* status;
};

__device__ __forceinline__ bool decode_tile(const Params& p, int t, int& row0, int& tn) {
    if (t >= p.tiles_m * p.tiles_n) return false;
    const int per_group = kGroupM * p.tiles_n;
    const int grp = t / per_group, in_grp = t - grp * per_group;
    const int gm = min(kGroupM, p.tiles_m - grp * kGroupM);
    tn = in_grp / gm;
    row0 = (grp * kGroupM + in_grp % gm) * BM;
    return true;
}

// Stores one 32 x 32 block staged in shared memory (row = lane order, 16-byte chunk j of row r at j ^ (r & 7)).
template <bool RES>
__device__ __forceinline__ void store_block(const Params& p, const uint8_t* stage, int lane, int row0, int valid, int col0,
                                            int ncols) {
    const DenseCall& c = p.c;
    const int chunk = lane & 7, rsub = lane >> 3, col = col0 + 4 * chunk;
    if (col >= ncols) return;
    if (RES && p.vec) {
        // residual rows are requested together: one memory round trip per block, not one per row
        float4 res[8];
        {
#pragma unroll
            for (int i8 = 0; i8 < 8; ++i8) {
                const int rr = 4 * i8 + rsub;
                res[i8] = rr < valid ? *reinterpret_cast<const float4*>(c.residual + static_cast<size_t>(row0 + rr) * c.ldo + col)
                                     : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        }
#pragma unroll
        for (int i8 = 0; i8 < 8; ++i8) {
            const int rr = 4 * i8 + rsub;
            if (rr >= valid) continue;
            float4 f = *reinterpret_cast<const float4*>(stage + rr * 128 + ((chunk ^ (rr & 7)) << 4));
            f.x += res[i8].x; f.y += res[i8].y; f.z += res[i8].z; f.w += res[i8].w;
            *reinterpret_cast<float4*>(c.out_f32 + static_cast<size_t>(row0 + rr) * c.ldo + col) = f;
        }
        return;
    }
#pragma unroll
    for (int i8 = 0; i8 < 8; ++i8) {
        const int rr = 4 * i8 + rsub;
        if (rr >= valid) continue;
        const float4 f = *reinterpret_cast<const float4*>(stage + rr * 128 + ((chunk ^ (rr & 7)) << 4));
        const size_t o = static_cast<size_t>(row0 + rr) * c.ldo + col;
        if (p.vec && c.out_f32) {
            *reinterpret_cast<float4*>(c.out_f32 + o) = f;
        } else if (p.vec) {
            *reinterpret_cast<uint2*>(c.out_b16 + o) = make_uint2(pack_bf16(f.x, f.y), pack_bf16(f.z, f.w));
        } else {
            const float v[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (col + e >= ncols) break;
                if (c.out_f32) c.out_f32[o + e] = RES ? c.residual[o + e] + v[e] : v[e];
                else c.out_b16[o + e] = __float2bfloat16_rn(v[e]);
            }
        }
    }
}

template <int BN, bool RES>
__global__ void __launch_bounds__(kThreads, 1)
dense_tcgen05_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, const Params p) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    constexpr int kStages = stages_for(BN);
    constexpr int kABytes = BM * BKB;
    constexpr int kBBytes = BN * BKB;
    constexpr int kStageBytes = kABytes + kBBytes;
    constexpr uint32_t kTmemCols = 2 * BN;
    uint8_t* epi_stage = smem + kStages * kStageBytes;                 // 8 warps x 4 KB
    uint64_t* full = reinterpret_cast<uint64_t*>(epi_stage + kEpiWarps * 4096);
    uint64_t* empty = full + kMaxStages;
    uint64_t* tmem_full = empty + kMaxStages;
    uint64_t* tmem_empty = tmem_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tmem_empty + 2);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kblocks = (p.c.K + BKE - 1) / BKE;

    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&tmem_full[b], 1); mbar_init(&tmem_empty[b], kEpiWarps); }
        fence_mbar_init();
        fence_proxy_async();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(kTmemCols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_launch_dependents();
    pdl_wait();

    if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            int it = 0, row0, tn;
            bool alive = true;
            for (int tile = blockIdx.x; alive && decode_tile(p, tile, row0, tn); tile += gridDim.x) {
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % kStages;
                    if (it >= kStages) {
                        alive = mbar_wait_bounded(&empty[s], ((it / kStages) - 1) & 1, p.status);
                        if (!alive) break;
                    }
                    uint8_t* a_dst = smem + s * kStageBytes;
                    mbar_arrive_expect_tx(&full[s], kStageBytes);
                    tma_load_2d(a_dst, &map_a, kb * BKE, row0, &full[s]);
                    tma_load_2d(a_dst + kABytes, &map_b, kb * BKE, tn * BN, &full[s]);
                }
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        if (lane == 0) {
            const uint32_t idesc = idesc_bf16(BN);
            int it = 0, local = 0, row0, tn;
            bool alive = true;
            for (int tile = blockIdx.x; alive && decode_tile(p, tile, row0, tn); tile += gridDim.x, ++local) {
                const int buf = local & 1;
                if (local >= 2) {
                    alive = mbar_wait_bounded(&tmem_empty[buf], ((local >> 1) - 1) & 1, p.status);
                    if (!alive) break;
                }
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + buf * BN;
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % kStages;
                    alive = mbar_wait_bounded(&full[s], (it / kStages) & 1, p.status);
                    if (!alive) break;
                    tc_fence_after();
                    const uint32_t a_addr = smem_u32(smem + s * kStageBytes);
                    const uint32_t b_addr = a_addr + kABytes;
#pragma unroll
                    for (int kk = 0; kk < BKB / 32; ++kk)
                        umma_f16(d_tmem, smem_desc_sw128(a_addr + kk * 32), smem_desc_sw128(b_addr + kk * 32), idesc, (kb | kk) != 0 ? 1u : 0u);
                    umma_commit(&empty[s]);
                }
                if (alive) umma_commit(&tmem_full[buf]);
            }
        }
    } else {
        // ---------------- epilogue warps ----------------
        const int quarter = warp & 3;          // TMEM lanes 32*quarter .. +31 are this warp's
        const int half = (warp - 2) >> 2;      // which of the two warps of the quarter
        uint8_t* stage = epi_stage + (warp - 2) * 4096;
        const bool pair = p.c.pair_cols > 0;
        const Activation act = activation_of(p.c.act);
        int local = 0, tile_row0, tn;
        bool alive = true;
        for (int tile = blockIdx.x; alive && decode_tile(p, tile, tile_row0, tn); tile += gridDim.x, ++local) {
            const int buf = local & 1;
            alive = mbar_wait_bounded(&tmem_full[buf], (local >> 1) & 1, p.status);
            alive = __all_sync(0xffffffffu, alive);
            if (!alive) break;
            tc_fence_after();
            const int row0 = tile_row0 + quarter * 32;
            const int valid = min(32, p.c.M - row0);
            const uint32_t t_row = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16) + buf * BN;
            const int nblocks = min(BN / 32, (p.c.N - tn * BN + 31) / 32);
            // blocks of 32 columns: every other one is this warp's -- of a gated layer every other pair
            const int step = pair ? 2 : 1;
            uint32_t r[32], rn[32];
            if (half * step < nblocks) tmem_ld32(t_row + half * step * 32, r);
#pragma unroll 1
            for (int b = half * step; b < nblocks; b += 2 * step) {
                const int n0 = tn * BN + b * 32;
                const float bias_l = p.c.bias && n0 + lane < p.c.N ? __ldg(p.c.bias + n0 + lane) : 0.0f;
                int col0 = n0, ncols = p.c.N;
                float v[32];
                tmem_ld_wait();
                if (pair) {
                    tmem_ld32(t_row + (b + 1) * 32, rn);      // N is a multiple of 64
                    const float bias_u = p.c.bias ? __ldg(p.c.bias + n0 + 32 + lane) : 0.0f;
                    tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        const float g = __uint_as_float(r[i]) + __shfl_sync(0xffffffffu, bias_l, i);
                        const float u = __uint_as_float(rn[i]) + __shfl_sync(0xffffffffu, bias_u, i);
                        v[i] = activate(act, g) * u;
                    }
                    if (b + 4 < nblocks) tmem_ld32(t_row + (b + 4) * 32, r);
                    col0 = n0 >> 1;
                    ncols = p.c.pair_cols;
                } else {
                    if (b + 2 < nblocks) tmem_ld32(t_row + (b + 2) * 32, rn);   // in flight while this block is stored
                    if (p.c.bias) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]) + __shfl_sync(0xffffffffu, bias_l, i);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
                    }
                }
                __syncwarp();
#pragma unroll
                for (int j = 0; j < 8; ++j)
                    *reinterpret_cast<float4*>(stage + lane * 128 + ((j ^ (lane & 7)) << 4)) =
                        make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]);
                __syncwarp();
                if (valid > 0) store_block<RES>(p, stage, lane, row0, valid, col0, ncols);
                if (!pair) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) r[i] = rn[i];
                }
            }
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&tmem_empty[buf]);
        }
    }

    // common exit: all roles meet, then the allocating warp releases TMEM
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(kTmemCols) : "memory");
    }
}

template <int BN, bool RES>
cudaError_t launch_kernel(const CUtensorMap& ma, const CUtensorMap& mb, const Params& p, cudaStream_t st) {
    static bool done[64] = {};
    constexpr size_t smem = smem_for(BN);
    static_assert(smem <= 227 * 1024, "shared memory of a CTA");
    const cudaError_t e = allow_smem(dense_tcgen05_kernel<BN, RES>, smem, done);
    if (e != cudaSuccess) return e;
    const int tiles = p.tiles_m * p.tiles_n;
    return launch_dependent(dense_tcgen05_kernel<BN, RES>, dim3(tiles < kNumSm ? tiles : kNumSm), dim3(kThreads), smem, st, ma, mb, p);
}
template <int BN>
cudaError_t launch_bn(const CUtensorMap& ma, const CUtensorMap& mb, const Params& p, cudaStream_t st) {
    return p.c.residual ? launch_kernel<BN, true>(ma, mb, p, st) : launch_kernel<BN, false>(ma, mb, p, st);
}

}  // namespace

bool dense_tensor_supported(const DenseCall& c) {
    return c.K % 8 == 0 && c.ldx % 8 == 0 && c.ldw % 8 == 0 && (reinterpret_cast<uintptr_t>(c.x) & 15) == 0 &&
           (reinterpret_cast<uintptr_t>(c.w) & 15) == 0 && (!c.pair_cols || c.N % 64 == 0);
}

cudaError_t launch_dense_tensor(const DenseCall& c, cudaStream_t st) {
    Params p{};
    p.c = c;
    p.status = device_status_ptr();
    if (!p.status) return cudaErrorUnknown;
    const int cols = c.pair_cols ? c.pair_cols : c.N;
    p.vec = (cols % 4 == 0) && (c.ldo % 4 == 0) && (reinterpret_cast<uintptr_t>(c.out_f32) & 15) == 0 &&
            (reinterpret_cast<uintptr_t>(c.out_b16) & 7) == 0 && (reinterpret_cast<uintptr_t>(c.residual) & 15) == 0;
    // the widest tile that fills the SMs
    int bn = c.N > 128 ? 256 : (c.N > 64 ? 128 : 64);
    const long long tm = (c.M + BM - 1) / BM;
    auto tiles = [&](int b) { return tm * ((c.N + b - 1) / b); };
    auto fill = [&](int b) {
        const long long t = tiles(b);
        return static_cast<double>(t) / (static_cast<double>((t + kNumSm - 1) / kNumSm) * kNumSm);
    };
    if (bn == 256 && fill(128) > 1.15 * fill(256)) bn = 128;
    if (bn == 128 && tiles(128) < 100 && c.N > 64) bn = 64;
    p.tiles_m = static_cast<int>(tm);
    p.tiles_n = (c.N + bn - 1) / bn;
    CUtensorMap ma, mb;
    if (!make_map(&ma, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, c.x, c.M, c.K, BKE, BM, CU_TENSOR_MAP_SWIZZLE_128B, c.ldx))
        return cudaErrorUnknown;
    if (!make_map(&mb, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, c.w, c.N, c.K, BKE, bn, CU_TENSOR_MAP_SWIZZLE_128B, c.ldw)) return cudaErrorUnknown;
    return bn == 256 ? launch_bn<256>(ma, mb, p, st) : (bn == 128 ? launch_bn<128>(ma, mb, p, st) : launch_bn<64>(ma, mb, p, st));
}

}  // namespace stack
}  // namespace tbl
