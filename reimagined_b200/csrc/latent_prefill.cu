// Latent attention of a portion of a prompt: keys and values of the whole context are expanded from the cached latents
// by two tensor-core GEMMs, then a flash-attention kernel on tcgen05 runs over them.
//
//   latent_gather_kernel    the cached rows of every sequence of the step, contiguous and zero-padded to whole blocks
//   (GEMM)                  keys  [sequence x context][heads*dim]        = gathered latents x W_uk^T
//   (GEMM)                  values^T [heads*vdim][sequence x context]     = W_uv x gathered latents^T: already in the
//                           K-major form the second product wants
//   latent_query_kernel     queries in bf16 with their rotated part rotated
//   latent_prefill_kernel   256 queries of one head per CTA, two tiles of 128 that take turns on the tensor cores: while
//                           one tile's four softmax warps work, the other tile's products run (flash.cuh).
// Roles: warps 0-3 and 4-7 softmax of tile 0 and 1 (a thread per query row), warp 8 TMA, warp 9 MMA issue.
// Every wait is bounded; a role that gives up records the status word and falls through to the common exit.
#include <cuda.h>

#include "flash.cuh"
#include "latent.cuh"

namespace tbl {
namespace stack {
namespace {

using namespace flash;

constexpr int kMaxSub = 3;                   // sub-tiles of a query or key tile: unrotated part, then rotated part
constexpr int kMaxRing = 8;

struct PrefillParams {
    const int32_t *slots, *positions;
    const float* gate;         // [rows][ldg]: gate columns of the stacked projections
    bf16* out;                 // [rows][H*vd]
    int* status;
    int ldg, H, d, rd, vd, n_tok, ctx, tiles, k_stages, v_stages;
    float scale_log2;
};

__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* __restrict__ cache, const int32_t* __restrict__ slots,
                                                            const int32_t* __restrict__ positions, int capacity, int cw, int n_tok,
                                                            int ctx, bf16* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.y, slot = slots[seq], n = min(positions[slot] + n_tok, capacity), per = cw / 8;
    const size_t total = static_cast<size_t>(ctx) * per;
    for (size_t i = static_cast<size_t>(blockIdx.x) * 256 + threadIdx.x; i < total; i += static_cast<size_t>(gridDim.x) * 256) {
        const int t = static_cast<int>(i / per), c = static_cast<int>(i - static_cast<size_t>(t) * per);
        uint4 v = make_uint4(0, 0, 0, 0);
        if (t < n) v = *reinterpret_cast<const uint4*>(cache + (static_cast<size_t>(slot) * capacity + t) * cw + c * 8);
        reinterpret_cast<uint4*>(out)[static_cast<size_t>(seq) * total + i] = v;
    }
}

// one warp per (row, head)
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentParams p, int rows, bf16* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t unit = static_cast<size_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
    if (unit >= static_cast<size_t>(rows) * p.H) return;
    const int lane = threadIdx.x & 31, n = p.d + p.rd, half = p.rd / 2;
    const int row = static_cast<int>(unit / p.H);
    const int slot = p.slots[row / p.n_tok];
    const int pos = min(max(p.positions[slot] + row % p.n_tok, 0), p.rope_positions - 1);
    const float* q = p.q + unit * n;
    bf16* o = out + unit * n;
    for (int e = 4 * lane; e < p.d; e += 128) {
        const float4 v = *reinterpret_cast<const float4*>(q + e);
        *reinterpret_cast<uint2*>(o + e) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    }
    const float *cs = p.rope_cos + static_cast<size_t>(pos) * half, *sn = p.rope_sin + static_cast<size_t>(pos) * half;
    for (int i = lane; i < half; i += 32) {
        const float c = __ldg(cs + i), s = __ldg(sn + i), u = q[p.d + i], v = q[p.d + half + i];
        o[p.d + i] = __float2bfloat16_rn(u * c - v * s);
        o[p.d + half + i] = __float2bfloat16_rn(v * c + u * s);
    }
}

__global__ void __launch_bounds__(kThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_v, const PrefillParams p) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int sub_d = (p.d + 63) / 64, sub_r = (p.rd + 63) / 64, nsub = sub_d + sub_r;
    const int q_bytes = nsub * kSubBytes, k_bytes = nsub * kSubBytes, v_bytes = p.vd * 128;      // V: 64 tokens per entry
    uint8_t* q_smem = smem;                                    // two tiles
    uint8_t* k_smem = q_smem + 2 * q_bytes;                    // ring of key blocks
    uint8_t* v_smem = k_smem + p.k_stages * k_bytes;           // ring of half blocks of values (entries 1024-byte aligned: vd % 8 == 0)
    uint64_t* bars = reinterpret_cast<uint64_t*>(v_smem + p.v_stages * v_bytes);
    uint64_t *q_full = bars, *k_full = bars + 1, *k_empty = k_full + kMaxRing, *v_full = k_empty + kMaxRing, *v_empty = v_full + kMaxRing,
             *s_full = v_empty + kMaxRing, *p_full = s_full + 2, *o_full = p_full + 4;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 2);

    const int warp = uniform_warp(), lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < kMaxRing; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
        for (int w = 0; w < 2; ++w) { mbar_init(&s_full[w], 1); mbar_init(&p_full[2 * w], 4); mbar_init(&p_full[2 * w + 1], 4); mbar_init(&o_full[w], 1); }
        fence_mbar_init();
        fence_proxy_async();
    }
    if (warp == kMmaWarp) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(smem_u32(tmem_slot)) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_launch_dependents();
    pdl_wait();

    // long rows first: the last tiles of a prompt see the most context
    const int tile = p.tiles - 1 - blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    const int q0 = tile * 2 * kBlock;                          // first query of the CTA within its sequence's portion
    const int pos0 = p.positions[p.slots[seq]] + q0;           // and its position
    auto blocks_of = [&](int w) {                              // blocks a tile sees
        const int rows = min(kBlock, p.n_tok - q0 - w * kBlock);
        return rows > 0 ? min(pos0 + w * kBlock + rows - 1, p.ctx - 1) / kBlock + 1 : 0;
    };
    const int nblk0 = blocks_of(0), nblk1 = blocks_of(1);
    const int nmax = max(nblk0, nblk1);
    const int row_q = seq * p.n_tok + q0, row_k = seq * p.ctx;

    if (warp == kTmaWarp) {
        // ---------------- TMA ----------------
        if (elect_one()) {
            const int tiles_q = nblk1 > 0 ? 2 : 1, n = p.d + p.rd;
            mbar_arrive_expect_tx(q_full, tiles_q * q_bytes);
            for (int w = 0; w < tiles_q; ++w) {
                for (int s = 0; s < sub_d; ++s)
                    tma_load_2d(q_smem + w * q_bytes + s * kSubBytes, &map_q, head * n + 64 * s, row_q + w * kBlock, q_full);
                for (int s = 0; s < sub_r; ++s)
                    tma_load_2d(q_smem + w * q_bytes + (sub_d + s) * kSubBytes, &map_q, head * n + p.d + 64 * s, row_q + w * kBlock, q_full);
            }
            bool alive = true;
            int vi = 0;
            for (int j = 0; alive && j < nmax; ++j) {
                const int ks = j % p.k_stages;
                if (j >= p.k_stages) alive = mbar_wait_bounded(&k_empty[ks], ((j / p.k_stages) - 1) & 1, p.status);
                if (!alive) break;
                mbar_arrive_expect_tx(&k_full[ks], k_bytes);
                for (int s = 0; s < sub_d; ++s)
                    tma_load_2d(k_smem + ks * k_bytes + s * kSubBytes, &map_k, head * p.d + 64 * s, row_k + j * kBlock, &k_full[ks]);
                for (int s = 0; s < sub_r; ++s)
                    tma_load_2d(k_smem + ks * k_bytes + (sub_d + s) * kSubBytes, &map_r, 64 * s, row_k + j * kBlock, &k_full[ks]);
                for (int h = 0; h < 2; ++h, ++vi) {
                    const int vs = vi % p.v_stages;
                    if (vi >= p.v_stages) alive = mbar_wait_bounded(&v_empty[vs], ((vi / p.v_stages) - 1) & 1, p.status);
                    if (!alive) break;
                    mbar_arrive_expect_tx(&v_full[vs], v_bytes);
                    tma_load_2d(v_smem + vs * v_bytes, &map_v, row_k + j * kBlock + 64 * h, head * p.vd, &v_full[vs]);
                }
            }
        }
    } else if (warp == kMmaWarp) {
        // ---------------- MMA ----------------
        if (elect_one()) {
            const uint32_t is = idesc_bf16(kBlock), iv = idesc_bf16(p.vd);
            bool alive = mbar_wait_bounded(q_full, 0, p.status);
            tc_fence_after();
            // One thread issues everything, so the loop carries ring positions and descriptors along instead of working them
            // out per product (a descriptor counts 16-byte units).
            const uint64_t q_desc = smem_desc_sw128(smem_u32(q_smem)), k_desc = smem_desc_sw128(smem_u32(k_smem)),
                           v_desc = smem_desc_sw128(smem_u32(v_smem));
            const int nd = p.d / 16, nr = p.rd / 16;
            int ks = 0, v0 = 0, v1 = 1;       // ring slots of the next key block and of this block's value halves
            uint32_t kp = 0, vp0 = 0, vp1 = 0;
            // The order S0(0) S1(0) | PV0(j) S0(j+1) PV1(j) S1(j+1) | ...: each softmax runs under the other tile's products.
            for (int j = -1; alive && j < nmax; ++j) {
#pragma unroll
                for (int w = 0; w < 2; ++w) {
                    if (j >= 0 && j < (w ? nblk1 : nblk0)) {
                        const uint32_t o = tmem + kOCol + w * 128;
#pragma unroll
                        for (int h = 0; h < 2; ++h) {
                            const int vs = h ? v1 : v0;
                            alive = mbar_wait_bounded(&p_full[2 * w + h], j & 1, p.status);
                            if (!alive) break;
                            alive = mbar_wait_bounded(&v_full[vs], h ? vp1 : vp0, p.status);
                            if (!alive) break;
                            tc_fence_after();
                            const uint64_t bd = v_desc + static_cast<uint64_t>(vs) * (v_bytes / 16);
                            const uint32_t pc = tmem + w * kBlock + h * 64;
#pragma unroll
                            for (int k = 0; k < 4; ++k) {          // 16 tokens each: columns 32 (k / 2) + 8 (k & 1), + 16 for the low term
                                umma_f16_ta(o, pc + (k >> 1) * 32 + (k & 1) * 8, bd + 2 * k, iv, (h | k) != 0 ? 1u : (j != 0 ? 1u : 0u));
                                umma_f16_ta(o, pc + (k >> 1) * 32 + (k & 1) * 8 + 16, bd + 2 * k, iv, 1);
                            }
                            // the entry is free once the last tile that uses it has read it
                            if (w == 1 || j >= nblk1) umma_commit(&v_empty[vs]);
                        }
                        if (!alive) break;
                        if (j == (w ? nblk1 : nblk0) - 1) umma_commit(&o_full[w]);
                    }
                    const int jn = j + 1;
                    if (jn < (w ? nblk1 : nblk0)) {
                        // first use of a key block waits for it
                        if (w == 0 || jn >= nblk0) {
                            alive = mbar_wait_bounded(&k_full[ks], kp, p.status);
                            if (!alive) break;
                            tc_fence_after();
                        }
                        const uint64_t a = q_desc + static_cast<uint64_t>(w) * (q_bytes / 16), b = k_desc + static_cast<uint64_t>(ks) * (k_bytes / 16);
                        const uint64_t rot = static_cast<uint64_t>(sub_d) * (kSubBytes / 16);
                        products(tmem + w * kBlock, a, b, nd, is, 0);
                        products(tmem + w * kBlock, a + rot, b + rot, nr, is, 1);
                        umma_commit(&s_full[w]);
                        if (w == 1 || jn >= nblk1) umma_commit(&k_empty[ks]);
                    }
                }
                if (++ks == p.k_stages) { ks = 0; kp ^= 1; }
                if (j >= 0) {                                      // two value halves further on
                    v0 += 2;
                    if (v0 >= p.v_stages) { v0 -= p.v_stages; vp0 ^= 1; }
                    v1 += 2;
                    if (v1 >= p.v_stages) { v1 -= p.v_stages; vp1 ^= 1; }
                }
            }
        }
    } else {
        // ---------------- softmax: a thread per query row ----------------
        const int w = warp >> 2, quarter = warp & 3;
        const int r = quarter * 32 + lane;                     // row of the tile
        const int pos = pos0 + w * kBlock + r;                 // sees tokens 0 .. pos
        const uint32_t lanes = static_cast<uint32_t>(quarter * 32) << 16;
        const uint32_t s_col = tmem + lanes + w * kBlock, o_col = tmem + lanes + kOCol + w * 128;
        const float c = p.scale_log2;
        float m = -INFINITY, l = 0.0f;
        bool alive = true;
        const int n = w == 0 ? nblk0 : nblk1;
        for (int j = 0; j < n; ++j) {
            alive = mbar_wait_bounded(&s_full[w], j & 1, p.status);
            alive = __all_sync(0xffffffffu, alive);
            if (!alive) break;
            tc_fence_after();
            softmax_block(s_col, o_col, p.vd, pos - j * kBlock, c, j == 0, m, l, p_full + 2 * w, lane);
        }
        if (alive && n > 0) {
            alive = mbar_wait_bounded(&o_full[w], 0, p.status);
            alive = __all_sync(0xffffffffu, alive);
            if (alive) {
                tc_fence_after();
                const int q = q0 + w * kBlock + r;
                const bool ok = q < p.n_tok;
                const size_t row = static_cast<size_t>(seq) * p.n_tok + (ok ? q : 0);
                const float inv = 1.0f / l;
                const float* g = p.gate + row * p.ldg + head * p.vd;
                bf16* o = p.out + (row * p.H + head) * p.vd;
                for (int ch = 0; ch * 32 < p.vd; ++ch) {
                    uint32_t x[32];
                    tmem_ld32(o_col + ch * 32, x);
                    tmem_ld_wait();
                    if (ok) {
                        const int cols = min(32, p.vd - ch * 32);
#pragma unroll
                        for (int i = 0; i < 32; i += 8) {
                            if (i >= cols) break;
                            uint32_t y[4];
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                const float g0 = __ldg(g + ch * 32 + i + 2 * e), g1 = __ldg(g + ch * 32 + i + 2 * e + 1);
                                y[e] = pack_bf16(__uint_as_float(x[i + 2 * e]) * inv * sigmoid_f(g0),
                                                 __uint_as_float(x[i + 2 * e + 1]) * inv * sigmoid_f(g1));
                            }
                            *reinterpret_cast<uint4*>(o + ch * 32 + i) = make_uint4(y[0], y[1], y[2], y[3]);
                        }
                    }
                }
            }
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == kMmaWarp) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;" ::"r"(tmem) : "memory");
    }
}

constexpr size_t kFixedSmem = 1024 + 8 * (1 + 4 * kMaxRing + 8) + 16;

int sub_tiles(const tbl_latent_mixer& m) { return (m.dim + 63) / 64 + (m.rot_dim + 63) / 64; }

}  // namespace

bool latent_expanded_supported(const tbl_latent_mixer& m) {
    return m.dim % 16 == 0 && m.rot_dim % 16 == 0 && m.vdim % 16 == 0 && m.vdim <= 128 && m.kv_rank % 8 == 0 && m.scale > 0.0f &&
           sub_tiles(m) <= kMaxSub;
}

int latent_expanded_context(int context) { return static_cast<int>(round_up(context, kBlock)); }

int launch_latent_expanded(const tbl_latent_mixer& m, const LatentParams& p, int n_seq, cudaStream_t st) {
    const int ctx = p.context, rows = n_seq * p.n_tok;          // padded to whole blocks by the caller
    bf16* gathered = p.gathered;
    const int grid = ceil_div(static_cast<long long>(ctx) * (p.cw / 8), 256);
    if (n_seq > 65535 || static_cast<long long>(n_seq) * ctx > 2147483647LL) return TBL_ERR_SHAPE;
    if (launch_dependent(latent_gather_kernel, dim3(grid < 4 * kNumSm ? grid : 4 * kNumSm, n_seq), dim3(256), 0, st,
                         static_cast<const bf16*>(p.cache), p.slots, p.positions, p.capacity, p.cw, p.n_tok, ctx, gathered) != cudaSuccess)
        return TBL_ERR_CUDA;
    DenseCall k{};
    k.x = gathered; k.w = p.uk; k.ldx = p.cw; k.M = n_seq * ctx; k.K = p.R; k.N = p.H * p.d; k.out_b16 = p.keys; k.ldo = k.N;
    int rc = launch_dense(TBL_BF16, kDenseTensor, k, st);
    if (rc != TBL_OK) return rc;
    DenseCall v{};
    v.x = p.uv; v.w = gathered; v.ldx = p.R; v.ldw = p.cw; v.M = p.H * p.vd; v.K = p.R; v.N = n_seq * ctx; v.out_b16 = p.values; v.ldo = v.N;
    rc = launch_dense(TBL_BF16, kDenseTensor, v, st);
    if (rc != TBL_OK) return rc;
    bf16* q = static_cast<bf16*>(p.qa);
    if (launch_dependent(latent_query_kernel, dim3(ceil_div(static_cast<long long>(rows) * p.H, 8)), dim3(256), 0, st, p, rows, q) != cudaSuccess)
        return TBL_ERR_CUDA;

    PrefillParams f{};
    f.slots = p.slots; f.positions = p.positions; f.gate = p.proj + p.q_rank + p.R + p.rd; f.out = static_cast<bf16*>(p.out); f.status = p.status;
    f.ldg = p.ld; f.H = p.H; f.d = p.d; f.rd = p.rd; f.vd = p.vd; f.n_tok = p.n_tok; f.ctx = ctx; f.tiles = ceil_div(p.n_tok, 2 * kBlock);
    f.scale_log2 = p.scale * 1.4426950408889634f;
    const int nsub = sub_tiles(m);
    const size_t tile = static_cast<size_t>(nsub) * kSubBytes, half = static_cast<size_t>(p.vd) * 128;
    const size_t room = 227 * 1024 - kFixedSmem - 2 * tile;
    f.k_stages = 2;
    f.v_stages = static_cast<int>((room - 2 * tile) / half);
    f.v_stages = f.v_stages > 4 ? 4 : f.v_stages;          // at least a whole block: two halves
    if (f.v_stages < 2) return TBL_ERR_SHAPE;
    const size_t smem = kFixedSmem + 4 * tile + f.v_stages * half;
    CUtensorMap mq, mk, mr, mv;
    const auto t = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    if (!make_map(&mq, t, 2, q, rows, static_cast<uint64_t>(p.H) * (p.d + p.rd), 64, kBlock) ||
        !make_map(&mk, t, 2, p.keys, static_cast<uint64_t>(n_seq) * ctx, static_cast<uint64_t>(p.H) * p.d, 64, kBlock) ||
        !make_map(&mr, t, 2, gathered + p.R, static_cast<uint64_t>(n_seq) * ctx, p.rd, 64, kBlock, CU_TENSOR_MAP_SWIZZLE_128B, p.cw) ||
        !make_map(&mv, t, 2, p.values, static_cast<uint64_t>(p.H) * p.vd, static_cast<uint64_t>(n_seq) * ctx, 64, p.vd))
        return TBL_ERR_CUDA;
    static bool done[64] = {};
    if (allow_smem(latent_prefill_kernel, smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    return launch_dependent(latent_prefill_kernel, dim3(f.tiles, p.H, n_seq), dim3(kThreads), smem, st, mq, mk, mr, mv, f) == cudaSuccess
               ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace stack
}  // namespace tbl
