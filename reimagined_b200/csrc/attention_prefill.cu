// Flash attention on tcgen05 over the cache itself, for portions of prompts.
//
// With one map per head the two query tiles of a CTA (flash.cuh) are 256 queries of a head.  With two maps they are the
// two maps of the same 128 queries: both read the same values, and the epilogue, with both outputs in tensor memory, combines
// them, norms the head and gates it.  Keys come from the cache as K-major sub-tiles; values stay as they are cached, one
// token per row, and enter the second product as an MN-major operand.
// Heads with more than 128 value columns run in chunks of 128 that leave their sums to attention_merge_kernel.
// Roles: warps 0-7 softmax, warp 8 TMA, warp 9 MMA issue.  Every wait is bounded; a role that gives up records the status
// word and falls through to the common exit.
#include <cuda.h>

#include "attention.cuh"
#include "flash.cuh"

namespace tbl {
namespace stack {
namespace {

using namespace flash;

constexpr int kMaxRing = 8;
constexpr int kChunk = 128;                  // value columns of a CTA
constexpr int kVBox = 64 * 128;              // 64 tokens x 64 value columns

struct FlashParams {
    const int32_t *slots, *positions;
    const float* gate;         // [rows][ldg]: gate columns of the projections, or null
    bf16* out;                 // [rows][H * vd]
    float *part_m, *part_l, *part_o;             // heads in chunks: [rows][H][maps] ([vp])
    int* status;
    int ldg, H, G, group, maps, dp, vd, vp, capacity, n_tok, tiles, chunks, k_stages, v_stages, vec;
    float scale_log2, lambda, out_scale, eps;
};

// values as they lie in the cache: 64 columns (128 bytes, swizzled) per token row, groups of 8 tokens 1024 bytes apart (SBO),
// the next 64 columns a box further on (LBO)
__device__ __forceinline__ uint64_t smem_desc_rows(uint32_t addr) {
    return static_cast<uint64_t>((addr & 0x3FFFFu) >> 4) | (static_cast<uint64_t>(kVBox / 16) << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
constexpr uint32_t kTransposeB = 1u << 16;       // instruction descriptor: B is MN-major

__device__ __forceinline__ void softmax_warps_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
static_assert(kSoftWarps * 32 == 256, "the barrier above");

// up to 32 neighbouring outputs of a row, times f and the gate
__device__ __forceinline__ void store_row(const FlashParams& p, const float (&v)[32], float f, int cols, const float* gate, bf16* out) {
    if (p.vec) {                                 // vd % 8 == 0: whole groups of eight
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
            if (i >= cols) break;
            float g[8];
            if (gate) {
                const float4 a = __ldg(reinterpret_cast<const float4*>(gate + i)), b = __ldg(reinterpret_cast<const float4*>(gate + i + 4));
                g[0] = a.x; g[1] = a.y; g[2] = a.z; g[3] = a.w; g[4] = b.x; g[5] = b.y; g[6] = b.z; g[7] = b.w;
            }
            uint32_t y[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float g0 = gate ? sigmoid_f(g[2 * e]) : 1.0f, g1 = gate ? sigmoid_f(g[2 * e + 1]) : 1.0f;
                y[e] = pack_bf16(v[i + 2 * e] * f * g0, v[i + 2 * e + 1] * f * g1);
            }
            *reinterpret_cast<uint4*>(out + i) = make_uint4(y[0], y[1], y[2], y[3]);
        }
    } else {
#pragma unroll
        for (int i = 0; i < 32; ++i)
            if (i < cols) out[i] = __float2bfloat16_rn(v[i] * f * (gate ? sigmoid_f(__ldg(gate + i)) : 1.0f));
    }
}

__global__ void __launch_bounds__(kThreads, 1)
attention_flash_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                       const __grid_constant__ CUtensorMap map_v, const FlashParams p) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const bool two = p.maps == 2;
    const int nsub = (p.dp + 63) / 64;
    const int chunk = blockIdx.y % p.chunks, head = blockIdx.y / p.chunks, seq = blockIdx.z;
    const int vcols = min(kChunk, p.vp - chunk * kChunk), vboxes = (vcols + 63) / 64;
    const int q_bytes = nsub * kSubBytes, k_bytes = p.maps * nsub * kSubBytes, v_bytes = vboxes * kVBox;      // V: 64 tokens per entry
    uint8_t* q_smem = smem;                                    // two tiles
    uint8_t* k_smem = q_smem + 2 * q_bytes;                    // ring of key blocks
    uint8_t* v_smem = k_smem + p.k_stages * k_bytes;           // ring of half blocks of values
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
    const int tile = p.tiles - 1 - blockIdx.x;
    const int q0 = tile * (two ? kBlock : 2 * kBlock);         // first query of the CTA within its sequence's portion
    const int slot = p.slots[seq], pos0 = p.positions[slot] + q0;
    auto blocks_of = [&](int w) {                              // blocks a tile sees
        const int off = two ? 0 : w * kBlock, rows = min(kBlock, p.n_tok - q0 - off);
        return rows > 0 ? min(pos0 + off + rows - 1, p.capacity - 1) / kBlock + 1 : 0;
    };
    const int nblk0 = blocks_of(0), nblk1 = blocks_of(1);
    const int nmax = max(nblk0, nblk1);
    const int row_q = seq * p.n_tok + q0, row_k = (slot * p.G + head / p.group) * p.capacity;

    if (warp == kTmaWarp) {
        // ---------------- TMA ----------------
        if (elect_one()) {
            const int tiles_q = nblk1 > 0 ? 2 : 1;
            mbar_arrive_expect_tx(q_full, tiles_q * q_bytes);
            for (int w = 0; w < tiles_q; ++w)
                for (int s = 0; s < nsub; ++s)
                    tma_load_2d(q_smem + w * q_bytes + s * kSubBytes, &map_q, (two ? head * 2 + w : head) * p.dp + 64 * s,
                                row_q + (two ? 0 : w * kBlock), q_full);
            const int v_col = p.maps * p.dp + chunk * kChunk;
            bool alive = true;
            int vi = 0;
            for (int j = 0; alive && j < nmax; ++j) {
                const int ks = j % p.k_stages;
                if (j >= p.k_stages) alive = mbar_wait_bounded(&k_empty[ks], ((j / p.k_stages) - 1) & 1, p.status);
                if (!alive) break;
                mbar_arrive_expect_tx(&k_full[ks], k_bytes);
                for (int m = 0; m < p.maps; ++m)
                    for (int s = 0; s < nsub; ++s)
                        tma_load_2d(k_smem + ks * k_bytes + (m * nsub + s) * kSubBytes, &map_k, m * p.dp + 64 * s, row_k + j * kBlock, &k_full[ks]);
                for (int h = 0; h < 2; ++h, ++vi) {
                    const int vs = vi % p.v_stages;
                    if (vi >= p.v_stages) alive = mbar_wait_bounded(&v_empty[vs], ((vi / p.v_stages) - 1) & 1, p.status);
                    if (!alive) break;
                    mbar_arrive_expect_tx(&v_full[vs], v_bytes);
                    for (int b = 0; b < vboxes; ++b)
                        tma_load_2d(v_smem + vs * v_bytes + b * kVBox, &map_v, v_col + 64 * b, row_k + j * kBlock + 64 * h, &v_full[vs]);
                }
            }
        }
    } else if (warp == kMmaWarp) {
        // ---------------- MMA ----------------
        if (elect_one()) {
            const uint32_t is = idesc_bf16(kBlock), iv = idesc_bf16(vcols) | kTransposeB;
            bool alive = mbar_wait_bounded(q_full, 0, p.status);
            tc_fence_after();
            // ring positions and descriptors are carried along instead of worked out per product
            const uint64_t q_desc = smem_desc_sw128(smem_u32(q_smem)), k_desc = smem_desc_sw128(smem_u32(k_smem)),
                           v_desc = smem_desc_rows(smem_u32(v_smem));
            const int nd = p.dp / 16;
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
                                umma_f16_ta(o, pc + (k >> 1) * 32 + (k & 1) * 8, bd + 128 * k, iv, (h | k) != 0 ? 1u : (j != 0 ? 1u : 0u));
                                umma_f16_ta(o, pc + (k >> 1) * 32 + (k & 1) * 8 + 16, bd + 128 * k, iv, 1);
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
                        const uint64_t a = q_desc + static_cast<uint64_t>(w) * (q_bytes / 16);
                        const uint64_t b = k_desc + static_cast<uint64_t>(ks) * (k_bytes / 16) + (two ? static_cast<uint64_t>(w) * (q_bytes / 16) : 0);
                        products(tmem + w * kBlock, a, b, nd, is, 0);
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
        const int in_cta = (two ? 0 : w * kBlock) + r;
        const int pos = pos0 + in_cta;                         // sees tokens 0 .. pos
        const uint32_t lanes = static_cast<uint32_t>(quarter * 32) << 16;
        const uint32_t s_col = tmem + lanes + w * kBlock, o_col = tmem + lanes + kOCol + w * 128;
        float m = -INFINITY, l = 0.0f;
        bool alive = true;
        const int n = w == 0 ? nblk0 : nblk1;
        for (int j = 0; j < n; ++j) {
            alive = mbar_wait_bounded(&s_full[w], j & 1, p.status);
            alive = __all_sync(0xffffffffu, alive);
            if (!alive) break;
            tc_fence_after();
            softmax_block(s_col, o_col, vcols, pos - j * kBlock, p.scale_log2, j == 0, m, l, p_full + 2 * w, lane);
        }
        const int q = q0 + in_cta;
        const bool ok = q < p.n_tok;
        const size_t row = static_cast<size_t>(seq) * p.n_tok + (ok ? q : 0);
        const int c0 = chunk * kChunk, cols = min(kChunk, p.vd - c0);          // this CTA's columns of the head
        const float* gate = p.gate ? p.gate + row * p.ldg + head * p.vd : nullptr;
        bf16* out = p.out + (row * p.H + head) * p.vd;
        if (p.chunks > 1) {
            // the sums as they are
            if (alive && n > 0) {
                alive = mbar_wait_bounded(&o_full[w], 0, p.status);
                alive = __all_sync(0xffffffffu, alive);
            }
            if (alive && n > 0) {
                tc_fence_after();
                const size_t unit = (row * p.H + head) * p.maps + (two ? w : 0);
                if (ok && chunk == 0) { p.part_m[unit] = m; p.part_l[unit] = l; }
                float* dst = p.part_o + unit * p.vp + c0;
                for (int ch = 0; ch * 32 < cols; ++ch) {
                    uint32_t x[32];
                    tmem_ld32(o_col + ch * 32, x);
                    tmem_ld_wait();
                    if (ok) {
#pragma unroll
                        for (int i = 0; i < 32; i += 4)
                            if (ch * 32 + i < vcols)          // vp is a multiple of 16
                                *reinterpret_cast<uint4*>(dst + ch * 32 + i) = make_uint4(x[i], x[i + 1], x[i + 2], x[i + 3]);
                    }
                }
            }
        } else if (two) {
            // both maps of a query belong to this CTA: the two groups of warps take alternating blocks of 32 columns.  All
            // products are done once both outputs are, so the query tiles' room serves the exchange of sums.
            if (alive) alive = mbar_wait_bounded(&o_full[0], 0, p.status);
            if (alive) alive = mbar_wait_bounded(&o_full[1], 0, p.status);
            alive = __all_sync(0xffffffffu, alive);
            tc_fence_after();
            float *l_s = reinterpret_cast<float*>(q_smem), *ss_s = l_s + 2 * kBlock;
            l_s[w * kBlock + r] = l;
            softmax_warps_sync();
            const float f0 = 1.0f / l_s[r], f1 = -p.lambda / l_s[kBlock + r];
            const uint32_t o0 = tmem + lanes + kOCol, o1 = o0 + 128;
            float v[2][32], ss = 0.0f;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int ch = w + 2 * i;
                if (alive && ch * 32 < cols) {
                    uint32_t x[32], y[32];
                    tmem_ld32(o0 + ch * 32, x);
                    tmem_ld32(o1 + ch * 32, y);
                    tmem_ld_wait();
#pragma unroll
                    for (int e = 0; e < 32; ++e) {
                        v[i][e] = ch * 32 + e < cols ? fmaf(__uint_as_float(y[e]), f1, __uint_as_float(x[e]) * f0) : 0.0f;
                        ss = fmaf(v[i][e], v[i][e], ss);
                    }
                }
            }
            ss_s[w * kBlock + r] = ss;
            softmax_warps_sync();
            const float f = p.out_scale / sqrtf((ss_s[r] + ss_s[kBlock + r]) / static_cast<float>(p.vd) + p.eps);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int ch = w + 2 * i;
                if (alive && ok && ch * 32 < cols) store_row(p, v[i], f, cols - ch * 32, gate ? gate + ch * 32 : nullptr, out + ch * 32);
            }
        } else if (alive && n > 0) {
            alive = mbar_wait_bounded(&o_full[w], 0, p.status);
            alive = __all_sync(0xffffffffu, alive);
            if (alive) {
                tc_fence_after();
                for (int ch = 0; ch * 32 < cols; ++ch) {
                    uint32_t x[32];
                    float v[32];
                    tmem_ld32(o_col + ch * 32, x);
                    tmem_ld_wait();
#pragma unroll
                    for (int e = 0; e < 32; ++e) v[e] = __uint_as_float(x[e]);
                    if (ok) store_row(p, v, 1.0f / l, cols - ch * 32, gate ? gate + ch * 32 : nullptr, out + ch * 32);
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
constexpr size_t kRoom = 227 * 1024 - kFixedSmem;

struct Rings { int k, v; size_t smem; };

// As many key blocks and value halves as fit; two of each at least.
Rings pick_rings(int maps, int dp, int vp) {
    const size_t q = static_cast<size_t>((dp + 63) / 64) * kSubBytes, k = maps * q;
    const size_t v = static_cast<size_t>((vp < kChunk ? vp : kChunk) + 63) / 64 * kVBox;
    Rings r{2, 2, 0};
    auto bytes = [&](int nk, int nv) { return 2 * q + nk * k + nv * v; };
    if (bytes(2, 2) > kRoom) return Rings{0, 0, 0};
    for (bool grown = true; grown;) {
        grown = false;
        if (r.v < 6 && r.v <= 2 * (r.k - 1) && bytes(r.k, r.v + 1) <= kRoom) { ++r.v; grown = true; }
        else if (r.k < 4 && bytes(r.k + 1, r.v) <= kRoom) { ++r.k; grown = true; }
        else if (r.v < 6 && bytes(r.k, r.v + 1) <= kRoom) { ++r.v; grown = true; }
    }
    r.smem = kFixedSmem + bytes(r.k, r.v);
    return r;
}

}  // namespace

bool attention_flash_supported(const tbl_attention_mixer& m) {
    return m.scale > 0.0f && m.heads * ((m.vdim + kChunk - 1) / kChunk) <= 65535 &&
           pick_rings(m.maps, static_cast<int>(round_up(m.dim, 16)), static_cast<int>(round_up(m.vdim, 16))).k > 0;
}

bool attention_flash_whole(const tbl_attention_mixer& m) { return m.vdim <= kChunk; }

int launch_attention_flash(const AttnParams& p, int n_seq, cudaStream_t st) {
    const long long rows = static_cast<long long>(n_seq) * p.n_tok, cached = static_cast<long long>(p.n_slots) * p.G * p.capacity;
    if (n_seq > 65535 || rows > 2147483647LL || cached > 2147483647LL) return TBL_ERR_SHAPE;
    const Rings rings = pick_rings(p.maps, p.dp, p.vp);
    FlashParams f{};
    f.slots = p.slots; f.positions = p.positions; f.gate = p.g_off < 0 ? nullptr : p.proj + p.g_off; f.out = static_cast<bf16*>(p.out);
    f.part_m = p.part_m; f.part_l = p.part_l; f.part_o = p.part_o; f.status = p.status;
    f.ldg = p.ld; f.H = p.H; f.G = p.G; f.group = p.group; f.maps = p.maps; f.dp = p.dp; f.vd = p.vd; f.vp = p.vp; f.capacity = p.capacity;
    f.n_tok = p.n_tok; f.tiles = ceil_div(p.n_tok, p.maps == 2 ? kBlock : 2 * kBlock); f.chunks = ceil_div(p.vp, kChunk);
    f.k_stages = rings.k; f.v_stages = rings.v; f.vec = p.vec && p.vd % 8 == 0;
    f.scale_log2 = p.scale_log2; f.lambda = p.lambda; f.out_scale = p.out_scale; f.eps = p.eps;
    CUtensorMap mq, mk, mv;
    const auto t = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    if (!make_map(&mq, t, 2, p.q16, rows, static_cast<uint64_t>(p.H) * p.maps * p.dp, 64, kBlock) ||
        !make_map(&mk, t, 2, p.cache, cached, p.cw, 64, kBlock) || !make_map(&mv, t, 2, p.cache, cached, p.cw, 64, 64))
        return TBL_ERR_CUDA;
    static bool done[64] = {};
    if (allow_smem(attention_flash_kernel, rings.smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    return launch_dependent(attention_flash_kernel, dim3(f.tiles, p.H * f.chunks, n_seq), dim3(kThreads), rings.smem, st, mq, mk, mv, f) ==
                   cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace stack
}  // namespace tbl
