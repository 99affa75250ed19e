// Attention of a few query rows over a long cache (decode, short portions): the cache streams through shared memory once
// per block of 16 query rows that share a key/value head.
//
// A CTA handles (sequence, kv head, block of rows, split of the context) in tiles of 64 tokens, brought in by TMA ahead of
// their use as sub-tiles of 64 columns with the 128-byte swizzle (conflict-free for ldmatrix).  The products are warp-level
// MMAs (16 x 8 x 16, bf16): a warp owns one map and 16 tokens of every tile, with its own maximum, sum and output, so that
// a tile costs one barrier; the quarters meet in shared memory at the end.
// The scores' fragments become the weights' fragments in place, as two bf16 terms (hi + lo: 16 bits of mantissa).
// The splits of the context are a cluster: its CTAs read each other's sums through distributed shared memory, combine the
// maps, norm the heads and gate the output, a row at a time each.  Only a context that wants more CTAs than a cluster has
// leaves partial sums for attention_merge_kernel.  A decode step appends its token here: the CTA whose split holds it
// takes it from the projections and writes it to the cache.
#include <cooperative_groups.h>
#include <cuda.h>

#include "attention.cuh"
#include "tc05.cuh"

namespace tbl {
namespace stack {
namespace {

namespace cg = cooperative_groups;

constexpr int kTile = 64, kRows = 16, kQuarters = 4, kMaxStages = 4;
constexpr float kRescale = 8.0f;

constexpr int kSub = kTile * 128;               // bytes of a sub-tile: 64 tokens x 64 columns
__host__ __device__ __forceinline__ int sub_tiles(int cw) { return (cw + 63) / 64; }

size_t query_smem(int maps, int dp) { return 2 * static_cast<size_t>(kRows) * maps * (dp + 8); }
size_t merge_smem(int maps, int vp) { return sizeof(float) * kQuarters * maps * kRows * static_cast<size_t>(vp); }
size_t tiles_smem(int maps, int dp, int vp, int stages) {
    const size_t tiles = static_cast<size_t>(stages) * sub_tiles(maps * dp + vp) * kSub, merge = merge_smem(maps, vp);
    return tiles > merge ? tiles : merge;
}
size_t stream_smem(int maps, int dp, int vp, int stages) { return 1024 + tiles_smem(maps, dp, vp, stages) + query_smem(maps, dp); }

// MAPS: maps per head; VN: value columns in steps of 16 a warp has room for.  clustered: the splits are a cluster
template <int MAPS, int VN>
__global__ void __launch_bounds__(32 * kQuarters * MAPS) attention_stream_kernel(const __grid_constant__ CUtensorMap map_c, const AttnParams p,
                                                                               const int stages, const int q_at, const int clustered) {
    constexpr int kThreads = 32 * kQuarters * MAPS;
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    __shared__ float m_s[kQuarters][MAPS][kRows], l_s[kQuarters][MAPS][kRows], top_s[MAPS][kRows], sum_s[MAPS][kRows], red_s[kQuarters * MAPS];
    __shared__ float fac_s[MAPS][kClusterSplits];
    __shared__ __align__(8) uint64_t full[kMaxStages];
    const int ldq = p.dp + 8, tile_bytes = sub_tiles(p.cw) * kSub;
    uint8_t* t_s = smem;                                                // [stages][sub-tile][64 tokens][128 bytes]
    float* o_s = reinterpret_cast<float*>(smem);                        // afterwards: [quarter][MAPS][16][vp]
    bf16* q_s = reinterpret_cast<bf16*>(smem + q_at);                   // [MAPS][16][ldq]
    const int tid = threadIdx.x, warp = tc05::uniform_warp(), lane = tid & 31, map = warp % MAPS, quarter = warp / MAPS;
    const int seq = blockIdx.x / p.G, g = blockIdx.x % p.G, first = blockIdx.y * kRows, split = blockIdx.z;
    const int total = p.n_tok * p.group;
    if (tid == 0) {
        for (int s = 0; s < kMaxStages; ++s) mbar_init(&full[s], 1);
        fence_mbar_init();
        fence_proxy_async();
    }
    __syncthreads();
    pdl_wait();
    const int slot = p.slots[seq], pos0 = p.positions[slot];
    const int n = min(pos0 + min(total - 1, first + kRows - 1) / p.group + 1, p.capacity);       // tokens the last row sees
    const int per = ((n + p.splits - 1) / p.splits + kTile - 1) / kTile * kTile;
    const int t0 = min(split * per, n), t1 = min(n, t0 + per);
    bf16* cache = static_cast<bf16*>(p.cache) + cache_row(p, slot, g, 0);
    // a decode step's token (n_tok == 1, at pos0) comes from the projections, not from the cache
    int fresh = -1;
    if (p.append) {
        if (pos0 < 0 || pos0 >= p.capacity || (p.temperature && pos0 >= p.temperature_positions)) {
            if (tid == 0 && split == 0) atomicOr(p.status, TBL_DEV_CACHE_FULL);
        } else {
            if (pos0 >= t0 && pos0 < t1) fresh = pos0;
        }
    }
    // Rows past the split's end come along: their tokens are masked, and a weight of zero only needs a finite value beside it.
    const int row0 = (slot * p.G + g) * p.capacity;
    auto load_tile = [&](int stage, int t) {
        if (warp == 0 && t < t1 && tc05::elect_one()) {
            mbar_arrive_expect_tx(&full[stage], tile_bytes);
            for (int c = 0; c * 64 < p.cw; ++c) tc05::tma_load_2d(t_s + stage * tile_bytes + c * kSub, &map_c, c * 64, row0 + t, &full[stage]);
        }
    };
    for (int s = 0; s < kMaxStages - 1; ++s)
        if (s < stages - 1) load_tile(s, t0 + s * kTile);
    for (int i = tid; i < MAPS * kRows * p.dp; i += kThreads) {
        const int r = i / (MAPS * p.dp), e = i - r * MAPS * p.dp, m = e / p.dp, c = e - m * p.dp, at = first + r;
        float q = 0.0f;
        if (at < total && c < p.d) {
            const int t = at / p.group, head = g * p.group + at % p.group;
            q = p.proj[(static_cast<size_t>(seq) * p.n_tok + t) * p.ld + (head * MAPS + m) * p.d + c] * temperature_of(p, pos0 + t);
        }
        q_s[(m * kRows + r) * ldq + c] = __float2bfloat16_rn(q);
    }
    float o[VN][2][4];
#pragma unroll
    for (int j = 0; j < VN; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[j][e >> 2][e & 3] = 0.0f;
    float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};       // rows lane / 4 and lane / 4 + 8; this lane's share of the sums
    int last[2];                                                        // last token each of them sees
#pragma unroll
    for (int h = 0; h < 2; ++h) last[h] = min(pos0 + min(first + (lane >> 2) + 8 * h, total - 1) / p.group, t1 - 1);
    const int tiles16 = p.vp / 16;
    const uint32_t a_addr = smem_u32(q_s + (map * kRows + (lane & 15)) * ldq + (lane >> 4) * 8);
    const bool upper = total - first > kRows / 2;                      // rows 8 .. 15 in use
    const int all_see = min(pos0 + first / p.group, t1 - 1);            // the last token that every row sees
    bool alive = true;
    uint32_t phase = 0;
    int stage = 0;
    for (int t = t0; t < t1; t += kTile) {
        // (after a wait that gave up nothing more is asked for, and what is on its way gets a short time)
        alive = __all_sync(0xffffffffu, mbar_wait_bounded(&full[stage], phase, p.status, alive ? kWaitSpinLimit : 1024)) && alive;
        __syncthreads();                                     // the tile is there, and the one before it is no longer read
        {
            const int ahead = stage == 0 ? stages - 1 : stage - 1;
            if (alive) load_tile(ahead, t + (stages - 1) * kTile);
        }
        if (fresh >= t && fresh < t + kTile) {               // in the last tile of one split
            const float* pr = p.proj + static_cast<size_t>(seq) * p.ld;
            for (int c = tid; c < p.cw; c += kThreads) {
                const bf16 v = __float2bfloat16_rn(cache_value(p, pr, g, c));
                const int r = fresh - t;
                reinterpret_cast<bf16*>(t_s + stage * tile_bytes + (c >> 6) * kSub + r * 128 + ((((c >> 3) & 7) ^ (r & 7)) << 4))[c & 7] = v;
                cache[static_cast<size_t>(fresh) * p.cw + c] = v;
            }
            __syncthreads();
        }
        const uint32_t tile = smem_u32(t_s + stage * tile_bytes) + quarter * 16 * 128;
        if (++stage == stages) { stage = 0; phase ^= 1; }
        // scores: 16 rows x 16 tokens
        float s[2][4] = {};
        const uint32_t k_row = tile + ((lane & 7) + (lane >> 4) * 8) * 128;
        const uint32_t k_mix = ((lane >> 3) & 1) ^ (lane & 7);            // 16-byte piece c of a row r lies at c ^ (r & 7)
#pragma unroll 4
        for (int k = 0; k < p.dp; k += 16) {
            uint32_t a[4], b[4];
            const int piece = (map * p.dp + k) >> 3;
            ldsm4(a, a_addr + k * 2);
            ldsm4(b, k_row + (piece >> 3) * kSub + (((piece & 7) ^ k_mix) << 4));
            mma(s[0], a, b[0], b[1]);
            mma(s[1], a, b[2], b[3]);
        }
        const int token = t + quarter * 16 + (lane & 3) * 2;
        const bool whole = t + kTile - 1 <= all_see;         // nothing of the tile is masked
        uint32_t hi[4] = {}, lo[4] = {};
        float f[2] = {1.0f, 1.0f};
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            if (h == 1 && !upper) break;
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] = s[e >> 1][2 * h + (e & 1)] * p.scale_log2;
            if (!whole) {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (token + (e >> 1) * 8 + (e & 1) > last[h]) x[e] = -INFINITY;
            }
            float top = fmaxf(fmaxf(x[0], x[1]), fmaxf(x[2], x[3]));
            top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
            top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
            // the maximum only moves when it grows by 2^8: then output and sum are rescaled
            const float mn = top > mx[h] + kRescale ? top : mx[h], base = mn == -INFINITY ? 0.0f : mn;   // nothing seen yet: all weights zero
            f[h] = mn == mx[h] ? 1.0f : ex2(mx[h] - base);
            mx[h] = mn;
#pragma unroll
            for (int e = 0; e < 4; ++e) x[e] = ex2(x[e] - base);
            sum[h] = fmaf(sum[h], f[h], (x[0] + x[1]) + (x[2] + x[3]));
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                hi[2 * e + h] = pack_bf16(x[2 * e], x[2 * e + 1]);
                lo[2 * e + h] = pack_bf16(x[2 * e] - bf_lo(hi[2 * e + h]), x[2 * e + 1] - bf_hi(hi[2 * e + h]));
            }
        }
        if (__any_sync(0xffffffffu, f[0] != 1.0f || f[1] != 1.0f)) {
#pragma unroll
            for (int j = 0; j < VN; ++j)
#pragma unroll
                for (int q = 0; q < 2; ++q) { o[j][q][0] *= f[0]; o[j][q][1] *= f[0]; o[j][q][2] *= f[1]; o[j][q][3] *= f[1]; }
        }
        const uint32_t v_row = tile + (lane & 15) * 128, v_mix = (lane >> 4) ^ (lane & 7);
#pragma unroll
        for (int j = 0; j < VN; ++j) {
            if (j < tiles16) {
                uint32_t b[4];
                const int piece = (MAPS * p.dp >> 3) + 2 * j;
                ldsm4t(b, v_row + (piece >> 3) * kSub + (((piece & 7) ^ v_mix) << 4));
                mma(o[j][0], hi, b[0], b[1]);
                mma(o[j][1], hi, b[2], b[3]);
                mma(o[j][0], lo, b[0], b[1]);
                mma(o[j][1], lo, b[2], b[3]);
            }
        }
    }
    __syncthreads();                                         // tiles are done with: their room takes the outputs
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 1);
        sum[h] += __shfl_xor_sync(0xffffffffu, sum[h], 2);
        if ((lane & 3) == 0) { m_s[quarter][map][(lane >> 2) + 8 * h] = mx[h]; l_s[quarter][map][(lane >> 2) + 8 * h] = sum[h]; }
    }
    float* mine = o_s + static_cast<size_t>((quarter * MAPS + map) * kRows) * p.vp;
#pragma unroll
    for (int j = 0; j < VN; ++j)
        if (j < tiles16) {
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
                for (int h = 0; h < 2; ++h)
                    *reinterpret_cast<float2*>(mine + ((lane >> 2) + 8 * h) * p.vp + j * 16 + q * 8 + (lane & 3) * 2) =
                        make_float2(o[j][q][2 * h], o[j][q][2 * h + 1]);
        }
    __syncthreads();
    pdl_launch_dependents();
    // the quarters come together: sums of this split, a warp per row
    const size_t quarter_step = static_cast<size_t>(MAPS) * kRows * p.vp;
    const int rows = min(kRows, total - first);
    for (int r = warp; r < rows; r += kQuarters * MAPS) {
#pragma unroll
        for (int m = 0; m < MAPS; ++m) {
            float fac[kQuarters], top = m_s[0][m][r], l = 0.0f;
#pragma unroll
            for (int k = 1; k < kQuarters; ++k) top = fmaxf(top, m_s[k][m][r]);
#pragma unroll
            for (int k = 0; k < kQuarters; ++k) {
                fac[k] = m_s[k][m][r] == -INFINITY ? 0.0f : ex2(m_s[k][m][r] - top);
                l = fmaf(l_s[k][m][r], fac[k], l);
            }
            if (lane == 0) { top_s[m][r] = top; sum_s[m][r] = l; }
            float* src = o_s + static_cast<size_t>(m * kRows + r) * p.vp;
            for (int c = lane; c < p.vd; c += 32) {
                float v = 0.0f;
#pragma unroll
                for (int k = 0; k < kQuarters; ++k) v = fmaf(src[k * quarter_step + c], fac[k], v);
                src[c] = v;                                  // over the first quarter, which only this lane reads
            }
        }
    }
    if (p.splits > 1 && !clustered) {
        __syncwarp();
        for (int r = warp; r < rows; r += kQuarters * MAPS) {
            const int t = (first + r) / p.group, head = g * p.group + (first + r) % p.group;
            const size_t unit = ((static_cast<size_t>(seq) * p.n_tok + t) * p.H + head) * MAPS;
#pragma unroll
            for (int m = 0; m < MAPS; ++m) {
                const size_t u = (unit + m) * p.splits + split;
                if (lane == 0) { p.part_m[u] = top_s[m][r]; p.part_l[u] = sum_s[m][r]; }
                for (int c = lane; c < p.vd; c += 32) p.part_o[u * p.vp + c] = o_s[static_cast<size_t>(m * kRows + r) * p.vp + c];
            }
        }
        return;
    }
    cg::cluster_group cluster = cg::this_cluster();
    if (p.splits > 1) cluster.sync();
    else __syncthreads();
    // a row at a time: row r is finished by split r mod splits.  v_s (the second quarter's room, read by nobody else): the
    // maps' weighted averages.
    float* v_s = o_s + quarter_step;
    for (int r = split; r < rows; r += p.splits) {
        if (warp < MAPS) {                                   // a lane per split
            const float top = lane < p.splits ? *cluster.map_shared_rank(&top_s[warp][r], lane) : -INFINITY;
            const float l = lane < p.splits ? *cluster.map_shared_rank(&sum_s[warp][r], lane) : 0.0f;
            const float most = warp_max(top), f = top == -INFINITY ? 0.0f : ex2(top - most);
            const float total_l = warp_sum(l * f);
            if (lane < kClusterSplits) fac_s[warp][lane] = f * ((warp == 0 ? 1.0f : -p.lambda) / total_l);
        }
        __syncthreads();
        for (int i = tid; i < MAPS * p.vp; i += kThreads) {
            const int m = MAPS == 2 && i >= p.vp, c = i - m * p.vp;
            const float* src = o_s + static_cast<size_t>(m * kRows + r) * p.vp + (c < p.vd ? c : 0);
            float v = 0.0f;
#pragma unroll
            for (int k = 0; k < kClusterSplits; ++k)
                if (k < p.splits) v = fmaf(*cluster.map_shared_rank(src, k), fac_s[m][k], v);
            v_s[i] = v;
        }
        __syncthreads();
        float x[VN * 16 / kThreads + 1], ss = 0.0f;
#pragma unroll
        for (int i = 0; i < VN * 16 / kThreads + 1; ++i) {
            const int c = tid + i * kThreads;
            x[i] = c < p.vd ? v_s[c] + (MAPS == 2 ? v_s[p.vp + c] : 0.0f) : 0.0f;
            ss = fmaf(x[i], x[i], ss);
        }
        float f = 1.0f;
        if (MAPS == 2) {
            ss = warp_sum(ss);
            if (lane == 0) red_s[warp] = ss;
            __syncthreads();
            ss = 0.0f;
#pragma unroll
            for (int k = 0; k < kQuarters * MAPS; ++k) ss += red_s[k];
            f = p.out_scale / sqrtf(ss / static_cast<float>(p.vd) + p.eps);
        }
        const int t = (first + r) / p.group, head = g * p.group + (first + r) % p.group;
        const size_t row = static_cast<size_t>(seq) * p.n_tok + t;
        const float* gate = p.g_off < 0 ? nullptr : p.proj + row * p.ld + p.g_off + head * p.vd;
        bf16* out = static_cast<bf16*>(p.out) + (row * p.H + head) * p.vd;
#pragma unroll
        for (int i = 0; i < VN * 16 / kThreads + 1; ++i) {
            const int c = tid + i * kThreads;
            if (c < p.vd) out[c] = __float2bfloat16_rn(x[i] * f * (gate ? sigmoid_f(gate[c]) : 1.0f));
        }
        __syncthreads();                                     // v_s, red_s and fac_s are free again
    }
    if (p.splits > 1) cluster.sync();                        // nobody leaves while a neighbour may still read its sums
}

// Tiles in shared memory: two CTAs of an SM take no more than kShare together.  Shared memory comes off the SM's first-level
// cache, and the linear layers on either side, whose CTAs share the SM with this kernel's, read their activations through that.
constexpr size_t kShare = 160 * 1024;

int pick_stages(int maps, int dp, int vp) {
    for (int s = kMaxStages; s > 2; --s)
        if (stream_smem(maps, dp, vp, s) <= kShare / 2) return s;
    return stream_smem(maps, dp, vp, 2) <= 220 * 1024 ? 2 : 0;
}

template <int MAPS, int VN>
cudaError_t launch(const AttnParams& p, int n_seq, cudaStream_t st) {
    static bool done[64] = {};
    const dim3 grid(n_seq * p.G, ceil_div(static_cast<long long>(p.n_tok) * p.group, kRows), p.splits);
    const int stages = pick_stages(MAPS, p.dp, p.vp);
    const size_t smem = stream_smem(MAPS, p.dp, p.vp, stages);
    const cudaError_t e = allow_smem(attention_stream_kernel<MAPS, VN>, smem, done);
    if (e != cudaSuccess) return e;
    if (grid.y > 65535) return cudaErrorInvalidValue;
    const bool clustered = p.splits > 1 && p.splits <= kClusterSplits;
    const long long cached = static_cast<long long>(p.n_slots) * p.G * p.capacity;
    CUtensorMap map_c;
    if (cached > 2147483647LL || !tc05::make_map(&map_c, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.cache, cached, p.cw, 64, kTile))
        return cudaErrorInvalidValue;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid; cfg.blockDim = dim3(32 * kQuarters * MAPS); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = 1; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = p.splits;
    cfg.attrs = attr; cfg.numAttrs = clustered ? 2 : 1;
    const cudaError_t r = cudaLaunchKernelEx(&cfg, attention_stream_kernel<MAPS, VN>, map_c, p, stages,
                                             static_cast<int>(tiles_smem(MAPS, p.dp, p.vp, stages)), static_cast<int>(clustered));
    note_launch();
    return r;
}

template <int MAPS>
cudaError_t launch_vn(const AttnParams& p, int n_seq, cudaStream_t st) {
    if (p.vp <= 64) return launch<MAPS, 4>(p, n_seq, st);
    if (p.vp <= 128) return launch<MAPS, 8>(p, n_seq, st);
    return launch<MAPS, 16>(p, n_seq, st);
}

}  // namespace

bool attention_stream_supported(const tbl_attention_mixer& m) {
    const int dp = static_cast<int>(round_up(m.dim, 16)), vp = static_cast<int>(round_up(m.vdim, 16));
    return vp <= 256 && pick_stages(m.maps, dp, vp) > 0;
}

int launch_attention_stream(const AttnParams& p, int n_seq, cudaStream_t st) {
    return (p.maps == 2 ? launch_vn<2>(p, n_seq, st) : launch_vn<1>(p, n_seq, st)) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace stack
}  // namespace tbl
