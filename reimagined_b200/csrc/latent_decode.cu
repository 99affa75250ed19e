// Attention over the latent cache on tensor cores: all heads of a block share the cached rows, so a tile of 64 cached
// tokens is one small product with the absorbed queries (S = Q' C^T) and one with the weights (O += P C), and the cache
// is read from memory once per head block.  The products are warp-level MMAs (16 x 8 x 16, bf16): with 16 or 32 heads
// the kernel is bound by the cache's bytes, not by the MMA rate.  Weights are kept as two bf16 terms (hi + lo).
// A CTA handles (row, block of 16 MT heads, split of the context).  The query side of W_uk before it and W_uv with the
// output gate after it are batched products over the heads (dense_rows.cu).
#include "latent.cuh"

namespace tbl {
namespace stack {
namespace {

constexpr int kTile = 64;               // cached tokens per tile
constexpr int kWarps = 8;
constexpr int kSLd = kTile + 4;         // floats between score rows
constexpr int kPLd = kTile + 8;         // bf16 between weight rows: odd number of 16-byte units

__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}

size_t tensor_smem(int width, int heads) {
    return static_cast<size_t>(heads + 2 * kTile) * (width + 8) * 2 + sizeof(float) * heads * kSLd + 2 * 2 * heads * kPLd + sizeof(float) * heads;
}

template <int MT, int TPW>
__global__ void __launch_bounds__(32 * kWarps) latent_tensor_kernel(const LatentParams p) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr int HB = 16 * MT, RPW = HB / kWarps;           // heads of the CTA, score rows per warp
    const int W = p.R + p.rd, ld = W + 8;                    // an odd number of 16-byte units: conflict-free ldmatrix
    bf16* q_s = reinterpret_cast<bf16*>(smem);               // [HB][ld]
    bf16* c_s = q_s + HB * ld;                               // [2][kTile][ld]
    float* s_s = reinterpret_cast<float*>(c_s + 2 * kTile * ld);
    bf16* p_s = reinterpret_cast<bf16*>(s_s + HB * kSLd);    // hi [HB][kPLd], lo
    float* f_s = reinterpret_cast<float*>(p_s + 2 * HB * kPLd);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row = blockIdx.x, h0 = blockIdx.y * HB, split = blockIdx.z;
    pdl_launch_dependents();
    pdl_wait();
    const int slot = p.slots[row / p.n_tok];
    const int n = min(p.positions[slot] + row % p.n_tok + 1, p.capacity);
    const int per = ((n + p.splits - 1) / p.splits + kTile - 1) / kTile * kTile;
    const int t0 = min(split * per, n), t1 = min(n, t0 + per);
    const bf16* cache = static_cast<const bf16*>(p.cache) + static_cast<size_t>(slot) * p.capacity * p.cw;
    const int chunks = W / 8;
    auto load_tile = [&](int stage, int t) {
        const uint32_t base = smem_u32(c_s + stage * kTile * ld);
        // a warp takes every eighth row, its lanes the 16-byte pieces: no division per piece
#pragma unroll
        for (int r = warp; r < kTile; r += kWarps) {
            const bool ok = t + r < t1;
            const bf16* src = cache + static_cast<size_t>(ok ? t + r : 0) * p.cw;
            for (int c = lane; c < chunks; c += 32) cp16(base + (r * ld + c * 8) * 2, src + c * 8, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(0, t0);
    const bf16* qa = static_cast<const bf16*>(p.qa) + static_cast<size_t>(row) * p.H * p.R;
    const int lat_chunks = p.R / 8;
    for (int i = tid; i < HB * lat_chunks; i += 32 * kWarps) {
        const int r = i / lat_chunks, c = i - r * lat_chunks;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h0 + r < p.H) v = *reinterpret_cast<const uint4*>(qa + static_cast<size_t>(h0 + r) * p.R + c * 8);
        *reinterpret_cast<uint4*>(q_s + r * ld + c * 8) = v;
    }
    // the rotated part of the queries, rotated here
    const int half = p.rd / 2, pos = min(n - 1, p.rope_positions - 1);
    const float *cs = p.rope_cos + static_cast<size_t>(pos) * half, *sn = p.rope_sin + static_cast<size_t>(pos) * half;
    for (int i = tid; i < HB * half; i += 32 * kWarps) {
        const int r = i / half, e = i - r * half;
        float a = 0.0f, b = 0.0f;
        if (h0 + r < p.H) {
            const bf16* q = p.q16 + (static_cast<size_t>(row) * p.H + h0 + r) * (p.d + p.rd) + p.d;
            const float u = to_f(q[e]), v = to_f(q[e + half]), c = __ldg(cs + e), s = __ldg(sn + e);
            a = u * c - v * s;
            b = v * c + u * s;
        }
        q_s[r * ld + p.R + e] = __float2bfloat16_rn(a);
        q_s[r * ld + p.R + half + e] = __float2bfloat16_rn(b);
    }
    const int tiles16 = p.R / 16;                            // column tiles of O: warp, warp + 8, ...
    float o[MT][TPW][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < TPW; ++j)
#pragma unroll
            for (int e = 0; e < 8; ++e) o[m][j][e >> 2][e & 3] = 0.0f;
    float mx[RPW], sum[RPW];
#pragma unroll
    for (int i = 0; i < RPW; ++i) { mx[i] = -INFINITY; sum[i] = 0.0f; }
    const float c2 = p.scale * 1.4426950408889634f;
    int stage = 0;
    for (int t = t0; t < t1; t += kTile, stage ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                     // the tile is there, and the other buffer is no longer read
        if (t + kTile < t1) load_tile(stage ^ 1, t + kTile);
        const bf16* ct = c_s + stage * kTile * ld;
        // scores: warp w takes tokens 8w .. 8w + 7
        float s[MT][4], s2[MT][4];                           // two sums each: half as long a chain of dependent MMAs
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[m][e] = s2[m][e] = 0.0f;
        const uint32_t b_addr = smem_u32(ct + (warp * 8 + (lane & 7)) * ld + (lane >> 3) * 8);
        const uint32_t a_addr = smem_u32(q_s + (lane & 15) * ld + (lane >> 4) * 8);
        int k = 0;
#pragma unroll 3
        for (; k + 32 <= W; k += 32) {
            uint32_t b[4], a[4];
            ldsm4(b, b_addr + k * 2);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                ldsm4(a, a_addr + (m * 16 * ld + k) * 2);
                mma(s[m], a, b[0], b[1]);
                ldsm4(a, a_addr + (m * 16 * ld + k + 16) * 2);
                mma(s2[m], a, b[2], b[3]);
            }
        }
        if (k < W) {
            uint32_t b[2], a[4];
            asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(b[0]), "=r"(b[1])
                         : "r"(smem_u32(ct + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8 + k)));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                ldsm4(a, a_addr + (m * 16 * ld + k) * 2);
                mma(s[m], a, b[0], b[1]);
            }
        }
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            float* d = s_s + (m * 16 + (lane >> 2)) * kSLd + warp * 8 + (lane & 3) * 2;
            *reinterpret_cast<float2*>(d) = make_float2(s[m][0] + s2[m][0], s[m][1] + s2[m][1]);
            *reinterpret_cast<float2*>(d + 8 * kSLd) = make_float2(s[m][2] + s2[m][2], s[m][3] + s2[m][3]);
        }
        __syncthreads();
        // softmax: a warp owns RPW score rows, two tokens per lane
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
            const int r = warp * RPW + i;
            const float2 v = *reinterpret_cast<const float2*>(s_s + r * kSLd + 2 * lane);
            const float x0 = t + 2 * lane < t1 ? v.x * c2 : -INFINITY, x1 = t + 2 * lane + 1 < t1 ? v.y * c2 : -INFINITY;
            const float mn = fmaxf(mx[i], warp_max(fmaxf(x0, x1)));          // finite: every tile has a token
            const float f = ex2(mx[i] - mn), p0 = ex2(x0 - mn), p1 = ex2(x1 - mn);
            mx[i] = mn;
            sum[i] = fmaf(sum[i], f, p0 + p1);               // this lane's share
            const uint32_t hi = pack_bf16(p0, p1);
            reinterpret_cast<uint32_t*>(p_s + r * kPLd)[lane] = hi;
            reinterpret_cast<uint32_t*>(p_s + (HB + r) * kPLd)[lane] = pack_bf16(p0 - bf_lo(hi), p1 - bf_hi(hi));
            if (lane == 0) f_s[r] = f;
        }
        __syncthreads();
        // values
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float f0 = f_s[m * 16 + (lane >> 2)], f1 = f_s[m * 16 + 8 + (lane >> 2)];
            if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {
#pragma unroll
                for (int j = 0; j < TPW; ++j)
#pragma unroll
                    for (int q = 0; q < 2; ++q) { o[m][j][q][0] *= f0; o[m][j][q][1] *= f0; o[m][j][q][2] *= f1; o[m][j][q][3] *= f1; }
            }
        }
#pragma unroll
        for (int kk = 0; kk < kTile; kk += 16) {
            uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const uint32_t a = smem_u32(p_s + (m * 16 + (lane & 15)) * kPLd + kk + (lane >> 4) * 8);
                ldsm4(hi[m], a);
                ldsm4(lo[m], a + HB * kPLd * 2);
            }
#pragma unroll
            for (int j = 0; j < TPW; ++j) {
                const int c = warp + kWarps * j;
                if (c < tiles16) {
                    uint32_t b[4];
                    ldsm4t(b, smem_u32(ct + (kk + (lane & 15)) * ld + c * 16 + (lane >> 4) * 8));
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma(o[m][j][0], hi[m], b[0], b[1]);
                        mma(o[m][j][1], hi[m], b[2], b[3]);
                        mma(o[m][j][0], lo[m], b[0], b[1]);
                        mma(o[m][j][1], lo[m], b[2], b[3]);
                    }
                }
            }
        }
    }
    // one split: the result itself; several: the partial sums
    const bool whole = p.splits == 1;
    const size_t unit0 = (static_cast<size_t>(row) * p.H + h0) * p.splits + split;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
        const int r = warp * RPW + i;
        const float l = warp_sum(sum[i]);
        if (lane == 0) f_s[r] = 1.0f / l;
        if (lane == 0 && !whole && h0 + r < p.H) {
            p.part_m[unit0 + static_cast<size_t>(r) * p.splits] = mx[i];
            p.part_l[unit0 + static_cast<size_t>(r) * p.splits] = l;
        }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < TPW; ++j) {
            const int c = warp + kWarps * j;
            if (c >= tiles16) continue;
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int r = m * 16 + e * 8 + (lane >> 2), col = c * 16 + q * 8 + (lane & 3) * 2;
                    if (h0 + r >= p.H) continue;
                    const float a = o[m][j][q][2 * e], b = o[m][j][q][2 * e + 1];
                    if (whole)
                        *reinterpret_cast<uint32_t*>(p.lat + (static_cast<size_t>(row) * p.H + h0 + r) * p.R + col) = pack_bf16(a * f_s[r], b * f_s[r]);
                    else
                        *reinterpret_cast<float2*>(p.part_o + (unit0 + static_cast<size_t>(r) * p.splits) * p.R + col) = make_float2(a, b);
                }
        }
}

// One CTA per (row, head): the splits of the context come together.  Four groups of 128 threads take every fourth split,
// four columns per thread.
constexpr int kMergeThreads = 512;

__global__ void __launch_bounds__(kMergeThreads) latent_merge_kernel(const LatentParams p) {
    __shared__ float fac[1024], red[16], total_s;
    __shared__ float4 part[4][128];
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, col = tid & 127, group = tid >> 7;
    const size_t unit = static_cast<size_t>(blockIdx.x) * p.H + blockIdx.y;
    pdl_wait();
    const float *pm = p.part_m + unit * p.splits, *pl = p.part_l + unit * p.splits;
    float m = -INFINITY;
    for (int s = tid; s < p.splits; s += kMergeThreads) m = fmaxf(m, pm[s]);
    m = warp_max(m);
    if (lane == 0) red[warp] = m;
    __syncthreads();
#pragma unroll
    for (int w = 0; w < 16; ++w) m = fmaxf(m, red[w]);
    float l = 0.0f;
    for (int s = tid; s < p.splits; s += kMergeThreads) {
        fac[s] = ex2(pm[s] - m);
        l = fmaf(pl[s], fac[s], l);
    }
    l = warp_sum(l);
    __syncthreads();
    if (lane == 0) red[warp] = l;
    __syncthreads();
    if (tid == 0) {
        float t = 0.0f;
        for (int w = 0; w < 16; ++w) t += red[w];
        total_s = 1.0f / t;
    }
    float4 a = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (4 * col < p.R) {
        const float* o = p.part_o + unit * p.splits * p.R + 4 * col;
#pragma unroll 8
        for (int s = group; s < p.splits; s += 4) {
            const float4 v = *reinterpret_cast<const float4*>(o + static_cast<size_t>(s) * p.R);
            const float f = fac[s];
            a.x = fmaf(v.x, f, a.x); a.y = fmaf(v.y, f, a.y); a.z = fmaf(v.z, f, a.z); a.w = fmaf(v.w, f, a.w);
        }
    }
    part[group][col] = a;
    __syncthreads();
    if (group == 0 && 4 * col < p.R) {
#pragma unroll
        for (int g = 1; g < 4; ++g) { const float4 v = part[g][col]; a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w; }
        const float t = total_s;
        *reinterpret_cast<uint2*>(p.lat + unit * p.R + 4 * col) = make_uint2(pack_bf16(a.x * t, a.y * t), pack_bf16(a.z * t, a.w * t));
    }
}

template <int MT, int TPW>
cudaError_t launch(const LatentParams& p, int rows, cudaStream_t st) {
    static bool done[64] = {};
    const size_t smem = tensor_smem(p.R + p.rd, 16 * MT);
    const cudaError_t e = allow_smem(latent_tensor_kernel<MT, TPW>, smem, done);
    if (e != cudaSuccess) return e;
    return launch_dependent(latent_tensor_kernel<MT, TPW>, dim3(rows, ceil_div(p.H, 16 * MT), p.splits), dim3(32 * kWarps), smem, st, p);
}

}  // namespace

int latent_tensor_heads(const tbl_latent_mixer& m) { return m.heads > 16 ? 32 : 16; }

bool latent_tensor_supported(const tbl_latent_mixer& m) {
    return m.uk_t && m.dim % 8 == 0 && m.kv_rank % 16 == 0 && m.rot_dim % 16 == 0 && m.kv_rank <= 512 &&
           tensor_smem(m.kv_rank + m.rot_dim, latent_tensor_heads(m)) <= 227 * 1024;
}

int launch_latent_tensor(const LatentParams& p, int rows, cudaStream_t st) {
    DenseCall a{};              // q' = W_uk^T q, all heads in one launch
    a.x = p.q16; a.w = p.uk_t; a.ldx = p.H * (p.d + p.rd); a.M = rows; a.K = p.d; a.N = p.R;
    a.out_b16 = static_cast<bf16*>(p.qa); a.ldo = p.H * p.R;
    a.batch = p.H; a.batch_x = p.d + p.rd; a.batch_w = static_cast<long long>(p.R) * p.d; a.batch_out = p.R;
    int rc = launch_dense(TBL_BF16, kDenseRows, a, st);
    if (rc != TBL_OK) return rc;
    const int tpw = ceil_div(p.R, 16 * kWarps);
    cudaError_t e;
    if (p.H > 16) e = tpw <= 1 ? launch<2, 1>(p, rows, st) : (tpw <= 2 ? launch<2, 2>(p, rows, st) : launch<2, 4>(p, rows, st));
    else e = tpw <= 1 ? launch<1, 1>(p, rows, st) : (tpw <= 2 ? launch<1, 2>(p, rows, st) : launch<1, 4>(p, rows, st));
    if (e != cudaSuccess) return TBL_ERR_CUDA;
    if (p.splits > 1 && launch_dependent(latent_merge_kernel, dim3(rows, p.H), dim3(kMergeThreads), 0, st, p) != cudaSuccess) return TBL_ERR_CUDA;
    DenseCall v{};              // W_uv and the output gate
    v.x = p.lat; v.w = p.uv; v.ldx = p.H * p.R; v.M = rows; v.K = p.R; v.N = p.vd;
    v.out_b16 = static_cast<bf16*>(p.out); v.ldo = p.H * p.vd;
    v.batch = p.H; v.batch_x = p.R; v.batch_w = static_cast<long long>(p.vd) * p.R; v.batch_out = p.vd;
    v.gate = p.proj + p.q_rank + p.R + p.rd; v.ldg = p.ld; v.batch_gate = p.vd;
    return launch_dense(TBL_BF16, kDenseRows, v, st);
}

}  // namespace stack
}  // namespace tbl
