// The row operators between the layers of a stack: embedding row or learned average over the depth, the store of
// the residual stream, and the RMS norm that opens the next sublayer, in one kernel.
#include <cooperative_groups.h>

#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

namespace cg = cooperative_groups;

constexpr int kRowThreads = 256;

// A row is handled by a cluster of CL CTAs (few rows: the depth average reads one array per layer, more than one SM
// pulls quickly), each with its share of the columns; the sum of squares goes through distributed shared memory.
template <typename T, int CL>
__global__ void __launch_bounds__(kRowThreads) depth_norm_kernel(const DepthNorm p) {
    extern __shared__ float row[];
    __shared__ float red[kRowThreads / 32];
    __shared__ float part;
    pdl_launch_dependents();
    const int r = blockIdx.x / CL, rank = blockIdx.x % CL;
    const int share = ((p.width + 4 * CL - 1) / (4 * CL)) * 4;
    const int c0 = rank * share, c1 = min(p.width, c0 + share);
    pdl_wait();
    if (p.positions && blockIdx.x == 0)
        for (int s = threadIdx.x; s < p.n_seq; s += kRowThreads) p.positions[p.slots[s]] += p.n_tok;
    float ss = 0.0f;
    if (p.tokens) {
        const int id = p.tokens[r];
        const bool ok = id >= 0 && id < p.vocab;
        const bf16* src = p.table + static_cast<size_t>(ok ? id : 0) * p.width;
        for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
            const float v = ok ? __bfloat162float(src[c]) * p.embed_scale : 0.0f;
            row[c - c0] = v;
            ss += v * v;
        }
    } else {
        const size_t base = static_cast<size_t>(p.row_index ? p.row_index[r] : r) * p.width;
        if ((p.width & 3) == 0) {
            for (int c = c0 + 4 * threadIdx.x; c < c1; c += 4 * kRowThreads) {
                const float* h = p.history + base + c;
                float4 v;
                if (p.weights) {
                    v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    int j = 0;
                    for (; j + 8 <= p.count; j += 8) {
                        float4 t[8];
#pragma unroll
                        for (int q = 0; q < 8; ++q) t[q] = *reinterpret_cast<const float4*>(h + (j + q) * p.stride);
#pragma unroll
                        for (int q = 0; q < 8; ++q) {
                            const float w = __ldg(p.weights + j + q);
                            v.x = fmaf(w, t[q].x, v.x); v.y = fmaf(w, t[q].y, v.y);
                            v.z = fmaf(w, t[q].z, v.z); v.w = fmaf(w, t[q].w, v.w);
                        }
                    }
#pragma unroll 4
                    for (; j < p.count; ++j) {
                        const float4 t = *reinterpret_cast<const float4*>(h + j * p.stride);
                        const float w = __ldg(p.weights + j);
                        v.x = fmaf(w, t.x, v.x); v.y = fmaf(w, t.y, v.y); v.z = fmaf(w, t.z, v.z); v.w = fmaf(w, t.w, v.w);
                    }
                } else {
                    v = *reinterpret_cast<const float4*>(h + (p.count - 1) * p.stride);
                }
                *reinterpret_cast<float4*>(row + c - c0) = v;
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
        } else {
            for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
                const float* h = p.history + base + c;
                float v = 0.0f;
                if (p.weights) {
                    for (int j = 0; j < p.count; ++j) v = fmaf(__ldg(p.weights + j), h[j * p.stride], v);
                } else {
                    v = h[(p.count - 1) * p.stride];
                }
                row[c - c0] = v;
                ss += v * v;
            }
        }
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float total = 0.0f;
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) total += red[w];
    if constexpr (CL > 1) {
        cg::cluster_group cluster = cg::this_cluster();
        if (threadIdx.x == 0) part = total;
        cluster.sync();
        total = 0.0f;
        for (int k = 0; k < CL; ++k) total += *cluster.map_shared_rank(&part, k);
        cluster.sync();      // nobody leaves while a neighbour may still read its partial sum
    }
    const float inv = 1.0f / sqrtf(total / static_cast<float>(p.width) + p.eps);
    const size_t out = static_cast<size_t>(r) * p.width;
    T* h = static_cast<T*>(p.h);
    for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
        const float v = row[c - c0];
        if (p.x) p.x[out + c] = v;
        if (p.trace) p.trace[out + c] = v;
        if (h) h[out + c] = from_f<T>(v * inv * __ldg(p.norm + c));
    }
}

template <typename T, int CL>
int launch_depth_norm_cl(const DepthNorm& p, cudaStream_t st) {
    const int share = ((p.width + 4 * CL - 1) / (4 * CL)) * 4;
    const size_t smem = sizeof(float) * share;
    static bool done[64] = {};
    if (smem > 200 * 1024) return TBL_ERR_SHAPE;
    if (allow_smem(depth_norm_kernel<T, CL>, smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(p.rows * CL); cfg.blockDim = dim3(kRowThreads); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = CL; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr; cfg.numAttrs = CL > 1 ? 2 : 1;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, depth_norm_kernel<T, CL>, p);
    note_launch();
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace

int launch_depth_norm(int precision, const DepthNorm& p, cudaStream_t st) {
    if (p.rows <= 0) return TBL_OK;
    const bool spread = p.rows <= 32 && p.width >= 512;
    if (precision == TBL_BF16) return spread ? launch_depth_norm_cl<bf16, 8>(p, st) : launch_depth_norm_cl<bf16, 1>(p, st);
    return spread ? launch_depth_norm_cl<float, 8>(p, st) : launch_depth_norm_cl<float, 1>(p, st);
}

}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" int tbl_depth_norm(const float* history_dev, size_t history_stride, int count, const float* weights_dev,
                              int precision, const int32_t* row_index_dev, int rows, int width, float eps,
                              const float* norm_dev, float* x_dev, void* h_dev, void* stream) {
    if (!history_dev || count <= 0 || rows <= 0 || width <= 0 || (h_dev && !norm_dev) || (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    DepthNorm p{};
    p.history = history_dev; p.stride = history_stride; p.count = count; p.weights = weights_dev; p.row_index = row_index_dev;
    p.rows = rows; p.width = width; p.eps = eps; p.norm = norm_dev; p.x = x_dev; p.h = h_dev;
    return launch_depth_norm(precision, p, static_cast<cudaStream_t>(stream));
}
