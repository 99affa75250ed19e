// The row operators between the layers of a stack: embedding row, learned average over the depth or update of several
// residual streams, the store of the residual, and the norm that opens the next sublayer (RMS or Dynamic Tanh), in one
// kernel.
#include <cooperative_groups.h>

#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

namespace cg = cooperative_groups;

constexpr int kRowThreads = 256;

// K neighbouring columns of S residual streams: the update by the last sublayer's result, the store, the plain sum, and
// the next sublayer's input u.  `at` is the place in the source arrays, `trace_at` in the trace.
template <int S, int K>
__device__ __forceinline__ void stream_columns(const DepthNorm& p, size_t at, size_t trace_at, const float* embedded, float (&u)[K]) {
    float x[S][K];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        if (embedded) {
#pragma unroll
            for (int k = 0; k < K; ++k) x[s][k] = embedded[k];
        } else if constexpr (K == 4) {
            const float4 t = *reinterpret_cast<const float4*>(p.stream + s * p.stride + at);
            x[s][0] = t.x; x[s][1] = t.y; x[s][2] = t.z; x[s][3] = t.w;
        } else {
            x[s][0] = p.stream[s * p.stride + at];
        }
    }
    if (p.y) {
        float y[K], z[S][K];
        if constexpr (K == 4) {
            const float4 t = *reinterpret_cast<const float4*>(p.y + at);
            y[0] = t.x; y[1] = t.y; y[2] = t.z; y[3] = t.w;
        } else {
            y[0] = p.y[at];
        }
#pragma unroll
        for (int t = 0; t < S; ++t) {
#pragma unroll
            for (int k = 0; k < K; ++k) z[t][k] = __ldg(p.out_weights + t) * y[k];
#pragma unroll
            for (int s = 0; s < S; ++s) {
                const float m = __ldg(p.mix + s * S + t);
#pragma unroll
                for (int k = 0; k < K; ++k) z[t][k] = fmaf(m, x[s][k], z[t][k]);
            }
        }
#pragma unroll
        for (int s = 0; s < S; ++s)
#pragma unroll
            for (int k = 0; k < K; ++k) x[s][k] = z[s][k];
    }
    if (p.store) {
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if constexpr (K == 4) *reinterpret_cast<float4*>(p.stream + s * p.stride + at) = make_float4(x[s][0], x[s][1], x[s][2], x[s][3]);
            else p.stream[s * p.stride + at] = x[s][0];
        }
    }
#pragma unroll
    for (int k = 0; k < K; ++k) {
        float sum = 0.0f;
        u[k] = 0.0f;
#pragma unroll
        for (int s = 0; s < S; ++s) {
            sum += x[s][k];
            u[k] = p.weights ? fmaf(__ldg(p.weights + s), x[s][k], u[k]) : sum;
        }
        if (p.trace) p.trace[trace_at + k] = sum;
    }
}

// A row is handled by a cluster of CL CTAs (few rows: the depth average reads one array per layer, more than one SM
// pulls quickly), each with its share of the columns; the sum of squares goes through distributed shared memory.
// S: residual streams, 0 for a single one.
template <typename T, int CL, int S>
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
    if constexpr (S > 0) {
        const size_t own = static_cast<size_t>(r) * p.width;
        const size_t base = p.row_index ? static_cast<size_t>(p.row_index[r]) * p.width : own;
        const int id = p.tokens ? p.tokens[r] : 0;
        const bool ok = id >= 0 && id < p.vocab;
        const bf16* src = p.table + static_cast<size_t>(ok ? id : 0) * p.width;
        if ((p.width & 3) == 0) {
            for (int c = c0 + 4 * threadIdx.x; c < c1; c += 4 * kRowThreads) {
                float e[4], u[4];
                if (p.tokens) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) e[k] = ok ? __bfloat162float(src[c + k]) * p.embed_scale : 0.0f;
                }
                stream_columns<S, 4>(p, base + c, own + c, p.tokens ? e : nullptr, u);
                *reinterpret_cast<float4*>(row + c - c0) = make_float4(u[0], u[1], u[2], u[3]);
                ss += u[0] * u[0] + u[1] * u[1] + u[2] * u[2] + u[3] * u[3];
            }
        } else {
            for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
                float e[1], u[1];
                if (p.tokens) e[0] = ok ? __bfloat162float(src[c]) * p.embed_scale : 0.0f;
                stream_columns<S, 1>(p, base + c, own + c, p.tokens ? e : nullptr, u);
                row[c - c0] = u[0];
                ss += u[0] * u[0];
            }
        }
    } else if (p.tokens) {
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
    float inv = 0.0f;
    if (p.norm_kind == TBL_NORM_RMS) {
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
        inv = 1.0f / sqrtf(total / static_cast<float>(p.width) + p.eps);
    } else {
        __syncthreads();
    }
    const size_t out = static_cast<size_t>(r) * p.width;
    T* h = static_cast<T*>(p.h);
    for (int c = c0 + threadIdx.x; c < c1; c += kRowThreads) {
        const float v = row[c - c0];
        if (p.x) p.x[out + c] = v;
        if (S == 0 && p.trace) p.trace[out + c] = v;
        if (h)
            h[out + c] = from_f<T>(p.norm_kind == TBL_NORM_RMS ? v * inv * __ldg(p.norm + c)
                                                               : fmaf(tanhf(p.alpha * v), __ldg(p.norm + c), __ldg(p.norm_bias + c)));
    }
}

template <typename T, int CL, int S>
int launch_depth_norm_cl(const DepthNorm& p, cudaStream_t st) {
    const int share = ((p.width + 4 * CL - 1) / (4 * CL)) * 4;
    const size_t smem = sizeof(float) * share;
    static bool done[64] = {};
    if (smem > 200 * 1024) return TBL_ERR_SHAPE;
    if (allow_smem(depth_norm_kernel<T, CL, S>, smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3(p.rows * CL); cfg.blockDim = dim3(kRowThreads); cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = CL; attr[1].val.clusterDim.y = 1; attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr; cfg.numAttrs = CL > 1 ? 2 : 1;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, depth_norm_kernel<T, CL, S>, p);
    note_launch();
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

template <typename T, int CL>
int launch_depth_norm_streams(const DepthNorm& p, cudaStream_t st) {
    switch (p.streams) {
        case 0: return launch_depth_norm_cl<T, CL, 0>(p, st);
        case 1: return launch_depth_norm_cl<T, CL, 1>(p, st);
        case 2: return launch_depth_norm_cl<T, CL, 2>(p, st);
        case 3: return launch_depth_norm_cl<T, CL, 3>(p, st);
        case 4: return launch_depth_norm_cl<T, CL, 4>(p, st);
        case 5: return launch_depth_norm_cl<T, CL, 5>(p, st);
        case 6: return launch_depth_norm_cl<T, CL, 6>(p, st);
        case 7: return launch_depth_norm_cl<T, CL, 7>(p, st);
        case 8: return launch_depth_norm_cl<T, CL, 8>(p, st);
        default: return TBL_ERR_UNSUPPORTED;
    }
}

}  // namespace

int launch_depth_norm(int precision, const DepthNorm& p, cudaStream_t st) {
    static_assert(TBL_MAX_STREAMS == 8, "the cases above");
    if (p.rows <= 0) return TBL_OK;
    const bool spread = p.rows <= 32 && p.width >= 512;
    if (precision == TBL_BF16) return spread ? launch_depth_norm_streams<bf16, 8>(p, st) : launch_depth_norm_streams<bf16, 1>(p, st);
    return spread ? launch_depth_norm_streams<float, 8>(p, st) : launch_depth_norm_streams<float, 1>(p, st);
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

extern "C" int tbl_stream_norm(float* streams_dev, size_t stride, int streams, const float* y_dev, const float* mix_dev,
                               const float* out_weights_dev, int store, const float* in_weights_dev, int precision,
                               const int32_t* row_index_dev, int rows, int width, int norm_kind, float eps, float alpha,
                               const float* norm_dev, const float* norm_bias_dev, float* sum_dev, void* h_dev, void* stream) {
    if (!streams_dev || streams <= 0 || rows <= 0 || width <= 0 || (h_dev && !norm_dev) || (y_dev && (!mix_dev || !out_weights_dev)) ||
        (row_index_dev && store) || (precision != TBL_F32 && precision != TBL_BF16) ||
        (norm_kind != TBL_NORM_RMS && norm_kind != TBL_NORM_DYNAMIC_TANH) || (norm_kind == TBL_NORM_DYNAMIC_TANH && h_dev && !norm_bias_dev))
        return TBL_ERR_INVALID_ARG;
    if (streams > TBL_MAX_STREAMS) return TBL_ERR_UNSUPPORTED;
    if (width % 4 == 0 && (stride % 4 || (reinterpret_cast<uintptr_t>(streams_dev) & 15) || (reinterpret_cast<uintptr_t>(y_dev) & 15)))
        return TBL_ERR_ALIGNMENT;
    DepthNorm p{};
    p.stream = streams_dev; p.stride = stride; p.streams = streams; p.y = y_dev; p.mix = mix_dev; p.out_weights = out_weights_dev;
    p.store = store; p.weights = in_weights_dev; p.row_index = row_index_dev; p.rows = rows; p.width = width;
    p.norm_kind = norm_kind; p.eps = eps; p.alpha = alpha; p.norm = norm_dev; p.norm_bias = norm_bias_dev; p.trace = sum_dev; p.h = h_dev;
    return launch_depth_norm(precision, p, static_cast<cudaStream_t>(stream));
}
