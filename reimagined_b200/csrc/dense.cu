// Linear layers with bf16 weights: the kernel choice, the SIMT kernel (any shape, true fp32 arithmetic) and the fp32
// GEMV for a few rows.  The weight-streaming kernel for bf16 rows is in dense_rows.cu, the tcgen05 GEMM in
// dense_tcgen05.cu.
#include "stack.cuh"

namespace tbl {
namespace stack {
namespace {

__device__ __forceinline__ void store_out(const DenseCall& c, int m, int n, float v) {
    if (c.bias) v += __ldg(c.bias + n);
    if (c.out_f32) {
        const size_t i = static_cast<size_t>(m) * c.ldo + n;
        c.out_f32[i] = c.residual ? c.residual[i] + v : v;
    } else {
        c.out_b16[static_cast<size_t>(m) * c.ldo + n] = __float2bfloat16_rn(v);
    }
}

// One output of a gated pair: rows g and g + 32 of the weight are the gate and up rows of output column n.
__device__ __forceinline__ void store_pair(const DenseCall& c, int m, int n, int g, float gate, float up) {
    if (c.bias) { gate += __ldg(c.bias + g); up += __ldg(c.bias + g + TBL_PAIR_BLOCK); }
    const float v = activate(activation_of(c.act), gate) * up;
    if (c.out_f32) c.out_f32[static_cast<size_t>(m) * c.ldo + n] = v;
    else c.out_b16[static_cast<size_t>(m) * c.ldo + n] = __float2bfloat16_rn(v);
}

// ---- SIMT: 64 x 64 tile, 4 x 4 outputs per thread (columns tx + 16 j, so that a thread holds whole gated pairs) ----
template <typename T>
__global__ void __launch_bounds__(256) dense_simt_kernel(const DenseCall c) {
    constexpr int BK = 16;
    __shared__ float xs[BK][64 + 4], ws[BK][64 + 4];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const T* x = static_cast<const T*>(c.x);
    float acc[4][4] = {};
    pdl_launch_dependents();
    pdl_wait();
    for (int k0 = 0; k0 < c.K; k0 += BK) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = threadIdx.x + i * 256, k = e & 15, r = e >> 4;
            const int kk = k0 + k;
            xs[k][r] = (m0 + r < c.M && kk < c.K) ? to_f(x[static_cast<size_t>(m0 + r) * c.ldx + kk]) : 0.0f;
            ws[k][r] = (n0 + r < c.N && kk < c.K) ? to_f(c.w[static_cast<size_t>(n0 + r) * c.ldw + kk]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty + 16 * i]; b[i] = ws[k][tx + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty + 16 * i;
        if (m >= c.M) continue;
        if (c.pair_cols) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int g = n0 + tx + 16 * j, n = (n0 >> 1) + tx + 16 * j;
                if (n < c.pair_cols) store_pair(c, m, n, g, acc[i][j], acc[i][j + 2]);
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tx + 16 * j < c.N) store_out(c, m, n0 + tx + 16 * j, acc[i][j]);
        }
    }
}

// ---- GEMV: 1 .. 4 rows; the weights stream through registers once -------------------------------------------------
// A warp owns R weight rows (of a gated layer: R / 2 gate rows and their up rows) and walks K in steps of 256 elements,
// a 16-byte load per lane and row; the activation rows sit in shared memory as fp32.  The first weight loads are issued
// before the wait on the preceding kernel of the step.
constexpr int kGemvWarps = 8;
constexpr int kGemvMaxRows = 4;
constexpr size_t kGemvMaxSmem = 200 * 1024;

template <typename T, int M, int R>
__global__ void __launch_bounds__(32 * kGemvWarps) dense_gemv_kernel(const DenseCall c) {
    extern __shared__ __align__(16) float xs[];          // [M][K]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * kGemvWarps + warp;
    int rows[R];
    if (c.pair_cols) {
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
            const int n = unit * (R / 2) + i;             // output column
            rows[2 * i] = (n / TBL_PAIR_BLOCK) * 2 * TBL_PAIR_BLOCK + n % TBL_PAIR_BLOCK;
            rows[2 * i + 1] = rows[2 * i] + TBL_PAIR_BLOCK;
        }
    } else {
#pragma unroll
        for (int i = 0; i < R; ++i) rows[i] = unit * R + i;
    }
    const bf16* wp[R];
#pragma unroll
    for (int i = 0; i < R; ++i) wp[i] = c.w + static_cast<size_t>(min(rows[i], c.N - 1)) * c.ldw;
    const bool vec = ((c.K | c.ldw) & 7) == 0;
    const int kv = vec ? c.K : 0;
    uint4 w[R], wn[R];
    const int k_first = lane * 8;
#pragma unroll
    for (int i = 0; i < R; ++i) w[i] = k_first < kv ? __ldcs(reinterpret_cast<const uint4*>(wp[i] + k_first)) : make_uint4(0, 0, 0, 0);
    pdl_launch_dependents();
    pdl_wait();
    const T* x = static_cast<const T*>(c.x);
#pragma unroll
    for (int m = 0; m < M; ++m) {
        const T* xm = x + static_cast<size_t>(m) * c.ldx;
        if (sizeof(T) == 2 && vec && (c.ldx & 7) == 0) {
            for (int k = threadIdx.x * 8; k < c.K; k += 32 * kGemvWarps * 8) {
                const uint4 v = *reinterpret_cast<const uint4*>(xm + k);
                *reinterpret_cast<float4*>(xs + m * c.K + k) = make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y));
                *reinterpret_cast<float4*>(xs + m * c.K + k + 4) = make_float4(bf_lo(v.z), bf_hi(v.z), bf_lo(v.w), bf_hi(v.w));
            }
        } else {
            for (int k = threadIdx.x; k < c.K; k += 32 * kGemvWarps) xs[m * c.K + k] = to_f(xm[k]);
        }
    }
    __syncthreads();
    float acc[M][R] = {};
    for (int k = k_first; k < kv; k += 256) {
        const int kn = k + 256;
#pragma unroll
        for (int i = 0; i < R; ++i) wn[i] = kn < kv ? __ldcs(reinterpret_cast<const uint4*>(wp[i] + kn)) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int m = 0; m < M; ++m) {
            const float4 a = *reinterpret_cast<const float4*>(xs + m * c.K + k);
            const float4 b = *reinterpret_cast<const float4*>(xs + m * c.K + k + 4);
#pragma unroll
            for (int i = 0; i < R; ++i) {
                float s = acc[m][i];
                s = fmaf(bf_lo(w[i].x), a.x, s); s = fmaf(bf_hi(w[i].x), a.y, s);
                s = fmaf(bf_lo(w[i].y), a.z, s); s = fmaf(bf_hi(w[i].y), a.w, s);
                s = fmaf(bf_lo(w[i].z), b.x, s); s = fmaf(bf_hi(w[i].z), b.y, s);
                s = fmaf(bf_lo(w[i].w), b.z, s); s = fmaf(bf_hi(w[i].w), b.w, s);
                acc[m][i] = s;
            }
        }
#pragma unroll
        for (int i = 0; i < R; ++i) w[i] = wn[i];
    }
    for (int k = kv + lane; k < c.K; k += 32) {           // K not a multiple of 8: element by element
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const float v = to_f(wp[i][k]);
#pragma unroll
            for (int m = 0; m < M; ++m) acc[m][i] = fmaf(v, xs[m * c.K + k], acc[m][i]);
        }
    }
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int i = 0; i < R; ++i) acc[m][i] = warp_sum(acc[m][i]);
    if (lane >= M) return;
#pragma unroll
    for (int m = 0; m < M; ++m) {
        if (m != lane) continue;
        if (c.pair_cols) {
#pragma unroll
            for (int i = 0; i < R / 2; ++i) {
                const int n = unit * (R / 2) + i;
                if (n < c.pair_cols) store_pair(c, m, n, rows[2 * i], acc[m][2 * i], acc[m][2 * i + 1]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < R; ++i)
                if (rows[i] < c.N) store_out(c, m, rows[i], acc[m][i]);
        }
    }
}

template <typename T, int M, int R>
int launch_gemv_r(const DenseCall& c, cudaStream_t st) {
    static bool done[64] = {};
    const size_t smem = sizeof(float) * M * c.K;
    if (allow_smem(dense_gemv_kernel<T, M, R>, smem, done) != cudaSuccess) return TBL_ERR_CUDA;
    const int units = c.pair_cols ? ceil_div(c.pair_cols, R / 2) : ceil_div(c.N, R);
    return launch_dependent(dense_gemv_kernel<T, M, R>, dim3(ceil_div(units, kGemvWarps)), dim3(32 * kGemvWarps), smem, st, c) ==
                   cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

template <typename T, int M>
int launch_gemv_m(const DenseCall& c, cudaStream_t st) {
    // more rows per warp re-use the activations from shared memory, fewer keep every SM busy on short matrices
    const long long n = c.N;
    if (n >= 148LL * kGemvWarps * 4 * 4) return launch_gemv_r<T, M, 4>(c, st);
    if (n >= 148LL * kGemvWarps * 2 || c.pair_cols) return launch_gemv_r<T, M, 2>(c, st);
    return launch_gemv_r<T, M, 1>(c, st);
}

template <typename T>
int launch_gemv(const DenseCall& c, cudaStream_t st) {
    switch (c.M) {
        case 1: return launch_gemv_m<T, 1>(c, st);
        case 2: return launch_gemv_m<T, 2>(c, st);
        case 3: return launch_gemv_m<T, 3>(c, st);
        default: return launch_gemv_m<T, 4>(c, st);
    }
}

bool gemv_supported(const DenseCall& c) {
    return c.M <= kGemvMaxRows && sizeof(float) * c.M * c.K <= kGemvMaxSmem && (c.K % 4 == 0 || c.M == 1);
}

// Streaming the weights through warp-level MMAs beats the tcgen05 GEMM up to 16 rows, on narrow layers (too few tiles for
// the GEMM to fill the GPU) longer.
bool rows_pay(const DenseCall& c) {
    return c.batch > 0 || c.M <= 16 || static_cast<long long>(c.M) * c.N <= 32 * 4096;
}

}  // namespace

int launch_dense(int precision, int route, const DenseCall& call, cudaStream_t st) {
    if (call.M <= 0) return TBL_OK;
    DenseCall c = call;
    if (c.ldw == 0) c.ldw = c.K;
    const bool tensor = precision == TBL_BF16 && dense_tensor_supported(c);
    const bool rows = precision == TBL_BF16 && dense_rows_supported(c);
    if (route == kDenseAuto)
        route = rows && rows_pay(c) ? kDenseRows : (gemv_supported(c) ? kDenseGemv : (tensor ? kDenseTensor : kDenseSimt));
    if (route == kDenseRows) {
        if (!rows) return TBL_ERR_SHAPE;
        return launch_dense_rows(c, st) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
    }
    if (route == kDenseTensor) {
        if (!tensor) return TBL_ERR_SHAPE;
        return launch_dense_tensor(c, st) == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
    }
    if (route == kDenseGemv) {
        if (!gemv_supported(c)) return TBL_ERR_SHAPE;
        return precision == TBL_BF16 ? launch_gemv<bf16>(c, st) : launch_gemv<float>(c, st);
    }
    if (route != kDenseSimt) return TBL_ERR_INVALID_ARG;
    const dim3 grid(ceil_div(c.N, 64), ceil_div(c.M, 64));
    if (grid.y > 65535) return TBL_ERR_SHAPE;
    const cudaError_t e = precision == TBL_BF16 ? launch_dependent(dense_simt_kernel<bf16>, grid, dim3(256), 0, st, c)
                                                : launch_dependent(dense_simt_kernel<float>, grid, dim3(256), 0, st, c);
    return e == cudaSuccess ? TBL_OK : TBL_ERR_CUDA;
}

}  // namespace stack
}  // namespace tbl

using namespace tbl;
using namespace tbl::stack;

extern "C" {

int tbl_dense_forward(const tbl_dense_view* view, int precision, int route, const void* x_dev, int ldx, int rows,
                      const float* residual_dev, float* out_dev, void* stream) {
    if (!view || !view->weight || !x_dev || !out_dev || rows <= 0 || view->inputs <= 0 || view->outputs <= 0 || ldx < view->inputs ||
        (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    if (reinterpret_cast<uintptr_t>(view->weight) & 15) return TBL_ERR_ALIGNMENT;
    DenseCall c{};
    c.x = x_dev; c.w = static_cast<const bf16*>(view->weight); c.bias = view->bias; c.ldx = ldx;
    c.M = rows; c.K = view->inputs; c.N = view->outputs; c.out_f32 = out_dev; c.ldo = view->outputs; c.residual = residual_dev;
    return launch_dense(precision, route, c, static_cast<cudaStream_t>(stream));
}

int tbl_gated_dense_forward(const tbl_dense_view* gate_up, int precision, int route, const void* x_dev, int ldx, int rows,
                            int ff, void* out_dev, void* stream) {
    return tbl_gated_dense_act_forward(gate_up, precision, route, TBL_ACT_SILU, x_dev, ldx, rows, ff, out_dev, stream);
}

int tbl_gated_dense_act_forward(const tbl_dense_view* gate_up, int precision, int route, int activation, const void* x_dev, int ldx,
                                int rows, int ff, void* out_dev, void* stream) {
    if (activation != TBL_ACT_SILU && activation != TBL_ACT_GELU_TANH) return TBL_ERR_INVALID_ARG;
    if (!gate_up || !gate_up->weight || !x_dev || !out_dev || rows <= 0 || ff <= 0 || gate_up->inputs <= 0 ||
        ldx < gate_up->inputs || (precision != TBL_F32 && precision != TBL_BF16))
        return TBL_ERR_INVALID_ARG;
    if (gate_up->outputs != 2 * static_cast<int>(stack::round_up(ff, TBL_PAIR_BLOCK))) return TBL_ERR_SHAPE;
    if (reinterpret_cast<uintptr_t>(gate_up->weight) & 15) return TBL_ERR_ALIGNMENT;
    DenseCall c{};
    c.x = x_dev; c.w = static_cast<const bf16*>(gate_up->weight); c.bias = gate_up->bias; c.ldx = ldx;
    c.M = rows; c.K = gate_up->inputs; c.N = gate_up->outputs; c.ldo = ff; c.pair_cols = ff; c.act = activation;
    if (precision == TBL_BF16) c.out_b16 = static_cast<bf16*>(out_dev); else c.out_f32 = static_cast<float*>(out_dev);
    return launch_dense(precision, route, c, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
