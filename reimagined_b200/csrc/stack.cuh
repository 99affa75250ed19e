// Internal declarations shared by the translation units of libstack_b200.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/layer_stack.h"
#include "common.cuh"

namespace tbl {
namespace stack {

using bf16 = __nv_bfloat16;

constexpr int kNumSm = 148;

inline size_t round_up(size_t v, size_t a) { return (v + a - 1) / a * a; }
inline int ceil_div(long long a, long long b) { return static_cast<int>((a + b - 1) / b); }

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// Activation of a gated feed-forward, TBL_ACT_*: z sigmoid(z (lin + cubic z^2)).  With (1, 0) that is silu; the tanh form
// of gelu is z (1 + tanh(a)) / 2 = z sigmoid(2 a), a = sqrt(2/pi) (z + 0.044715 z^3).
struct Activation { float lin, cubic; };
__device__ __forceinline__ Activation activation_of(int act) {
    return act == TBL_ACT_GELU_TANH ? Activation{1.5957691216f, 0.0713548163f} : Activation{1.0f, 0.0f};
}
__device__ __forceinline__ float activate(const Activation& a, float z) { return z * sigmoid_f(z * fmaf(z * z, a.cubic, a.lin)); }

// the two bf16 halves of a 32-bit word, widened
__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

// warp-level MMA 16 x 8 x 16, bf16 operands, fp32 accumulators
__device__ __forceinline__ void mma16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    mma16816(d, a[0], a[1], a[2], a[3], b0, b1);
}

__device__ __forceinline__ float ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Launch as a programmatic dependent of the kernel before it on the stream: the kernel must call pdl_wait() before it
// touches anything an earlier kernel of the step writes.
template <typename... Params, typename... Args>
cudaError_t launch_dependent(void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args... args) {
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = 1;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, static_cast<Params>(args)...);
    note_launch();
    return e;
}

// Raises a kernel's dynamic shared memory limit once per device, to what its static shared memory leaves.
template <typename Kernel>
cudaError_t allow_smem(Kernel kernel, size_t bytes, bool (&done)[64]) {
    if (bytes <= 48 * 1024) return cudaSuccess;
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev >= 0 && dev < 64 && done[dev]) return cudaSuccess;
    cudaFuncAttributes attr{};
    cudaError_t e = cudaFuncGetAttributes(&attr, kernel);
    if (e == cudaSuccess)
        e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - static_cast<int>(attr.sharedSizeBytes));
    if (e == cudaSuccess && dev >= 0 && dev < 64) done[dev] = true;
    return e;
}

// ---- dense.cu / dense_tcgen05.cu: y = W x + b with bf16 weights ------------------------------------------------
struct DenseCall {
    const void* x;           // activations, the precision's type
    const bf16* w;           // [N, K], ldw between rows (0: K)
    const float* bias;       // [N] or null
    int ldx, M, K, N, ldw;
    float* out_f32;          // exactly one of the two outputs
    bf16* out_b16;
    int ldo, act;            // act: TBL_ACT_* of a gated pair
    const float* residual;   // fp32, ld = ldo, added to out_f32 (may alias it); null: none
    int pair_cols;           // > 0: rows of w alternate in blocks of 32 gate / 32 up rows, out = act(gate) * up,
                             //      clipped at this many columns
    // row-streaming kernel only: `batch` products of one launch (0: one), their strides in elements, and an output
    // gate: out *= sigmoid(gate[m * ldg + n])
    int batch, ldg, batch_gate;
    long long batch_w, batch_x, batch_out;
    const float* gate;
};
enum DenseRoute { kDenseAuto = 0, kDenseSimt = 1, kDenseGemv = 2, kDenseTensor = 3, kDenseRows = 4 };
int launch_dense(int precision, int route, const DenseCall& c, cudaStream_t st);
bool dense_rows_supported(const DenseCall& c);
cudaError_t launch_dense_rows(const DenseCall& c, cudaStream_t st);
bool dense_tensor_supported(const DenseCall& c);
cudaError_t launch_dense_tensor(const DenseCall& c, cudaStream_t st);

// ---- stack_glue.cu ----------------------------------------------------------------------------------------------
struct DepthNorm {
    const float* history;    // [count][rows of the source][width]
    size_t stride;
    int count;
    const float* weights;    // null: the last array alone
    const int32_t* tokens;   // not null: the row is table[token] * embed_scale instead (and history is not read)
    const bf16* table;
    int vocab;
    float embed_scale;
    const int32_t* row_index;
    int rows, width;
    float eps;
    // streams > 0: the source are this many residual streams instead, updated with the last sublayer's result first;
    // `weights` then make the sublayer input out of them (null: ones) and `trace` receives their plain sum
    int streams, store;      // store: write the updated streams back (embedding: write them)
    float* stream;           // [streams] arrays at `stride`
    const float *y, *mix, *out_weights;      // y null: no update
    int norm_kind;           // TBL_NORM_*
    float alpha;
    const float* norm_bias;
    const float* norm;       // null: no h
    float* x;
    float* trace;
    void* h;
    int32_t* positions;      // not null: block 0 adds n_tok to positions[slots[s]] for s < n_seq
    const int32_t* slots;
    int n_seq, n_tok;
};
int launch_depth_norm(int precision, const DepthNorm& p, cudaStream_t st);

// ---- delta_rule.cu ----------------------------------------------------------------------------------------------
size_t delta_workspace(const tbl_delta_mixer& m, int precision, int rows);
int launch_delta(const tbl_delta_mixer& m, int precision, int route, float eps, const float* proj, float* states,
                 const int32_t* slots, int n_seq, int n_tok, void* out, void* ws, cudaStream_t st);

// ---- latent_attention.cu ------------------------------------------------------------------------------------------
size_t latent_workspace(const tbl_latent_mixer& m, int precision, int n_seq, int n_tok, int context);
int launch_latent(const tbl_latent_mixer& m, int precision, int route, float eps, const float* proj, void* cache,
                  int capacity, const int32_t* slots, const int32_t* positions, int n_seq, int n_tok, int context,
                  void* out, void* ws, cudaStream_t st);
int latent_cache_width(const tbl_latent_mixer& m);     // cached numbers per token, padded to 16 bytes of bf16
// ---- attention.cu --------------------------------------------------------------------------------------------------
size_t attention_workspace(const tbl_attention_mixer& m, int precision, int n_seq, int n_tok, int context);
int launch_attention(const tbl_attention_mixer& m, int precision, int route, float eps, const float* proj, void* cache, int n_slots,
                     int capacity, const int32_t* slots, const int32_t* positions, int n_seq, int n_tok, int context, void* out,
                     void* ws, cudaStream_t st);
int attention_cache_width(const tbl_attention_mixer& m);      // cached numbers per token and key/value head
int check_attention(const tbl_attention_mixer& m, int width);

int check_delta(const tbl_delta_mixer& m, int width);
int check_latent(const tbl_latent_mixer& m, int width);

}  // namespace stack
}  // namespace tbl
