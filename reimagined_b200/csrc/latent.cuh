// Shared by the latent-attention translation units (latent_attention.cu, latent_decode.cu, latent_prefill.cu).
#pragma once

#include "stack.cuh"

namespace tbl {
namespace stack {

struct LatentParams {
    const float* proj;           // [rows][ld]: W_dq h | W_dkv h | W_g h
    const float *q_norm, *kv_norm, *rope_cos, *rope_sin;
    const bf16 *uk, *uk_t, *uv;
    void* cache;                 // [slots][capacity][cw], the precision's type: latent | rotated key part
    const int32_t *slots, *positions;
    void *cq, *qa;               // query latent [rows][ldq]; absorbed query [rows][H][cw], or the rotated query
    float* q;                    // [rows][H][d + rd]
    bf16 *q16, *lat;             // the same in bf16; attention's result in the latent space [rows][H][R]
    float *part_m, *part_l, *part_o;   // [rows][H][splits] ([R])
    bf16 *keys, *values, *gathered;    // expanded context: [sequence x context][H*d], [H*vd][sequence x context]; its latents
    void* out;                   // [rows][H*vd]
    int* status;
    int ld, ldq, cw, H, d, rd, vd, R, q_rank, capacity, rope_positions, n_tok, splits, context;
    float scale, eps;
};

// latent_decode.cu: attention over the latent cache on tensor cores
bool latent_tensor_supported(const tbl_latent_mixer& m);
int latent_tensor_heads(const tbl_latent_mixer& m);      // heads per CTA
int launch_latent_tensor(const LatentParams& p, int rows, cudaStream_t st);

// latent_prefill.cu: attention over expanded keys and values on tensor cores
bool latent_expanded_supported(const tbl_latent_mixer& m);
int latent_expanded_context(int context);                // padded to whole blocks
int launch_latent_expanded(const tbl_latent_mixer& m, const LatentParams& p, int n_seq, cudaStream_t st);

}  // namespace stack
}  // namespace tbl
