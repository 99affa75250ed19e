// Shared by the attention translation units (attention.cu, attention_decode.cu, attention_prefill.cu).
//
// Cache of a layer: [slot][kv head][token][cw], a token's row being its keys (one per map, each padded to dp) and its
// values (padded to vp); the padding is zero.  Query rows that share a key/value head -- the tokens of a sequence's
// portion x the query heads of the group -- are numbered token * group + head and handled in blocks of 16.
#pragma once

#include "stack.cuh"

namespace tbl {
namespace stack {

struct AttnParams {
    const float* proj;           // [rows][ld]: q | k | v | gate
    const float* temperature;    // per position; null: 1
    void* cache;                 // the precision's type
    const int32_t *slots, *positions;
    bf16* q16;                   // flash: queries x temperature, [rows][H][maps][dp]
    float *part_m, *part_l;      // [rows][H][maps][splits]: maximum (of score * log2 e) and sum of a split
    float* part_o;               // the same x [vp], not normalised
    void* out;                   // [rows][H * vd]
    int* status;
    int ld, k_off, v_off, g_off; // columns of proj; g_off < 0: no output gate
    int H, G, group, maps, d, vd, dp, vp, cw;
    int n_slots, capacity, temperature_positions, n_tok, splits, append, vec;
    float scale_log2, lambda, out_scale, eps;
};

__device__ __forceinline__ float temperature_of(const AttnParams& p, int pos) {
    return p.temperature ? __ldg(p.temperature + min(max(pos, 0), p.temperature_positions - 1)) : 1.0f;
}
// cache row of a token
__device__ __forceinline__ size_t cache_row(const AttnParams& p, int slot, int g, int token) {
    return ((static_cast<size_t>(slot) * p.G + g) * p.capacity + token) * p.cw;
}
// one number of a token's cache row, from the projections
__device__ __forceinline__ float cache_value(const AttnParams& p, const float* proj_row, int g, int c) {
    if (c < p.maps * p.dp) {
        const int map = c / p.dp, e = c - map * p.dp;
        return e < p.d ? proj_row[p.k_off + (g * p.maps + map) * p.d + e] : 0.0f;
    }
    const int e = c - p.maps * p.dp;
    return e < p.vd ? proj_row[p.v_off + g * p.vd + e] : 0.0f;
}

// attention_decode.cu: streams the cache, warp-level MMAs.  Up to kClusterSplits splits of the context are a cluster that
// finishes the rows itself, more leave partial sums.
constexpr int kClusterSplits = 8;
bool attention_stream_supported(const tbl_attention_mixer& m);
int launch_attention_stream(const AttnParams& p, int n_seq, cudaStream_t st);

// attention_prefill.cu: flash attention on tcgen05
bool attention_flash_supported(const tbl_attention_mixer& m);
bool attention_flash_whole(const tbl_attention_mixer& m);    // a CTA holds a head's whole output (otherwise it leaves partial sums)
int launch_attention_flash(const AttnParams& p, int n_seq, cudaStream_t st);

}  // namespace stack
}  // namespace tbl
